// Passes over rows of the 32-bit residual stream that do several things on one read of the row.
//
//   embed_rows_kernel   out[t] = table[tok] * scale + bigram row, then optionally an RMS norm whose result stays 32-bit. The
//                       bigram row of a token is (previous * mul_prev + token * mul_cur) mod buckets, of a sequence's first
//                       token the table's last row; the previous token of a portion's first row is the request's state.
//   two_norms_kernel    x (+= a second stream and a vector), then the RMS norms of x with two weights, one row sum for both
#include "common.cuh"

struct EmbedRowsArgs {
  const void* table;
  const void* bigram;        // [buckets + 1][H] or null
  const int* tok;            // [T]
  const int* pos;            // [T]
  const int* row_req;        // [T]
  const int* q_start;        // [R]
  const int* q_len;          // [R]
  const int* slot;           // [R]
  int* prev;                 // [slots]: the last token of what the request has run so far
  const float* norm_w;       // [H] or null
  float* out;                // [T][H]
  float* copy;               // [T][H] or null: the same rows once more
  int H, buckets;
  long long mul_prev, mul_cur;
  float scale, eps;
};

// The bigram row of row t. The block of a portion's first row is the only one that reads the request's state, and the one
// that then leaves the portion's last token in it. Called by one thread.
__device__ __forceinline__ int bigram_row(const EmbedRowsArgs& A, int t) {
  const int r = A.row_req[t], first = A.q_start[r];
  const long long cur = A.tok[t];
  long long before = 0;
  if (t == first) {
    before = A.prev[A.slot[r]];
    A.prev[A.slot[r]] = A.tok[first + A.q_len[r] - 1];
  } else {
    before = A.tok[t - 1];
  }
  return A.pos[t] == 0 ? A.buckets : (int)((before * A.mul_prev + cur * A.mul_cur) % A.buckets);
}

template <typename TE>
__global__ void __launch_bounds__(256) embed_rows_kernel(EmbedRowsArgs A) {
  __shared__ float sh[32];
  __shared__ int brow;
  hb_pdl_launch();
  hb_pdl_wait();
  const int t = blockIdx.x, H = A.H;
  if (A.bigram && threadIdx.x == 0) brow = bigram_row(A, t);
  __syncthreads();
  const TE* src = (const TE*)A.table + (size_t)A.tok[t] * H;
  const TE* bg = A.bigram ? (const TE*)A.bigram + (size_t)brow * H : nullptr;
  float* dst = A.out + (size_t)t * H;
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += 256) {
    const float v = __fadd_rn(__fmul_rn(hb_to_float(src[i]), A.scale), bg ? hb_to_float(bg[i]) : 0.f);
    dst[i] = v;
    ss = fmaf(v, v, ss);
  }
  const float inv = A.norm_w ? rsqrtf(hb_block_sum(ss, sh) / (float)H + A.eps) : 1.f;
  for (int i = threadIdx.x; i < H; i += 256) {        // a thread reads back what it wrote itself
    const float v = A.norm_w ? A.norm_w[i] * (dst[i] * inv) : dst[i];
    dst[i] = v;
    if (A.copy) A.copy[(size_t)t * H + i] = v;
  }
}

template <typename TE, int NV>
__global__ void __launch_bounds__(256) embed_rows_vec_kernel(EmbedRowsArgs A) {
  __shared__ float sh[32];
  __shared__ int brow;
  hb_pdl_launch();
  hb_pdl_wait();
  const int t = blockIdx.x, H = A.H, nvec = H >> 2;
  if (A.bigram && threadIdx.x == 0) brow = bigram_row(A, t);
  const TE* src = (const TE*)A.table + (size_t)A.tok[t] * H;
  float4 v[NV];
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = threadIdx.x + i * 256;
    v[i] = c < nvec ? hb_load4(src + 4 * c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  __syncthreads();
  const TE* bg = A.bigram ? (const TE*)A.bigram + (size_t)brow * H : nullptr;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = threadIdx.x + i * 256;
    const float4 b = bg && c < nvec ? hb_load4(bg + 4 * c) : make_float4(0.f, 0.f, 0.f, 0.f);
    v[i].x = __fadd_rn(__fmul_rn(v[i].x, A.scale), b.x);
    v[i].y = __fadd_rn(__fmul_rn(v[i].y, A.scale), b.y);
    v[i].z = __fadd_rn(__fmul_rn(v[i].z, A.scale), b.z);
    v[i].w = __fadd_rn(__fmul_rn(v[i].w, A.scale), b.w);
    ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss);
    ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss);
  }
  const float inv = A.norm_w ? rsqrtf(hb_block_sum(ss, sh) / (float)H + A.eps) : 1.f;
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = threadIdx.x + i * 256;
    if (c >= nvec) continue;
    float4 o = v[i];
    if (A.norm_w) {
      const float4 w = hb_load4(A.norm_w + 4 * c);
      o = make_float4(w.x * (o.x * inv), w.y * (o.y * inv), w.z * (o.z * inv), w.w * (o.w * inv));
    }
    hb_store4(A.out + (size_t)t * H + 4 * c, o);
    if (A.copy) hb_store4(A.copy + (size_t)t * H + 4 * c, o);
  }
}

// table, bigram: [*, H] of one element type; prev int32 [slots] (with bigram); norm_w float32 or null; copy or null.
HB_EXPORT int hb_embed_rows(const void* table, const void* bigram, int dt, const int* tok, const int* pos, const int* row_req,
                            const int* q_start, const int* q_len, const int* slot, int* prev, const float* norm_w, float* out,
                            float* copy, int T, int H, int buckets, long mul_prev, long mul_cur, float scale, float eps,
                            cudaStream_t s) {
  if (T <= 0) return 0;
  if (bigram && (buckets <= 0 || mul_prev < 0 || mul_cur < 0 || !pos || !row_req || !q_start || !q_len || !slot || !prev))
    HB_FAIL("hb_embed_rows: a bigram table needs its sizes, the rows' places and the requests' state");
  EmbedRowsArgs A{table, bigram, tok, pos, row_req, q_start, q_len, slot, prev, norm_w, out, copy, H, buckets, mul_prev, mul_cur, scale, eps};
  const bool aligned = !(((uintptr_t)table | (uintptr_t)bigram | (uintptr_t)norm_w | (uintptr_t)out | (uintptr_t)copy) & 15);
  if ((H & 3) == 0 && H <= 8192 && aligned) {
    if (H <= 2048) HB_DISPATCH_1(dt, "hb_embed_rows", (hb_launch(embed_rows_vec_kernel<TA, 2>, T, 256, 0, s, A)));
    else HB_DISPATCH_1(dt, "hb_embed_rows", (hb_launch(embed_rows_vec_kernel<TA, 8>, T, 256, 0, s, A)));
  } else {
    HB_DISPATCH_1(dt, "hb_embed_rows", (hb_launch(embed_rows_kernel<TA>, T, 256, 0, s, A)));
  }
  HB_CHECK_LAUNCH("hb_embed_rows");
  return 0;
}

// ---------------------------------------------------------------------------------------
// x[t] (+= add[t]) (+= vec), written back where it changed; y1 = w1 x / rms(x), y2 = w2 x / rms(x) (either may be absent).
// ---------------------------------------------------------------------------------------
struct TwoNormsArgs {
  float* x;              // [T][H]
  const float* add;      // [T][H] or null
  const float* vec;      // [H] or null
  const float* w1;       // [H]
  const float* w2;       // [H]
  void* y1;              // [T][H] or null
  void* y2;
  int H;
  float eps;
};

template <typename TO>
__global__ void __launch_bounds__(256) two_norms_kernel(TwoNormsArgs A) {
  __shared__ float sh[32];
  hb_pdl_launch();
  hb_pdl_wait();
  const int H = A.H;
  const size_t r = (size_t)blockIdx.x * H;
  float ss = 0.f;
  for (int i = threadIdx.x; i < H; i += 256) {
    float v = A.x[r + i];
    if (A.add) v = __fadd_rn(v, A.add[r + i]);
    if (A.vec) v = __fadd_rn(v, A.vec[i]);
    if (A.add || A.vec) A.x[r + i] = v;
    ss = fmaf(v, v, ss);
  }
  if (!A.y1 && !A.y2) return;
  const float inv = rsqrtf(hb_block_sum(ss, sh) / (float)H + A.eps);
  for (int i = threadIdx.x; i < H; i += 256) {
    const float v = A.x[r + i] * inv;
    if (A.y1) ((TO*)A.y1)[r + i] = hb_from_float<TO>(A.w1[i] * v);
    if (A.y2) ((TO*)A.y2)[r + i] = hb_from_float<TO>(A.w2[i] * v);
  }
}

template <typename TO, int NV>
__global__ void __launch_bounds__(256) two_norms_vec_kernel(TwoNormsArgs A) {
  __shared__ float sh[32];
  hb_pdl_launch();
  hb_pdl_wait();
  const int H = A.H, nvec = H >> 2;
  const size_t r = (size_t)blockIdx.x * H;
  float4 v[NV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = threadIdx.x + i * 256;
    v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < nvec) {
      v[i] = hb_load4(A.x + r + 4 * c);
      if (A.add) {
        const float4 a = hb_load4(A.add + r + 4 * c);
        v[i] = make_float4(__fadd_rn(v[i].x, a.x), __fadd_rn(v[i].y, a.y), __fadd_rn(v[i].z, a.z), __fadd_rn(v[i].w, a.w));
      }
      if (A.vec) {
        const float4 a = hb_load4(A.vec + 4 * c);
        v[i] = make_float4(__fadd_rn(v[i].x, a.x), __fadd_rn(v[i].y, a.y), __fadd_rn(v[i].z, a.z), __fadd_rn(v[i].w, a.w));
      }
      if (A.add || A.vec) hb_store4(A.x + r + 4 * c, v[i]);
    }
    ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss);
    ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss);
  }
  if (!A.y1 && !A.y2) return;
  const float inv = rsqrtf(hb_block_sum(ss, sh) / (float)H + A.eps);
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int c = threadIdx.x + i * 256;
    if (c >= nvec) continue;
    const float4 n = make_float4(v[i].x * inv, v[i].y * inv, v[i].z * inv, v[i].w * inv);
    if (A.y1) {
      const float4 w = hb_load4(A.w1 + 4 * c);
      hb_store4((TO*)A.y1 + r + 4 * c, make_float4(w.x * n.x, w.y * n.y, w.z * n.z, w.w * n.w));
    }
    if (A.y2) {
      const float4 w = hb_load4(A.w2 + 4 * c);
      hb_store4((TO*)A.y2 + r + 4 * c, make_float4(w.x * n.x, w.y * n.y, w.z * n.z, w.w * n.w));
    }
  }
}

HB_EXPORT int hb_two_norms(float* x, const float* add, const float* vec, const float* w1, const float* w2, void* y1, void* y2,
                           int y_dt, int T, int H, float eps, cudaStream_t s) {
  if (T <= 0) return 0;
  if ((y1 && !w1) || (y2 && !w2)) HB_FAIL("hb_two_norms: a norm without its weight");
  TwoNormsArgs A{x, add, vec, w1, w2, y1, y2, H, eps};
  const bool aligned = !(((uintptr_t)x | (uintptr_t)add | (uintptr_t)vec | (uintptr_t)w1 | (uintptr_t)w2 | (uintptr_t)y1 | (uintptr_t)y2) & 15);
  if ((H & 3) == 0 && H <= 8192 && aligned) {
    if (H <= 2048) HB_DISPATCH_1(y_dt, "hb_two_norms", (hb_launch(two_norms_vec_kernel<TA, 2>, T, 256, 0, s, A)));
    else if (H <= 4096) HB_DISPATCH_1(y_dt, "hb_two_norms", (hb_launch(two_norms_vec_kernel<TA, 4>, T, 256, 0, s, A)));
    else HB_DISPATCH_1(y_dt, "hb_two_norms", (hb_launch(two_norms_vec_kernel<TA, 8>, T, 256, 0, s, A)));
  } else {
    HB_DISPATCH_1(y_dt, "hb_two_norms", (hb_launch(two_norms_kernel<TA>, T, 256, 0, s, A)));
  }
  HB_CHECK_LAUNCH("hb_two_norms");
  return 0;
}
