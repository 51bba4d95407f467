// Recurrences with one state matrix per head, S [N][P] (key channel by value channel), carried from token to token in 32-bit:
//
//   linear   S <- a S + b k v^T;  n <- a n + b k;  o = S^T q,  nq = n . q         (a, b: a number per token and head)
//   delta    S <- a S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q
//
// The linear form with a normaliser n is the matrix memory of an exponentially gated LSTM; the delta form the gated delta
// rule. What does not depend on the state is made for all tokens at once by kernels of its own, what follows the read-out
// likewise, so that the serial part is the walk alone:
//   ms_exp_gates_kernel     log gates -> a, b and exp(-m) with the running maximum m (a max-plus scan over the tokens)
//   ms_delta_prepare_kernel q, k to unit length, k . q, the decay a and the write strength b
//   ms_walk_kernel          the walk
//   ms_finish_kernel        the normaliser, the head's root mean square, a weight and an output gate; rounded once
//   ms_single_kernel        all of it for requests that bring one token each (decoding)
// The value columns of S are independent of one another, so a head's columns are split over blocks. Long portions of the
// linear form run in pieces of L tokens over the whole GPU: every piece from a zero state (its own contribution and the
// product of its decays), then the pieces' starting states one after another (ms_carry_kernel), then every piece again
// from its starting state for o. Requests, lengths and state slots come from device arrays, so a decode step can be
// replayed from a CUDA graph; where a portion or a piece starts changes a token's result by rounding only.
#include "common.cuh"

constexpr int MS_PT_THREADS = 128;      // threads of the value columns of a block; a warp beside them keeps n (linear form)

struct StateArgs {
  const float* q; const float* k; const float* v; long ldq, ldk, ldv;     // rows; head h reads q, k of group h / (H / G)
  const float* a; const float* b;         // [T][H]
  const float* kq;                        // [T][G] (delta): k . q with q as it is in the rows
  float* state; float* nstate;            // [slots][H][N][P], [slots][H][N] or null
  const int* q_start; const int* q_len; const int* slot;
  float* y;                               // [T][H P]
  float* nq;                              // [T][H] (with nstate)
  int H, G, N, P, KS, PT, CH, vec4;
  float q_scale;                          // multiplies o and nq
  float* piece_state; float* piece_n; float* piece_decay;    // [all requests' pieces][H][N][P], [.][H][N], [.][H]
  int L, pieces;
};

enum { MS_WHOLE = 0, MS_PIECE_LOCAL = 1, MS_PIECE_OUT = 2 };

__device__ __forceinline__ void ms_cp16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void ms_cp4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
// The first piece of request r among all requests' pieces (they lie one after another).
__device__ __forceinline__ int ms_piece_base(const int* __restrict__ q_len, int r, int L) {
  int base = 0;
  for (int i = 0; i < r; i++) base += (q_len[i] + L - 1) / L;
  return base;
}

// grid (heads x column tiles, requests[, pieces]). KS neighbouring lanes share a value column; each holds DPT contiguous key
// channels of it. A token's k and q lie in shared memory padded with zeros to KS slices of DPT (and 4 floats of padding a
// slice, so that the slices fall on different banks): no bounds are checked in the walk. Rows come a chunk of CH tokens ahead
// by cp.async. The walk itself has no barrier.
template <int DPT, bool DELTA, int MODE>
__global__ void __launch_bounds__(MS_PT_THREADS + 32) ms_walk_kernel(StateArgs A) {
  extern __shared__ __align__(16) float msm[];
  hb_pdl_launch();
  hb_pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nthr = blockDim.x, nwarp = nthr >> 5;
  const int H = A.H, N = A.N, P = A.P, KS = A.KS, PT = A.PT, CH = A.CH;
  const int tiles = (P + PT - 1) / PT, h = blockIdx.x / tiles, p0 = (blockIdx.x - h * tiles) * PT;
  const int g = h / (H / A.G), r = blockIdx.y;
  const bool nwarp_here = !DELTA && tid >= MS_PT_THREADS;          // the warp that keeps the normaliser
  const int pl = nwarp_here ? 0 : tid / KS, ks = tid % KS, p = p0 + pl;
  const bool live = nwarp_here ? (p0 == 0 && lane < KS) : p < P;
  const int t0 = A.q_start[r];
  const int j_begin = MODE == MS_WHOLE ? 0 : (int)blockIdx.z * A.L;
  const int len = MODE == MS_WHOLE ? A.q_len[r] : min(A.q_len[r], j_begin + A.L);
  if (j_begin >= len) return;
  const int KQ = KS * (DPT + 4);
  const int RW = 2 * KQ + PT + 4;          // a token's row: [k | q | v of the tile | a, b, k . q, -]
  const size_t piece = MODE == MS_WHOLE ? 0 : (size_t)ms_piece_base(A.q_len, r, A.L) + blockIdx.z;
  float* S_g;
  if (nwarp_here) S_g = (MODE == MS_WHOLE ? A.nstate + ((size_t)A.slot[r] * H + h) * N : A.piece_n + (piece * H + h) * N);
  else S_g = (MODE == MS_WHOLE ? A.state + ((size_t)A.slot[r] * H + h) * N * P : A.piece_state + (piece * H + h) * N * P) + p;
  const int ss = nwarp_here ? 1 : P;
  float S[DPT];
#pragma unroll
  for (int i = 0; i < DPT; i++) {
    const int n = ks * DPT + i;
    S[i] = (MODE != MS_PIECE_LOCAL && live && n < N) ? S_g[(size_t)n * ss] : 0.f;
  }
  if (KS * DPT > N || p0 + PT > P) {          // the padding is read as zeros
    for (int i = tid; i < 2 * CH * RW; i += nthr) msm[i] = 0.f;
    __syncthreads();
  }
  const float* qh = A.q + (size_t)g * N;
  const float* kh = A.k + (size_t)g * N;
  const float* vh = A.v + (size_t)h * P + p0;
  const int np = min(PT, P - p0);
  auto pidx = [](int n) { return n + (n / DPT) * 4; };
  auto fetch = [&](int buf, int c0) {         // a warp a token
    const int n = min(CH, len - c0);
    for (int j = warp; j < n; j += nwarp) {
      float* row = msm + (buf * CH + j) * RW;
      const size_t t = (size_t)(t0 + c0 + j);
      if (A.vec4) {
        for (int c = lane * 4; c < N; c += 128) {
          ms_cp16(row + pidx(c), kh + t * A.ldk + c);
          if (MODE != MS_PIECE_LOCAL) ms_cp16(row + KQ + pidx(c), qh + t * A.ldq + c);
        }
        for (int c = lane * 4; c < np; c += 128) ms_cp16(row + 2 * KQ + c, vh + t * A.ldv + c);
      } else {
        for (int c = lane; c < N; c += 32) {
          ms_cp4(row + pidx(c), kh + t * A.ldk + c);
          if (MODE != MS_PIECE_LOCAL) ms_cp4(row + KQ + pidx(c), qh + t * A.ldq + c);
        }
        for (int c = lane; c < np; c += 32) ms_cp4(row + 2 * KQ + c, vh + t * A.ldv + c);
      }
      if (lane == 0) ms_cp4(row + 2 * KQ + PT, A.a + t * H + h);
      if (lane == 1) ms_cp4(row + 2 * KQ + PT + 1, A.b + t * H + h);
      if (DELTA && lane == 2) ms_cp4(row + 2 * KQ + PT + 2, A.kq + t * A.G + g);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, j_begin);
  float decays = 1.f;
  int buf = 0;
  const int sb = ks * (DPT + 4);
  float* yp = nwarp_here ? A.nq + (size_t)t0 * H + h : A.y + (size_t)t0 * H * P + (size_t)h * P + p;
  const size_t ystep = nwarp_here ? (size_t)H : (size_t)H * P;
  for (int c0 = j_begin; c0 < len; c0 += CH, buf ^= 1) {
    const int n = min(CH, len - c0);
    if (c0 + CH < len) {
      fetch(buf ^ 1, c0 + CH);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float* row = msm + buf * CH * RW;
    if (!nwarp_here || p0 == 0) {
#pragma unroll 2
      for (int j = 0; j < n; j++, row += RW) {
        const float4 sc = *(const float4*)(row + 2 * KQ + PT);           // a, b, k . q
        const float vv = nwarp_here ? 1.f : row[2 * KQ + pl];
        if constexpr (!DELTA) {
          const float xv = sc.y * vv;
          if constexpr (MODE == MS_PIECE_LOCAL) {
            decays *= sc.x;
#pragma unroll
            for (int i = 0; i < DPT; i += 4) {
              const float4 kv = *(const float4*)(row + sb + i);
              S[i] = fmaf(sc.x, S[i], kv.x * xv);
              S[i + 1] = fmaf(sc.x, S[i + 1], kv.y * xv);
              S[i + 2] = fmaf(sc.x, S[i + 2], kv.z * xv);
              S[i + 3] = fmaf(sc.x, S[i + 3], kv.w * xv);
            }
          } else {
            float o0 = 0.f, o1 = 0.f, o2 = 0.f, o3 = 0.f;
#pragma unroll
            for (int i = 0; i < DPT; i += 4) {
              const float4 kv = *(const float4*)(row + sb + i), qv = *(const float4*)(row + KQ + sb + i);
              S[i] = fmaf(sc.x, S[i], kv.x * xv);
              S[i + 1] = fmaf(sc.x, S[i + 1], kv.y * xv);
              S[i + 2] = fmaf(sc.x, S[i + 2], kv.z * xv);
              S[i + 3] = fmaf(sc.x, S[i + 3], kv.w * xv);
              o0 = fmaf(S[i], qv.x, o0);
              o1 = fmaf(S[i + 1], qv.y, o1);
              o2 = fmaf(S[i + 2], qv.z, o2);
              o3 = fmaf(S[i + 3], qv.w, o3);
            }
            float o = (o0 + o1) + (o2 + o3);
            for (int m = 1; m < KS; m <<= 1) o += __shfl_xor_sync(0xffffffffu, o, m);
            if (live && ks == 0) yp[(size_t)(c0 + j) * ystep] = o * A.q_scale;
          }
        } else {
          float o0 = 0.f, o1 = 0.f, u0 = 0.f, u1 = 0.f;
#pragma unroll
          for (int i = 0; i < DPT; i += 4) {
            const float4 kv = *(const float4*)(row + sb + i), qv = *(const float4*)(row + KQ + sb + i);
            u0 = fmaf(S[i], kv.x, u0);
            o0 = fmaf(S[i], qv.x, o0);
            u1 = fmaf(S[i + 1], kv.y, u1);
            o1 = fmaf(S[i + 1], qv.y, o1);
            u0 = fmaf(S[i + 2], kv.z, u0);
            o0 = fmaf(S[i + 2], qv.z, o0);
            u1 = fmaf(S[i + 3], kv.w, u1);
            o1 = fmaf(S[i + 3], qv.w, o1);
          }
          float u = u0 + u1, o = o0 + o1;
          for (int m = 1; m < KS; m <<= 1) {
            u += __shfl_xor_sync(0xffffffffu, u, m);
            o += __shfl_xor_sync(0xffffffffu, o, m);
          }
          // both sums read the state before this token: S^T q after the write is a S^T q + (k . q) u
          u = sc.y * fmaf(-sc.x, u, vv);
          o = fmaf(sc.z, u, sc.x * o);
          if (live && ks == 0) yp[(size_t)(c0 + j) * ystep] = o * A.q_scale;
#pragma unroll
          for (int i = 0; i < DPT; i += 4) {
            const float4 kv = *(const float4*)(row + sb + i);
            S[i] = fmaf(kv.x, u, sc.x * S[i]);
            S[i + 1] = fmaf(kv.y, u, sc.x * S[i + 1]);
            S[i + 2] = fmaf(kv.z, u, sc.x * S[i + 2]);
            S[i + 3] = fmaf(kv.w, u, sc.x * S[i + 3]);
          }
        }
      }
    }
    __syncthreads();                          // the buffer is free for the chunk after the next
  }
  if (MODE == MS_PIECE_OUT) return;
#pragma unroll
  for (int i = 0; i < DPT; i++) {
    const int n = ks * DPT + i;
    if (live && n < N) S_g[(size_t)n * ss] = S[i];
  }
  if (MODE == MS_PIECE_LOCAL && p0 == 0 && tid == 0) A.piece_decay[piece * H + h] = decays;
}

// The pieces' starting states, one after another: an element of (request, head) walks its pieces, leaves in each the state
// the piece starts from and carries (decay product) * state + the piece's own contribution on; the last goes to the slot.
__global__ void __launch_bounds__(256) ms_carry_kernel(StateArgs A) {
  hb_pdl_launch();
  hb_pdl_wait();
  const int r = blockIdx.y, NP = A.N * A.P, per = NP + (A.nstate ? A.N : 0);
  const size_t e = (size_t)blockIdx.x * 256 + threadIdx.x;
  if (e >= (size_t)A.H * per) return;
  const int h = (int)(e / per), i = (int)(e - (size_t)h * per), len = A.q_len[r];
  if (len <= 0) return;
  const bool isn = i >= NP;
  const size_t base = (size_t)ms_piece_base(A.q_len, r, A.L);
  const size_t step = (size_t)A.H * (isn ? A.N : NP);
  float* slot = isn ? A.nstate + ((size_t)A.slot[r] * A.H + h) * A.N + (i - NP) : A.state + ((size_t)A.slot[r] * A.H + h) * NP + i;
  float* ps = isn ? A.piece_n + (base * A.H + h) * A.N + (i - NP) : A.piece_state + (base * A.H + h) * NP + i;
  const float* pd = A.piece_decay + base * A.H + h;
  const int pieces = (len + A.L - 1) / A.L;
  float carry = *slot;
  for (int c0 = 0; c0 < pieces; c0 += 8) {                 // eight pieces' loads in flight, then their chain
    float own[8], dec[8];
#pragma unroll
    for (int k = 0; k < 8; k++) {
      const bool in = c0 + k < pieces;
      own[k] = in ? ps[(size_t)(c0 + k) * step] : 0.f;
      dec[k] = in ? pd[(size_t)(c0 + k) * A.H] : 1.f;
    }
#pragma unroll
    for (int k = 0; k < 8; k++) {
      if (c0 + k < pieces) {
        ps[(size_t)(c0 + k) * step] = carry;
        carry = fmaf(dec[k], carry, own[k]);
      }
    }
  }
  *slot = carry;
}

// threads a value column and key channels a thread for N key channels; 0: not a size the walk takes
static int ms_layout(int N, int* ks_out) {
  for (int ks = 4; ks <= 32; ks *= 2) {
    const int per = (N + ks - 1) / ks;
    if (per <= 32 || (ks == 32 && per <= 64)) {
      *ks_out = ks;
      return per <= 8 ? 8 : per <= 16 ? 16 : per <= 32 ? 32 : 64;
    }
  }
  return 0;
}

HB_EXPORT int hb_ms_walk(const float* q, long ldq, const float* k, long ldk, const float* v, long ldv, const float* a, const float* b,
                         const float* kq, float* state, float* nstate, const int* q_start, const int* q_len, const int* slot, float* y,
                         float* nq, int n_requests, int H, int G, int N, int P, float q_scale, int delta, int piece_len, int pieces,
                         float* piece_state, float* piece_n, float* piece_decay, cudaStream_t s) {
  if (n_requests <= 0) return 0;
  if (G <= 0 || H % G) HB_FAIL("hb_ms_walk: %d heads over %d groups", H, G);
  if (n_requests > 65535 || pieces > 65535) HB_FAIL("hb_ms_walk: the grid is too large");
  if (delta && (!kq || nstate || pieces > 0)) HB_FAIL("hb_ms_walk: the delta form takes k . q, no normaliser and no pieces");
  if (pieces > 0 && (piece_len <= 0 || !piece_state || !piece_decay || (nstate && !piece_n))) HB_FAIL("hb_ms_walk: %d pieces of %d", pieces, piece_len);
  if (nstate && !nq) HB_FAIL("hb_ms_walk: a normaliser needs a place for n . q");
  StateArgs A;
  int ks = 0;
  const int dpt = ms_layout(N, &ks);
  if (!dpt) HB_FAIL("hb_ms_walk: %d key channels do not fit a block's registers", N);
  A.q = q; A.k = k; A.v = v; A.ldq = ldq; A.ldk = ldk; A.ldv = ldv; A.a = a; A.b = b; A.kq = kq; A.state = state; A.nstate = nstate;
  A.q_start = q_start; A.q_len = q_len; A.slot = slot; A.y = y; A.nq = nq; A.H = H; A.G = G; A.N = N; A.P = P; A.KS = ks;
  A.PT = MS_PT_THREADS / ks; A.q_scale = q_scale; A.piece_state = piece_state; A.piece_n = piece_n; A.piece_decay = piece_decay;
  A.L = piece_len; A.pieces = pieces;
  A.vec4 = !((N | P) & 3) && !((ldq | ldk | ldv) & 3) && !(((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) & 15);
  const int RW = 2 * ks * (dpt + 4) + A.PT + 4;
  A.CH = 16;
  while (A.CH > 1 && (size_t)2 * A.CH * RW * sizeof(float) > 96 * 1024) A.CH /= 2;
  const size_t smem = (size_t)2 * A.CH * RW * sizeof(float);
  const int threads = MS_PT_THREADS + (nstate ? 32 : 0), tiles = (P + A.PT - 1) / A.PT;
#define MS_LAUNCH(DPT, DELTA, MODE, GRID)                                                                              \
  do {                                                                                                                 \
    auto kern = ms_walk_kernel<DPT, DELTA, MODE>;                                                                      \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);          \
    hb_launch(kern, GRID, dim3(threads), smem, s, A);                                                                  \
  } while (0)
#define MS_PICK(DELTA, MODE, GRID)                                \
  do {                                                            \
    if (dpt == 8) MS_LAUNCH(8, DELTA, MODE, GRID);                \
    else if (dpt == 16) MS_LAUNCH(16, DELTA, MODE, GRID);         \
    else if (dpt == 32) MS_LAUNCH(32, DELTA, MODE, GRID);         \
    else MS_LAUNCH(64, DELTA, MODE, GRID);                        \
  } while (0)
  if (delta) MS_PICK(true, MS_WHOLE, dim3(H * tiles, n_requests));
  else if (pieces <= 0) MS_PICK(false, MS_WHOLE, dim3(H * tiles, n_requests));
  else {
    const dim3 grid(H * tiles, n_requests, pieces);
    MS_PICK(false, MS_PIECE_LOCAL, grid);
    HB_CHECK_LAUNCH("hb_ms_walk");
    const size_t elems = (size_t)H * (N * P + (nstate ? N : 0));
    hb_launch(ms_carry_kernel, dim3((unsigned)((elems + 255) / 256), n_requests), dim3(256), 0, s, A);
    HB_CHECK_LAUNCH("hb_ms_walk");
    MS_PICK(false, MS_PIECE_OUT, grid);
  }
#undef MS_PICK
#undef MS_LAUNCH
  HB_CHECK_LAUNCH("hb_ms_walk");
  return 0;
}

// ---------------------------------------------------------------------------------------------------------------------
// What does not depend on the state.
// ---------------------------------------------------------------------------------------------------------------------
__device__ __forceinline__ float ms_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float ms_cap(float z, float cap) { return cap * tanhf(z / cap); }

// Exponential gates with a running maximum: li = cap tanh((zi + bi) / cap), lf = -softplus(-cap tanh((zf + bf) / cap));
// m_t = max(lf_t + m_(t-1), li_t);  a = exp(lf_t + m_(t-1) - m_t), b = exp(li_t - m_t), e = exp(-m_t). m is a maximum of sums,
// so a run of tokens acts on it as m -> max(m + F, M): a scan over the tokens, a warp's 32 by shuffles, then the warps' pairs.
// a and b are made from the m values themselves, so that however m was rounded, they fit together. grid (heads, requests).
template <typename TW>
__global__ void __launch_bounds__(1024) ms_exp_gates_kernel(const float* __restrict__ zi, const float* __restrict__ zf, long ldz,
                                                            const TW* __restrict__ bi, const TW* __restrict__ bf, float cap,
                                                            float* __restrict__ m_state, const int* __restrict__ q_start,
                                                            const int* __restrict__ q_len, const int* __restrict__ slot,
                                                            float* __restrict__ a, float* __restrict__ b, float* __restrict__ e, int H) {
  __shared__ float wF[32], wM[32], ms[1025];
  hb_pdl_launch();
  hb_pdl_wait();
  const int h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nthr = blockDim.x, nw = nthr >> 5;
  const int t0 = q_start[r], len = q_len[r];
  float* mp = m_state + (size_t)slot[r] * H + h;
  float m0 = *mp;
  const float vbi = hb_to_float(bi[h]), vbf = hb_to_float(bf[h]);
  for (int c0 = 0; c0 < len; c0 += nthr) {
    const int n = min(nthr, len - c0);
    const size_t t = (size_t)(t0 + c0 + tid);
    float li = -INFINITY, lf = 0.f;
    if (tid < n) {
      li = ms_cap(zi[t * ldz + h] + vbi, cap);
      lf = -ms_softplus(-ms_cap(zf[t * ldz + h] + vbf, cap));
    }
    float F = lf, M = li;
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float pF = __shfl_up_sync(0xffffffffu, F, d), pM = __shfl_up_sync(0xffffffffu, M, d);
      if (lane >= d) {
        M = fmaxf(pM + F, M);
        F += pF;
      }
    }
    if (lane == 31) { wF[warp] = F; wM[warp] = M; }
    __syncthreads();
    float mw = m0;                          // m before this warp's tokens
    for (int w = 0; w < warp; w++) mw = fmaxf(mw + wF[w], wM[w]);
    const float m = fmaxf(mw + F, M);
    ms[tid + 1] = m;
    if (tid == 0) ms[0] = m0;
    __syncthreads();
    if (tid < n) {
      a[t * H + h] = expf(lf + ms[tid] - m);
      b[t * H + h] = expf(li - m);
      e[t * H + h] = expf(-m);
    }
    m0 = ms[n];
    __syncthreads();
  }
  (void)nw;
  if (tid == 0 && len > 0) *mp = m0;
}

HB_EXPORT int hb_ms_exp_gates(const float* zi, const float* zf, long ldz, const void* bi, const void* bf, int w_dt, float cap,
                              float* m_state, const int* q_start, const int* q_len, const int* slot, float* a, float* b, float* e,
                              int n_requests, int max_q_len, int H, cudaStream_t s) {
  if (n_requests <= 0 || max_q_len <= 0) return 0;
  if (n_requests > 65535) HB_FAIL("hb_ms_exp_gates: the grid is too large");
  if (!(cap > 0.f)) HB_FAIL("hb_ms_exp_gates: a cap of %f", (double)cap);
  const int threads = max_q_len >= 1024 ? 1024 : (max_q_len + 31) / 32 * 32;
  HB_DISPATCH_1(w_dt, "hb_ms_exp_gates",
                (hb_launch(ms_exp_gates_kernel<TA>, dim3(H, n_requests), dim3(threads), 0, s, zi, zf, ldz, (const TA*)bi, (const TA*)bf,
                           cap, m_state, q_start, q_len, slot, a, b, e, H)));
  HB_CHECK_LAUNCH("hb_ms_exp_gates");
  return 0;
}

// Row t of qkv holds q [G][N], k [G][N] at q_off and k_off: each head's q and k become x / sqrt(sum x^2 + unit_eps), q also times
// q_scale, in place; kq[t][g] = k . q of the results; a = exp(-exp(A_log) softplus(za + dt_bias)), b = sigmoid(zb). A block a row.
template <typename TW>
__global__ void __launch_bounds__(128) ms_delta_prepare_kernel(float* __restrict__ qkv, long ld, int q_off, int k_off,
                                                               const float* __restrict__ za, const float* __restrict__ zb, long ldz,
                                                               const TW* __restrict__ a_log, const TW* __restrict__ dt_bias,
                                                               float* __restrict__ kq, float* __restrict__ a, float* __restrict__ b,
                                                               int H, int G, int N, float q_scale, float unit_eps) {
  hb_pdl_launch();
  hb_pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* row = qkv + (size_t)t * ld;
  for (int g = warp; g < G; g += 4) {
    float* q = row + q_off + (size_t)g * N;
    float* k = row + k_off + (size_t)g * N;
    float sq = 0.f, sk = 0.f, d = 0.f;
    for (int i = lane; i < N; i += 32) {
      const float qv = q[i], kv = k[i];
      sq = fmaf(qv, qv, sq);
      sk = fmaf(kv, kv, sk);
      d = fmaf(qv, kv, d);
    }
    const float fq = q_scale / sqrtf(hb_warp_sum(sq) + unit_eps), fk = 1.f / sqrtf(hb_warp_sum(sk) + unit_eps);
    d = hb_warp_sum(d);
    for (int i = lane; i < N; i += 32) {
      q[i] *= fq;
      k[i] *= fk;
    }
    if (lane == 0) kq[(size_t)t * G + g] = d * fq * fk;
  }
  for (int h = threadIdx.x; h < H; h += 128) {
    const float sp = ms_softplus(za[(size_t)t * ldz + h] + hb_to_float(dt_bias[h]));
    a[(size_t)t * H + h] = expf(-expf(hb_to_float(a_log[h])) * sp);
    b[(size_t)t * H + h] = 1.f / (1.f + expf(-zb[(size_t)t * ldz + h]));
  }
}

HB_EXPORT int hb_ms_delta_prepare(float* qkv, long ld, int q_off, int k_off, const float* za, const float* zb, long ldz,
                                  const void* a_log, const void* dt_bias, int w_dt, float* kq, float* a, float* b, int T, int H, int G,
                                  int N, float q_scale, float unit_eps, cudaStream_t s) {
  if (T <= 0) return 0;
  HB_DISPATCH_1(w_dt, "hb_ms_delta_prepare",
                (hb_launch(ms_delta_prepare_kernel<TA>, dim3(T), dim3(128), 0, s, qkv, ld, q_off, k_off, za, zb, ldz, (const TA*)a_log,
                           (const TA*)dt_bias, kq, a, b, H, G, N, q_scale, unit_eps)));
  HB_CHECK_LAUNCH("hb_ms_delta_prepare");
  return 0;
}

// ---------------------------------------------------------------------------------------------------------------------
// After the read-out: o / (max(|nq|, e) + den_eps) where there is a normaliser, / root mean square over the head's P values
// (eps inside the root), times a weight (shared by the heads, or one per channel), times the gate (silu or sigmoid). A warp
// a (token, head).
// ---------------------------------------------------------------------------------------------------------------------
template <typename TW, typename TO>
__global__ void __launch_bounds__(256) ms_finish_kernel(const float* __restrict__ y, const float* __restrict__ nq,
                                                        const float* __restrict__ e, float den_eps, const TW* __restrict__ w,
                                                        int w_shared, const float* __restrict__ gate, long ldg, int gate_silu,
                                                        TO* __restrict__ out, long ldo, long pairs, int H, int P, float eps) {
  hb_pdl_launch();
  hb_pdl_wait();
  const int lane = threadIdx.x & 31;
  const long pair = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (pair >= pairs) return;
  const long t = pair / H;
  const int h = (int)(pair - t * H);
  const float* yr = y + pair * P;
  float inv = 1.f;
  if (nq) inv = 1.f / (fmaxf(fabsf(nq[pair]), e[pair]) + den_eps);
  float ss = 0.f;
  for (int i = lane; i < P; i += 32) {
    const float v = yr[i] * inv;
    ss = fmaf(v, v, ss);
  }
  const float f = inv * rsqrtf(hb_warp_sum(ss) / (float)P + eps);
  const TW* wr = w + (w_shared ? 0 : (size_t)h * P);
  const float* gr = gate + t * ldg + (size_t)h * P;
  TO* orow = out + t * ldo + (size_t)h * P;
  for (int i = lane; i < P; i += 32) {
    const float z = gr[i], sg = 1.f / (1.f + expf(-z));
    orow[i] = hb_from_float<TO>(yr[i] * f * hb_to_float(wr[i]) * (gate_silu ? z * sg : sg));
  }
}

HB_EXPORT int hb_ms_finish(const float* y, const float* nq, const float* e, float den_eps, const void* w, int w_dt, int w_shared,
                           const float* gate, long ldg, int gate_silu, void* out, int o_dt, long ldo, int T, int H, int P, float eps,
                           cudaStream_t s) {
  if (T <= 0) return 0;
  if ((nq != nullptr) != (e != nullptr)) HB_FAIL("hb_ms_finish: a normaliser needs n . q and its floor");
  const long pairs = (long)T * H;
  HB_DISPATCH_2(w_dt, o_dt, "hb_ms_finish",
                (hb_launch(ms_finish_kernel<TA, TB>, dim3((unsigned)((pairs + 7) / 8)), dim3(256), 0, s, y, nq, e, den_eps, (const TA*)w,
                           w_shared, gate, ldg, gate_silu, (TB*)out, ldo, pairs, H, P, eps)));
  HB_CHECK_LAUNCH("hb_ms_finish");
  return 0;
}
