// Recurrences with one state matrix per head, S [N][P] (key channel by value channel), carried from token to token in 32-bit:
//
//   linear   S <- a S + b k v^T;  n <- a n + b k;  o = S^T q,  nq = n . q         (a, b: a number per token and head)
//   delta    S <- a S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q
//
// The linear form with a normaliser n is the matrix memory of an exponentially gated LSTM; the delta form the gated delta
// rule. What does not depend on the state is made for all tokens at once by kernels of its own, what follows the read-out
// likewise, so that the serial part is the walk alone:
//   ms_exp_gates_kernel     log gates -> a, b and exp(-m) with the running maximum m (a max-plus scan over the tokens)
//   ms_delta_prepare_kernel the factors that make q, k unit, products of neighbouring tokens' keys and queries, a and b
//   ms_walk_kernel          the walk of the linear form; ms_delta_walk_kernel that of the delta rule
//   ms_finish_kernel        the normaliser, the head's root mean square, a weight and an output gate; rounded once
//   ms_single_kernel        all of it for requests that bring one token each (decoding)
// The value columns of S are independent of one another, so a head's columns are split over blocks. Long portions of the
// linear form run in pieces of L tokens over the whole GPU: every piece from a zero state (its own contribution and the
// product of its decays), then the pieces' starting states one after another (ms_carry_kernel), then every piece again
// from its starting state for o. Requests, lengths and state slots come from device arrays, so a decode step can be
// replayed from a CUDA graph; where a portion or a piece starts changes a token's result by rounding only.
#include "common.cuh"

constexpr int MS_PT_THREADS = 128;      // threads of the value columns of a block

struct StateArgs {
  const float* q; const float* k; const float* v; long ldq, ldk, ldv;     // rows; head h reads q, k of group h / (H / G)
  const float* a; const float* b;         // [T][H]
  float* state; float* nstate;            // [slots][H][N][P], [slots][H][N] or null
  const int* q_start; const int* q_len; const int* slot;
  float* y;                               // [T][H P]
  float* nq;                              // [T][H] (with nstate)
  int H, G, N, P, vec4;
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

// Both walks: grid (heads x column tiles, requests[, pieces]). KS neighbouring lanes share two value columns; lane ks holds DPT
// key channels of them, four of every 4 KS (n = 4 KS (i / 4) + 4 ks + i % 4), so that the lanes read a row of k or q as it lies.
// Four warps walk; in the linear form a fifth keeps the normaliser. Rows come a chunk of CH tokens ahead by cp.async, every
// thread a few fixed pieces of them; one barrier a chunk. A token's row in shared memory is [k | q | v of the tile | its
// numbers], k and q filled up with zeros to KS DPT: no bounds are checked in the walk. Tokens go by four at a time; the last
// group of a portion is filled up with tokens that change nothing.
constexpr int MS_WARPS = MS_PT_THREADS / 32, MS_COLS = 2, MS_SCAL = 12;

template <int DPT, int KS, int SC> struct MsRow {
  static constexpr int PT = MS_PT_THREADS / KS * MS_COLS, KQ = KS * DPT, RW = 2 * KQ + PT + SC;
  static constexpr int CH = RW <= 384 ? 16 : RW <= 768 ? 8 : 4;
  static constexpr int NC = KQ / 4 < MS_PT_THREADS ? KQ / 4 : MS_PT_THREADS;      // pieces of a row of k a pass of the threads takes
  static constexpr size_t SMEM = (size_t)2 * CH * RW * sizeof(float);
};

// Four floats from columns [c, c + 4) of a row, those below `end`.
__device__ __forceinline__ void ms_piece(float* dst, const float* src, int c, int end, int vec4) {
  if (vec4) {
    if (c < end) ms_cp16(dst + c, src + c);
  } else {
#pragma unroll
    for (int e = 0; e < 4; e++)
      if (c + e < end) ms_cp4(dst + c + e, src + c + e);
  }
}

// The rows of a chunk's n tokens (kh, qh, vh: the first token's) into a chunk buffer, by the threads below MS_PT_THREADS.
template <int DPT, int KS, int SC, bool WITH_Q>
__device__ __forceinline__ void ms_fetch(float* chunk, const float* kh, long ldk, const float* qh, long ldq, const float* vh, long ldv, int N,
                                         int np, int vec4, int n, int tid) {
  using R = MsRow<DPT, KS, SC>;
  constexpr int TP = MS_PT_THREADS / R::NC, TV = MS_PT_THREADS / (R::PT / 4);
  static_assert(R::PT % 4 == 0 && MS_PT_THREADS % R::NC == 0, "whole passes");
#pragma unroll
  for (int i = 0; i < (R::CH + TP - 1) / TP; i++) {
    const int j = tid / R::NC + i * TP;
    if (j < n) {
      float* row = chunk + j * R::RW;
#pragma unroll
      for (int cc = 0; cc < R::KQ / 4; cc += R::NC) {
        const int c = (tid % R::NC + cc) * 4;
        ms_piece(row, kh + j * ldk, c, N, vec4);
        if (WITH_Q) ms_piece(row + R::KQ, qh + j * ldq, c, N, vec4);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < (R::CH + TV - 1) / TV; i++) {
    const int j = tid / (R::PT / 4) + i * TV;
    if (j < n) ms_piece(chunk + j * R::RW + 2 * R::KQ, vh + j * ldv, tid % (R::PT / 4) * 4, np, vec4);
  }
}

// Sums of eight values over KS neighbouring lanes, scattered: lane ks ends with the sum of value ks % 8.
template <int KS>
__device__ __forceinline__ float ms_reduce8(const float (&v)[8], int ks) {
  float w4[4], w2[2];
  const bool b2 = ks & 4, b1 = ks & 2, b0 = ks & 1;
#pragma unroll
  for (int j = 0; j < 4; j++) w4[j] = (b2 ? v[j + 4] : v[j]) + __shfl_xor_sync(0xffffffffu, b2 ? v[j] : v[j + 4], 4);
#pragma unroll
  for (int j = 0; j < 2; j++) w2[j] = (b1 ? w4[j + 2] : w4[j]) + __shfl_xor_sync(0xffffffffu, b1 ? w4[j] : w4[j + 2], 2);
  float r = (b0 ? w2[1] : w2[0]) + __shfl_xor_sync(0xffffffffu, b0 ? w2[0] : w2[1], 1);
#pragma unroll
  for (int m = 8; m < KS; m <<= 1) r += __shfl_xor_sync(0xffffffffu, r, m);
  return r;
}

template <int DPT, int KS, int MODE>
__global__ void __launch_bounds__(MS_PT_THREADS + 32) ms_walk_kernel(StateArgs A) {
  extern __shared__ __align__(16) float msm[];
  hb_pdl_launch();
  hb_pdl_wait();
  using R = MsRow<DPT, KS, 4>;             // numbers of a token: a, b, -, -
  constexpr int PT = R::PT, KQ = R::KQ, RW = R::RW, CH = R::CH;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int H = A.H, N = A.N, P = A.P;
  const int tiles = (P + PT - 1) / PT, h = blockIdx.x / tiles, p0 = (blockIdx.x - h * tiles) * PT;
  const int g = h / (H / A.G), r = blockIdx.y;
  const bool norm_warp = warp == MS_WARPS, walks = !norm_warp || p0 == 0;
  const int pl = norm_warp ? 0 : tid / KS * MS_COLS, ks = lane % KS;
  const int t0 = A.q_start[r];
  const int j_begin = MODE == MS_WHOLE ? 0 : (int)blockIdx.z * A.L;
  const int len = MODE == MS_WHOLE ? A.q_len[r] : min(A.q_len[r], j_begin + A.L);
  if (j_begin >= len) return;
  const size_t piece = MODE == MS_WHOLE ? 0 : (size_t)ms_piece_base(A.q_len, r, A.L) + blockIdx.z;
  // the normaliser is one column of value 1; its warp's lanes beyond KS repeat it and store nothing
  float* S_g = norm_warp ? (MODE == MS_WHOLE ? A.nstate + ((size_t)A.slot[r] * H + h) * N : A.piece_n + (piece * H + h) * N)
                         : (MODE == MS_WHOLE ? A.state + ((size_t)A.slot[r] * H + h) * N * P : A.piece_state + (piece * H + h) * N * P) + p0 + pl;
  const int ss = norm_warp ? 1 : P;
  bool live[MS_COLS];
#pragma unroll
  for (int c = 0; c < MS_COLS; c++) live[c] = norm_warp ? c == 0 && p0 == 0 && lane < KS : p0 + pl + c < P;
  float S[MS_COLS][DPT];
#pragma unroll
  for (int c = 0; c < MS_COLS; c++)
#pragma unroll
    for (int i = 0; i < DPT; i++) {
      const int n = i / 4 * (4 * KS) + 4 * ks + i % 4;
      S[c][i] = MODE != MS_PIECE_LOCAL && live[c] && n < N ? S_g[(size_t)n * ss + c] : 0.f;
    }
  for (int i = tid; i < 2 * CH * RW; i += blockDim.x) msm[i] = 0.f;      // padding, and rows past a portion's end, are read
  __syncthreads();
  auto fetch = [&](int buf, int c0) {
    const int n = min(CH, len - c0);
    const size_t t = (size_t)(t0 + c0);
    float* chunk = msm + buf * CH * RW;
    if (!norm_warp) {
      ms_fetch<DPT, KS, 4, MODE != MS_PIECE_LOCAL>(chunk, A.k + t * A.ldk + (size_t)g * N, A.ldk, A.q + t * A.ldq + (size_t)g * N, A.ldq,
                                                   A.v + t * A.ldv + (size_t)h * P + p0, A.ldv, N, min(PT, P - p0), A.vec4, n, tid);
      const int j = tid >> 1;                // a and b of a token: two threads
      if (j < n) ms_cp4(chunk + j * RW + 2 * KQ + PT + (tid & 1), (tid & 1 ? A.b : A.a) + (t + j) * H + h);
      else if (j < ((n + 3) & ~3)) chunk[j * RW + 2 * KQ + PT + (tid & 1)] = tid & 1 ? 0.f : 1.f;      // a token that changes nothing
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, j_begin);
  float decays = 1.f;
  int buf = 0;
  const int sb = 4 * ks;
  // lane ks ends with the result of token ks / 2 of a group and column ks % 2
  const int my_i = (ks & 7) >> 1, my_c = ks & 1;
  const bool stores = ks < 8 && (my_c ? live[1] : live[0]);
  const size_t ystep = norm_warp ? (size_t)H : (size_t)H * P;
  float* yg = (norm_warp ? A.nq + (size_t)t0 * H + h : A.y + (size_t)t0 * H * P + (size_t)h * P + p0 + pl + my_c) + (size_t)(j_begin + my_i) * ystep;
  for (int c0 = j_begin; c0 < len; c0 += CH, buf ^= 1) {
    const int n = min(CH, len - c0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                         // this chunk is in, and every warp is done with the one before it
    if (c0 + CH < len) fetch(buf ^ 1, c0 + CH);
    if (walks) {
      const float* row = msm + buf * CH * RW;
      for (int j0 = 0; j0 < n; j0 += 4, row += 4 * RW, yg += 4 * ystep) {
        float o[8];
#pragma unroll
        for (int i = 0; i < 4; i++) {
          const float2 ab = *(const float2*)(row + i * RW + 2 * KQ + PT);
          const float2 vv = norm_warp ? make_float2(1.f, 0.f) : *(const float2*)(row + i * RW + 2 * KQ + pl);
          const float x[MS_COLS] = {ab.y * vv.x, ab.y * vv.y};
          if (MODE == MS_PIECE_LOCAL) decays *= ab.x;
#pragma unroll
          for (int c = 0; c < MS_COLS; c++) o[2 * i + c] = 0.f;
#pragma unroll
          for (int d = 0; d < DPT; d += 4) {
            const float4 kv = *(const float4*)(row + i * RW + sb + d * KS);
            float4 qv;
            if (MODE != MS_PIECE_LOCAL) qv = *(const float4*)(row + i * RW + KQ + sb + d * KS);
#pragma unroll
            for (int c = 0; c < MS_COLS; c++) {
              S[c][d] = fmaf(ab.x, S[c][d], kv.x * x[c]);
              S[c][d + 1] = fmaf(ab.x, S[c][d + 1], kv.y * x[c]);
              S[c][d + 2] = fmaf(ab.x, S[c][d + 2], kv.z * x[c]);
              S[c][d + 3] = fmaf(ab.x, S[c][d + 3], kv.w * x[c]);
              if (MODE != MS_PIECE_LOCAL) {
                o[2 * i + c] = fmaf(S[c][d], qv.x, o[2 * i + c]);
                o[2 * i + c] = fmaf(S[c][d + 1], qv.y, o[2 * i + c]);
                o[2 * i + c] = fmaf(S[c][d + 2], qv.z, o[2 * i + c]);
                o[2 * i + c] = fmaf(S[c][d + 3], qv.w, o[2 * i + c]);
              }
            }
          }
        }
        if (MODE != MS_PIECE_LOCAL) {
          const float mine = ms_reduce8<KS>(o, ks);
          if (stores && j0 + my_i < n) *yg = mine * A.q_scale;
        }
      }
    }
  }
  if (MODE == MS_PIECE_OUT) return;
  asm volatile("" : "+l"(S_g));               // the addresses are made again here instead of being kept through the walk
#pragma unroll
  for (int c = 0; c < MS_COLS; c++)
#pragma unroll
    for (int i = 0; i < DPT; i++) {
      const int n = i / 4 * (4 * KS) + 4 * ks + i % 4;
      if (live[c] && n < N) S_g[(size_t)n * ss + c] = S[c][i];
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

#define MS_SIZES(X, ...)                        \
  do {                                          \
    if (N <= 32) X(4, 8, __VA_ARGS__);          \
    else if (N <= 64) X(8, 8, __VA_ARGS__);     \
    else if (N <= 128) X(16, 8, __VA_ARGS__);   \
    else if (N <= 256) X(16, 16, __VA_ARGS__);  \
    else if (N <= 512) X(16, 32, __VA_ARGS__);  \
    else X(32, 32, __VA_ARGS__);                \
  } while (0)

HB_EXPORT int hb_ms_walk(const float* q, long ldq, const float* k, long ldk, const float* v, long ldv, const float* a, const float* b,
                         float* state, float* nstate, const int* q_start, const int* q_len, const int* slot, float* y,
                         float* nq, int n_requests, int H, int G, int N, int P, float q_scale, int piece_len, int pieces,
                         float* piece_state, float* piece_n, float* piece_decay, cudaStream_t s) {
  if (n_requests <= 0) return 0;
  if (G <= 0 || H % G) HB_FAIL("hb_ms_walk: %d heads over %d groups", H, G);
  if (n_requests > 65535 || pieces > 65535) HB_FAIL("hb_ms_walk: the grid is too large");
  if (pieces > 0 && (piece_len <= 0 || !piece_state || !piece_decay || (nstate && !piece_n))) HB_FAIL("hb_ms_walk: %d pieces of %d", pieces, piece_len);
  if (nstate && !nq) HB_FAIL("hb_ms_walk: a normaliser needs a place for n . q");
  if (N > 1024) HB_FAIL("hb_ms_walk: %d key channels do not fit a block's registers", N);
  StateArgs A;
  A.q = q; A.k = k; A.v = v; A.ldq = ldq; A.ldk = ldk; A.ldv = ldv; A.a = a; A.b = b; A.state = state; A.nstate = nstate;
  A.q_start = q_start; A.q_len = q_len; A.slot = slot; A.y = y; A.nq = nq; A.H = H; A.G = G; A.N = N; A.P = P; A.q_scale = q_scale;
  A.piece_state = piece_state; A.piece_n = piece_n; A.piece_decay = piece_decay; A.L = piece_len; A.pieces = pieces;
  A.vec4 = !((N | P) & 3) && !((ldq | ldk | ldv) & 3) && !(((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) & 15);
  const int threads = MS_PT_THREADS + (nstate ? 32 : 0);
#define MS_LAUNCH(DPT, KS, MODE, GRID_Z)                                                                                \
  do {                                                                                                                  \
    using R = MsRow<DPT, KS, 4>;                                                                                        \
    const size_t smem = R::SMEM;                                                                                        \
    auto kern = ms_walk_kernel<DPT, KS, MODE>;                                                                          \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);           \
    hb_launch(kern, dim3(H * ((P + R::PT - 1) / R::PT), n_requests, GRID_Z), dim3(threads), smem, s, A);                \
  } while (0)
  if (pieces <= 0) MS_SIZES(MS_LAUNCH, MS_WHOLE, 1);
  else {
    MS_SIZES(MS_LAUNCH, MS_PIECE_LOCAL, pieces);
    HB_CHECK_LAUNCH("hb_ms_walk");
    const size_t elems = (size_t)H * (N * P + (nstate ? N : 0));
    hb_launch(ms_carry_kernel, dim3((unsigned)((elems + 255) / 256), n_requests), dim3(256), 0, s, A);
    HB_CHECK_LAUNCH("hb_ms_walk");
    MS_SIZES(MS_LAUNCH, MS_PIECE_OUT, pieces);
  }
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
  const int h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nthr = blockDim.x;
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

// What the delta rule's walk reads of a token beside its rows, MS_SCAL numbers per (token, head), with k^ and q^ the unit key and
// query (x / sqrt(sum x^2 + unit_eps), q^ also times q_scale), t - i the tokens before it in the same portion:
//   a = exp(-exp(A_log) softplus(za + dt_bias)), b = sigmoid(zb), the factors fk, fq that make k, q unit,
//   k^_t . k^_(t-1), .. (t-2), .. (t-3), q^_t . k^_t, q^_t . k^_(t-1), .. (t-2), .. (t-3), 0        (0 before the portion's start)
// A block a row, a warp a group.

template <typename TW>
__global__ void __launch_bounds__(256) ms_delta_prepare_kernel(const float* __restrict__ q_rows, const float* __restrict__ k_rows, long ld,
                                                               const float* __restrict__ za, const float* __restrict__ zb, long ldz,
                                                               const TW* __restrict__ a_log, const TW* __restrict__ dt_bias,
                                                               const int* __restrict__ row_req, const int* __restrict__ q_start,
                                                               float* __restrict__ scal, int H, int G, int N, float q_scale,
                                                               float unit_eps) {
  hb_pdl_launch();
  hb_pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5, HG = H / G;
  const int back = min(3, t - q_start[row_req[t]]);          // tokens before this one in its portion, up to three
  for (int g = warp; g < G; g += nw) {
    const float* q = q_rows + (size_t)t * ld + (size_t)g * N;
    const float* k = k_rows + (size_t)t * ld + (size_t)g * N;
    float qq = 0.f, kk[4] = {0.f, 0.f, 0.f, 0.f}, own[4] = {0.f, 0.f, 0.f, 0.f}, qk[4] = {0.f, 0.f, 0.f, 0.f};
    for (int i = lane; i < N; i += 32) {
      const float qv = q[i], kv = k[i];
      qq = fmaf(qv, qv, qq);
#pragma unroll
      for (int d = 0; d < 4; d++) {
        const float kd = d == 0 ? kv : d <= back ? k[i - (long)d * ld] : 0.f;
        own[d] = fmaf(kd, kd, own[d]);
        kk[d] = fmaf(kv, kd, kk[d]);
        qk[d] = fmaf(qv, kd, qk[d]);
      }
    }
    const float fq = q_scale / sqrtf(hb_warp_sum(qq) + unit_eps);
    float fk[4];
#pragma unroll
    for (int d = 0; d < 4; d++) {
      fk[d] = 1.f / sqrtf(hb_warp_sum(own[d]) + unit_eps);
      kk[d] = hb_warp_sum(kk[d]);
      qk[d] = hb_warp_sum(qk[d]);
    }
    for (int h = g * HG + lane; h < (g + 1) * HG; h += 32) {
      const float sp = ms_softplus(za[(size_t)t * ldz + h] + hb_to_float(dt_bias[h]));
      float4* o = (float4*)(scal + ((size_t)t * H + h) * MS_SCAL);
      o[0] = make_float4(expf(-expf(hb_to_float(a_log[h])) * sp), 1.f / (1.f + expf(-zb[(size_t)t * ldz + h])), fk[0], fq);
      o[1] = make_float4(kk[1] * fk[0] * fk[1], kk[2] * fk[0] * fk[2], kk[3] * fk[0] * fk[3], qk[0] * fq * fk[0]);
      o[2] = make_float4(qk[1] * fq * fk[1], qk[2] * fq * fk[2], qk[3] * fq * fk[3], 0.f);
    }
  }
}

HB_EXPORT int hb_ms_delta_prepare(const float* q, const float* k, long ld, const float* za, const float* zb, long ldz, const void* a_log,
                                  const void* dt_bias, int w_dt, const int* row_req, const int* q_start, float* scal, int T, int H, int G,
                                  int N, float q_scale, float unit_eps, cudaStream_t s) {
  if (T <= 0) return 0;
  if (G <= 0 || H % G) HB_FAIL("hb_ms_delta_prepare: %d heads over %d groups", H, G);
  const int threads = 32 * (G < 8 ? G : 8);
  HB_DISPATCH_1(w_dt, "hb_ms_delta_prepare",
                (hb_launch(ms_delta_prepare_kernel<TA>, dim3(T), dim3(threads), 0, s, q, k, ld, za, zb, ldz, (const TA*)a_log,
                           (const TA*)dt_bias, row_req, q_start, scal, H, G, N, q_scale, unit_eps)));
  HB_CHECK_LAUNCH("hb_ms_delta_prepare");
  return 0;
}

// ---------------------------------------------------------------------------------------------------------------------
// The delta rule's walk, four tokens at a time. With S the state before them, decays a_i and their running products g_i,
//     u_i = b_i (v_i - g_i S^T k^_i - sum over j < i of (a_(j+1) .. a_i) (k^_i . k^_j) u_j)
//     o_i = g_i S^T q^_i + sum over j <= i of (a_(j+1) .. a_i) (q^_i . k^_j) u_j
//     S  <- g_4 S + sum over j of (a_(j+1) .. a_4) k^_j u_j
// so that all eight products with S are independent of one another and the serial part of four tokens is a handful of
// multiply-adds.
// ---------------------------------------------------------------------------------------------------------------------
struct DeltaArgs {
  const float* q; const float* k; const float* v; long ldq, ldk, ldv;
  const float* scal;                      // [T][H][MS_SCAL]
  float* state;                           // [slots][H][N][P]
  const int* q_start; const int* q_len; const int* slot;
  float* y;                               // [T][H P]
  int H, G, N, P, vec4;
};

template <int DPT, int KS>
__global__ void __launch_bounds__(MS_PT_THREADS) ms_delta_walk_kernel(DeltaArgs A) {
  extern __shared__ __align__(16) float dsm[];
  hb_pdl_launch();
  hb_pdl_wait();
  using R = MsRow<DPT, KS, MS_SCAL>;
  constexpr int PT = R::PT, KQ = R::KQ, RW = R::RW, CH = R::CH;
  const int tid = threadIdx.x, lane = tid & 31;
  const int H = A.H, N = A.N, P = A.P;
  const int tiles = (P + PT - 1) / PT, h = blockIdx.x / tiles, p0 = (blockIdx.x - h * tiles) * PT;
  const int g = h / (H / A.G), r = blockIdx.y;
  const int pl = tid / KS * MS_COLS, ks = lane % KS;
  const int t0 = A.q_start[r], len = A.q_len[r];
  if (len <= 0) return;
  float* S_g = A.state + ((size_t)A.slot[r] * H + h) * N * P + p0 + pl;
  bool live[MS_COLS];
#pragma unroll
  for (int c = 0; c < MS_COLS; c++) live[c] = p0 + pl + c < P;
  float S[MS_COLS][DPT];
#pragma unroll
  for (int c = 0; c < MS_COLS; c++)
#pragma unroll
    for (int i = 0; i < DPT; i++) {
      const int n = i / 4 * (4 * KS) + 4 * ks + i % 4;
      S[c][i] = live[c] && n < N ? S_g[(size_t)n * P + c] : 0.f;
    }
  for (int i = tid; i < 2 * CH * RW; i += blockDim.x) dsm[i] = 0.f;      // padding, and rows past a portion's end, are read
  __syncthreads();
  auto fetch = [&](int buf, int c0) {
    const int n = min(CH, len - c0);
    const size_t t = (size_t)(t0 + c0);
    float* chunk = dsm + buf * CH * RW;
    ms_fetch<DPT, KS, MS_SCAL, true>(chunk, A.k + t * A.ldk + (size_t)g * N, A.ldk, A.q + t * A.ldq + (size_t)g * N, A.ldq,
                                     A.v + t * A.ldv + (size_t)h * P + p0, A.ldv, N, min(PT, P - p0), A.vec4, n, tid);
    const int j = tid >> 2, c = tid & 3;     // a token's numbers: three of four threads
    float* sc = chunk + j * RW + 2 * KQ + PT + 4 * c;
    if (c < MS_SCAL / 4) {
      if (j < n) ms_cp16(sc, A.scal + ((t + j) * H + h) * MS_SCAL + 4 * c);
      else if (j < ((n + 3) & ~3)) *(float4*)sc = make_float4(c == 0 ? 1.f : 0.f, 0.f, 0.f, 0.f);      // a token that changes nothing
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0, 0);
  int buf = 0;
  const int sb = 4 * ks;
  // lane ks ends with the result of token ks / 2 of a group and column ks % 2
  const int my_i = (ks & 7) >> 1, my_c = ks & 1, base = lane & ~7;
  const bool stores = ks < 8 && (my_c ? live[1] : live[0]);
  const size_t HP = (size_t)H * P;
  float* yg = A.y + (size_t)(t0 + my_i) * HP + (size_t)h * P + p0 + pl + my_c;
  for (int c0 = 0; c0 < len; c0 += CH, buf ^= 1) {
    const int n = min(CH, len - c0);
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                         // this chunk is in, and every warp is done with the one before it
    if (c0 + CH < len) fetch(buf ^ 1, c0 + CH);
    const float* row = dsm + buf * CH * RW;
    for (int j0 = 0; j0 < n; j0 += 4, row += 4 * RW, yg += 4 * HP) {
      float x[8], z[8];                      // (token, column)
#pragma unroll
      for (int i = 0; i < 8; i++) x[i] = z[i] = 0.f;
#pragma unroll
      for (int d = 0; d < DPT; d += 4)
#pragma unroll
        for (int i = 0; i < 4; i++) {
          const float4 kv = *(const float4*)(row + i * RW + sb + d * KS), qv = *(const float4*)(row + i * RW + KQ + sb + d * KS);
#pragma unroll
          for (int c = 0; c < MS_COLS; c++) {
            x[2 * i + c] = fmaf(S[c][d], kv.x, x[2 * i + c]); z[2 * i + c] = fmaf(S[c][d], qv.x, z[2 * i + c]);
            x[2 * i + c] = fmaf(S[c][d + 1], kv.y, x[2 * i + c]); z[2 * i + c] = fmaf(S[c][d + 1], qv.y, z[2 * i + c]);
            x[2 * i + c] = fmaf(S[c][d + 2], kv.z, x[2 * i + c]); z[2 * i + c] = fmaf(S[c][d + 2], qv.z, z[2 * i + c]);
            x[2 * i + c] = fmaf(S[c][d + 3], kv.w, x[2 * i + c]); z[2 * i + c] = fmaf(S[c][d + 3], qv.w, z[2 * i + c]);
          }
        }
      const float xm = ms_reduce8<KS>(x, ks), zm = ms_reduce8<KS>(z, ks);
#pragma unroll
      for (int i = 0; i < 8; i++) x[i] = __shfl_sync(0xffffffffu, xm, base + i);
      float a_[4], fk[4], gp = 1.f, u[4][MS_COLS], om = 0.f;
#pragma unroll
      for (int i = 0; i < 4; i++) {
        const float* sp = row + i * RW + 2 * KQ + PT;
        const float4 s0 = *(const float4*)sp, s1 = *(const float4*)(sp + 4), s2 = *(const float4*)(sp + 8);
        const float2 vv = *(const float2*)(row + i * RW + 2 * KQ + pl);
        const float kk[4] = {0.f, s1.x, s1.y, s1.z}, qk[4] = {s1.w, s2.x, s2.y, s2.z};
        a_[i] = s0.x;
        fk[i] = s0.z;
        gp *= s0.x;
        float dec[4];                        // dec[j] = a_(j+1) .. a_i
        dec[i] = 1.f;
#pragma unroll
        for (int j = i - 1; j >= 0; j--) dec[j] = dec[j + 1] * a_[j + 1];
        const float gk = gp * s0.z;
#pragma unroll
        for (int c = 0; c < MS_COLS; c++) {
          float ui = fmaf(-gk, x[2 * i + c], c ? vv.y : vv.x);
#pragma unroll
          for (int j = 0; j < i; j++) ui = fmaf(-kk[i - j] * dec[j], u[j][c], ui);
          u[i][c] = ui * s0.y;
        }
        if (my_i == i) {                     // this lane's own result
          om = gp * s0.w * zm;
#pragma unroll
          for (int j = 0; j <= i; j++) om = fmaf(qk[i - j] * dec[j], my_c ? u[j][1] : u[j][0], om);
        }
      }
      if (stores && j0 + my_i < n) *yg = om;
      float dec = 1.f;
#pragma unroll
      for (int i = 3; i >= 0; i--) {         // what the rows of k are multiplied by
        const float f = dec * fk[i];
        u[i][0] *= f;
        u[i][1] *= f;
        dec *= a_[i];
      }
#pragma unroll
      for (int d = 0; d < DPT; d += 4) {
#pragma unroll
        for (int c = 0; c < MS_COLS; c++) { S[c][d] *= gp; S[c][d + 1] *= gp; S[c][d + 2] *= gp; S[c][d + 3] *= gp; }
#pragma unroll
        for (int i = 0; i < 4; i++) {
          const float4 kv = *(const float4*)(row + i * RW + sb + d * KS);
#pragma unroll
          for (int c = 0; c < MS_COLS; c++) {
            S[c][d] = fmaf(kv.x, u[i][c], S[c][d]);
            S[c][d + 1] = fmaf(kv.y, u[i][c], S[c][d + 1]);
            S[c][d + 2] = fmaf(kv.z, u[i][c], S[c][d + 2]);
            S[c][d + 3] = fmaf(kv.w, u[i][c], S[c][d + 3]);
          }
        }
      }
    }
  }
  asm volatile("" : "+l"(S_g));               // the addresses are made again here instead of being kept through the walk
#pragma unroll
  for (int c = 0; c < MS_COLS; c++)
#pragma unroll
    for (int i = 0; i < DPT; i++) {
      const int n = i / 4 * (4 * KS) + 4 * ks + i % 4;
      if (live[c] && n < N) S_g[(size_t)n * P + c] = S[c][i];
    }
}

HB_EXPORT int hb_ms_delta_walk(const float* q, long ldq, const float* k, long ldk, const float* v, long ldv, const float* scal, float* state,
                               const int* q_start, const int* q_len, const int* slot, float* y, int n_requests, int H, int G, int N, int P,
                               cudaStream_t s) {
  if (n_requests <= 0) return 0;
  if (G <= 0 || H % G || n_requests > 65535) HB_FAIL("hb_ms_delta_walk: %d heads over %d groups, %d requests", H, G, n_requests);
  if (N > 1024) HB_FAIL("hb_ms_delta_walk: %d key channels do not fit a block's registers", N);
  DeltaArgs A;
  A.q = q; A.k = k; A.v = v; A.ldq = ldq; A.ldk = ldk; A.ldv = ldv; A.scal = scal; A.state = state; A.q_start = q_start; A.q_len = q_len;
  A.slot = slot; A.y = y; A.H = H; A.G = G; A.N = N; A.P = P;
  A.vec4 = !((N | P) & 3) && !((ldq | ldk | ldv) & 3) && !(((uintptr_t)q | (uintptr_t)k | (uintptr_t)v) & 15);
  if ((uintptr_t)scal & 15) HB_FAIL("hb_ms_delta_walk: the tokens' numbers must start on a 16-byte boundary");
#define MSD_LAUNCH(DPT, KS, UNUSED)                                                                                     \
  do {                                                                                                                  \
    using R = MsRow<DPT, KS, MS_SCAL>;                                                                                  \
    const size_t smem = R::SMEM;                                                                                        \
    auto kern = ms_delta_walk_kernel<DPT, KS>;                                                                          \
    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);           \
    hb_launch(kern, dim3(H * ((P + R::PT - 1) / R::PT), n_requests), dim3(MS_PT_THREADS), smem, s, A);                  \
  } while (0)
  MS_SIZES(MSD_LAUNCH, 0);
#undef MSD_LAUNCH
  HB_CHECK_LAUNCH("hb_ms_delta_walk");
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

// The same with four values a lane: P / 4 lanes (a power of two up to 32) share a (token, head).
template <typename TW, typename TO>
__global__ void __launch_bounds__(256) ms_finish_vec_kernel(const float* __restrict__ y, const float* __restrict__ nq,
                                                            const float* __restrict__ e, float den_eps, const TW* __restrict__ w,
                                                            int w_shared, const float* __restrict__ gate, long ldg, int gate_silu,
                                                            TO* __restrict__ out, long ldo, long pairs, int H, int P, float eps) {
  hb_pdl_launch();
  hb_pdl_wait();
  const int lanes = P >> 2;
  const long idx = (long)blockIdx.x * 256 + threadIdx.x;
  const long pair = min(idx / lanes, pairs - 1);        // lanes past the end repeat the last pair and store nothing
  const int i = (int)(idx & (lanes - 1)) * 4;
  const long t = pair / H;
  const int h = (int)(pair - t * H);
  float4 v = hb_load4(y + pair * P + i);
  const float4 z = hb_load4(gate + t * ldg + (size_t)h * P + i);
  const float4 wv = hb_load4(w + (w_shared ? 0 : (size_t)h * P) + i);
  float inv = 1.f;
  if (nq) inv = 1.f / (fmaxf(fabsf(nq[pair]), e[pair]) + den_eps);
  v.x *= inv; v.y *= inv; v.z *= inv; v.w *= inv;
  float ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, v.w * v.w)));
  for (int m = 1; m < lanes; m <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
  const float f = rsqrtf(ss / (float)P + eps);
  auto act = [&](float g) { const float sg = 1.f / (1.f + expf(-g)); return gate_silu ? g * sg : sg; };
  if (idx / lanes < pairs)
    hb_store4(out + t * ldo + (size_t)h * P + i, make_float4(v.x * f * wv.x * act(z.x), v.y * f * wv.y * act(z.y),
                                                             v.z * f * wv.z * act(z.z), v.w * f * wv.w * act(z.w)));
}

HB_EXPORT int hb_ms_finish(const float* y, const float* nq, const float* e, float den_eps, const void* w, int w_dt, int w_shared,
                           const float* gate, long ldg, int gate_silu, void* out, int o_dt, long ldo, int T, int H, int P, float eps,
                           cudaStream_t s) {
  if (T <= 0) return 0;
  if ((nq != nullptr) != (e != nullptr)) HB_FAIL("hb_ms_finish: a normaliser needs n . q and its floor");
  const long pairs = (long)T * H;
  const int lanes = P / 4;
  if (P % 4 == 0 && lanes <= 32 && !(lanes & (lanes - 1)) && !((ldg | ldo) & 3) &&
      !(((uintptr_t)y | (uintptr_t)gate | (uintptr_t)w | (uintptr_t)out) & 15)) {
    HB_DISPATCH_2(w_dt, o_dt, "hb_ms_finish",
                  (hb_launch(ms_finish_vec_kernel<TA, TB>, dim3((unsigned)((pairs * lanes + 255) / 256)), dim3(256), 0, s, y, nq, e,
                             den_eps, (const TA*)w, w_shared, gate, ldg, gate_silu, (TB*)out, ldo, pairs, H, P, eps)));
    HB_CHECK_LAUNCH("hb_ms_finish");
    return 0;
  }
  HB_DISPATCH_2(w_dt, o_dt, "hb_ms_finish",
                (hb_launch(ms_finish_kernel<TA, TB>, dim3((unsigned)((pairs + 7) / 8)), dim3(256), 0, s, y, nq, e, den_eps, (const TA*)w,
                           w_shared, gate, ldg, gate_silu, (TB*)out, ldo, pairs, H, P, eps)));
  HB_CHECK_LAUNCH("hb_ms_finish");
  return 0;
}

// ---------------------------------------------------------------------------------------------------------------------
// Requests that bring one token each: gates (or unit keys), the state's update, the read-out, the head norm, weight and gate
// in one kernel. A block owns (head, request): four neighbouring columns a thread, R key channels each (n = ty + i TY), so
// that the state is read and written in whole rows, every load asked for at once. Requests with another number of rows than
// one are left alone (the caller does not send them).
// ---------------------------------------------------------------------------------------------------------------------
constexpr int MS1_THREADS = 256;

struct SingleArgs {
  const float* q; const float* k; const float* v; long ldq, ldk, ldv;
  const float* z1; const float* z2; long ldz;             // linear: li, lf before bias and cap; delta: a, b before theirs
  const void* w1; const void* w2;                         // linear: bi, bf; delta: dt_bias, A_log       [H] each
  float cap, unit_eps, q_scale, den_eps, eps;
  float* state; float* nstate; float* mstate;
  const int* q_start; const int* q_len; const int* slot;
  const void* w; int w_shared;
  const float* gate; long ldg; int gate_silu;
  void* out; long ldo;
  int H, G, N, P;
};

template <int R, bool DELTA, typename TS, typename TW, typename TO>
__global__ void __launch_bounds__(MS1_THREADS) ms_single_kernel(SingleArgs A) {
  extern __shared__ __align__(16) float m1[];             // [N] k, [N] q, [TY][P] partial sums (delta: twice), [P] u or o
  __shared__ float red[32];
  hb_pdl_launch();
  hb_pdl_wait();
  const int h = blockIdx.x, r = blockIdx.y, tid = threadIdx.x;
  if (A.q_len[r] != 1) return;
  const int H = A.H, N = A.N, P = A.P, P4 = P >> 2, TY = MS1_THREADS / P4;
  const int tx = tid % P4, ty = tid / P4;
  const bool act = ty < TY;
  const size_t t = A.q_start[r], sl = A.slot[r];
  float* S_g = A.state + ((sl * H + h) * N) * P + 4 * tx;
  float4 S[R];
#pragma unroll
  for (int i = 0; i < R; i++) {
    const int n = ty + i * TY;
    S[i] = act && n < N ? *(const float4*)(S_g + (size_t)n * P) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float* sk = m1;
  float* sq = sk + N;
  float* part = sq + N;                                   // [TY][P]
  float* part2 = part + (size_t)TY * P;                   // [TY][P] (delta)
  const int g = h / (H / A.G);
  const float* qg = A.q + t * A.ldq + (size_t)g * N;
  const float* kg = A.k + t * A.ldk + (size_t)g * N;
  float s_q = 0.f, s_k = 0.f, s_kq = 0.f;
  for (int n = tid; n < N; n += MS1_THREADS) {
    const float kv = kg[n], qv = qg[n];
    sk[n] = kv;
    sq[n] = qv;
    s_q = fmaf(qv, qv, s_q);
    s_k = fmaf(kv, kv, s_k);
    s_kq = fmaf(kv, qv, s_kq);
  }
  const float4 v = act ? *(const float4*)(A.v + t * A.ldv + (size_t)h * P + 4 * tx) : make_float4(0.f, 0.f, 0.f, 0.f);
  const float z1 = A.z1[t * A.ldz + h], z2 = A.z2[t * A.ldz + h];
  const float c1 = hb_to_float(((const TS*)A.w1)[h]), c2 = hb_to_float(((const TS*)A.w2)[h]);
  float a, b, inv = 1.f, fq = A.q_scale, fk = 1.f;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if constexpr (!DELTA) {
    const float li = ms_cap(z1 + c1, A.cap), lf = -ms_softplus(-ms_cap(z2 + c2, A.cap));
    float* mp = A.mstate + sl * H + h;
    const float m0 = *mp, m = fmaxf(lf + m0, li);
    a = expf(lf + m0 - m);
    b = expf(li - m);
    float nq = 0.f;
    float* ng = A.nstate + (sl * H + h) * N;
    for (int n = tid; n < N; n += MS1_THREADS) {          // (a thread's own elements of k and q)
      const float nn = fmaf(a, ng[n], b * sk[n]);
      ng[n] = nn;
      nq = fmaf(nn, sq[n], nq);
    }
    nq = hb_block_sum(nq, red);                           // its barriers also make k, q visible and follow every read of m
    if (tid == 0) *mp = m;
    inv = 1.f / (fmaxf(fabsf(nq * A.q_scale), expf(-m)) + A.den_eps);
    const float4 xv = make_float4(b * v.x, b * v.y, b * v.z, b * v.w);
#pragma unroll
    for (int i = 0; i < R; i++) {
      const int n = ty + i * TY;
      if (act && n < N) {
        const float kn = sk[n], qn = sq[n];
        S[i] = make_float4(fmaf(a, S[i].x, kn * xv.x), fmaf(a, S[i].y, kn * xv.y), fmaf(a, S[i].z, kn * xv.z), fmaf(a, S[i].w, kn * xv.w));
        *(float4*)(S_g + (size_t)n * P) = S[i];
        o.x = fmaf(S[i].x, qn, o.x); o.y = fmaf(S[i].y, qn, o.y); o.z = fmaf(S[i].z, qn, o.z); o.w = fmaf(S[i].w, qn, o.w);
      }
    }
    if (act) *(float4*)(part + (size_t)ty * P + 4 * tx) = o;
    __syncthreads();
  } else {
    a = expf(-expf(c2) * ms_softplus(z1 + c1));
    b = 1.f / (1.f + expf(-z2));
    s_q = hb_block_sum(s_q, red);
    s_k = hb_block_sum(s_k, red);
    s_kq = hb_block_sum(s_kq, red);
    fq = A.q_scale / sqrtf(s_q + A.unit_eps);
    fk = 1.f / sqrtf(s_k + A.unit_eps);
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < R; i++) {
      const int n = ty + i * TY;
      if (act && n < N) {
        const float kn = sk[n], qn = sq[n];
        u.x = fmaf(S[i].x, kn, u.x); u.y = fmaf(S[i].y, kn, u.y); u.z = fmaf(S[i].z, kn, u.z); u.w = fmaf(S[i].w, kn, u.w);
        o.x = fmaf(S[i].x, qn, o.x); o.y = fmaf(S[i].y, qn, o.y); o.z = fmaf(S[i].z, qn, o.z); o.w = fmaf(S[i].w, qn, o.w);
      }
    }
    if (act) {
      *(float4*)(part + (size_t)ty * P + 4 * tx) = o;
      *(float4*)(part2 + (size_t)ty * P + 4 * tx) = u;
    }
    __syncthreads();
    float* su = part2 + (size_t)TY * P;                   // [P]
    for (int p = tid; p < P; p += MS1_THREADS) {
      float us = 0.f;
      for (int y = 0; y < TY; y++) us += part2[(size_t)y * P + p];
      su[p] = b * fmaf(-a, us * fk, A.v[t * A.ldv + (size_t)h * P + p]);
    }
    __syncthreads();
    const float4 uu = act ? *(const float4*)(su + 4 * tx) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < R; i++) {
      const int n = ty + i * TY;
      if (act && n < N) {
        const float kn = sk[n] * fk;
        *(float4*)(S_g + (size_t)n * P) = make_float4(fmaf(kn, uu.x, a * S[i].x), fmaf(kn, uu.y, a * S[i].y), fmaf(kn, uu.z, a * S[i].z),
                                                      fmaf(kn, uu.w, a * S[i].w));
      }
    }
  }
  // the read-out's partial sums joined, the head norm, the weight and the gate: a column a thread
  float* so = DELTA ? part2 + (size_t)TY * P : part + (size_t)TY * P;       // [P] (delta: u lies there, read before o replaces it)
  float ss = 0.f;
  for (int p = tid; p < P; p += MS1_THREADS) {
    float os = 0.f;
    for (int y = 0; y < TY; y++) os += part[(size_t)y * P + p];
    os *= fq;
    if (DELTA) os = fmaf(s_kq * fk * fq, so[p], a * os);
    else os *= inv;
    so[p] = os;                                           // (a thread's own elements)
    ss = fmaf(os, os, ss);
  }
  const float f = rsqrtf(hb_block_sum(ss, red) / (float)P + A.eps);
  const TW* wr = (const TW*)A.w + (A.w_shared ? 0 : (size_t)h * P);
  const float* gr = A.gate + t * A.ldg + (size_t)h * P;
  for (int p = tid; p < P; p += MS1_THREADS) {
    const float z = gr[p], sg = 1.f / (1.f + expf(-z));
    ((TO*)A.out)[t * A.ldo + (size_t)h * P + p] = hb_from_float<TO>(so[p] * f * hb_to_float(wr[p]) * (A.gate_silu ? z * sg : sg));
  }
}

static size_t ms_single_smem(int N, int P, int delta) {
  const int TY = MS1_THREADS / (P / 4);
  return (size_t)(2 * N + (delta ? 2 : 1) * TY * P + P) * sizeof(float);
}

HB_EXPORT int hb_ms_single_supported(int N, int P, int delta) {
  if (P <= 0 || P % 4 || P > 4 * MS1_THREADS || N <= 0) return 0;
  const int TY = MS1_THREADS / (P / 4);
  return (N + TY - 1) / TY <= 16 && (N & 3) == 0 && ms_single_smem(N, P, delta) <= 48 * 1024;
}

HB_EXPORT int hb_ms_single(const float* q, long ldq, const float* k, long ldk, const float* v, long ldv, const float* z1, const float* z2,
                           long ldz, const void* w1, const void* w2, int s_dt, float cap, float unit_eps, float q_scale, float den_eps,
                           float eps, float* state, float* nstate, float* mstate, const int* q_start, const int* q_len, const int* slot,
                           const void* w, int w_dt, int w_shared, const float* gate, long ldg, int gate_silu, void* out, int o_dt, long ldo,
                           int n_requests, int H, int G, int N, int P, int delta, cudaStream_t s) {
  if (n_requests <= 0) return 0;
  if (!hb_ms_single_supported(N, P, delta)) HB_FAIL("hb_ms_single: heads of %d x %d are not a size it takes", N, P);
  if (G <= 0 || H % G || n_requests > 65535) HB_FAIL("hb_ms_single: %d heads over %d groups, %d requests", H, G, n_requests);
  if ((ldv & 3) || ((uintptr_t)v & 15) || ((uintptr_t)state & 15)) HB_FAIL("hb_ms_single: values and state must start on 16-byte boundaries");
  if (!delta && (!nstate || !mstate || !(cap > 0.f))) HB_FAIL("hb_ms_single: the linear form needs its normaliser, its maximum and a cap");
  SingleArgs A;
  A.q = q; A.k = k; A.v = v; A.ldq = ldq; A.ldk = ldk; A.ldv = ldv; A.z1 = z1; A.z2 = z2; A.ldz = ldz; A.w1 = w1; A.w2 = w2; A.cap = cap;
  A.unit_eps = unit_eps; A.q_scale = q_scale; A.den_eps = den_eps; A.eps = eps; A.state = state; A.nstate = nstate; A.mstate = mstate;
  A.q_start = q_start; A.q_len = q_len; A.slot = slot; A.w = w; A.w_shared = w_shared; A.gate = gate; A.ldg = ldg; A.gate_silu = gate_silu;
  A.out = out; A.ldo = ldo; A.H = H; A.G = G; A.N = N; A.P = P;
  const int TY = MS1_THREADS / (P / 4), per = (N + TY - 1) / TY;
  const size_t smem = ms_single_smem(N, P, delta);
  // the small vectors (biases, A_log, norm weight) share an element type: 32-bit engine or bfloat16 weights
  if (s_dt != w_dt) HB_FAIL("hb_ms_single: gate vectors of type %d beside a norm weight of type %d", s_dt, w_dt);
#define MS1_LAUNCH(R, DELTA)                                                                                                  \
  HB_DISPATCH_2(w_dt, o_dt, "hb_ms_single",                                                                                   \
                (hb_launch(ms_single_kernel<R, DELTA, TA, TA, TB>, dim3(H, n_requests), dim3(MS1_THREADS), smem, s, A)))
#define MS1_PICK(DELTA)                        \
  do {                                         \
    if (per <= 4) MS1_LAUNCH(4, DELTA);        \
    else if (per <= 8) MS1_LAUNCH(8, DELTA);   \
    else MS1_LAUNCH(16, DELTA);                \
  } while (0)
  if (delta) MS1_PICK(true);
  else MS1_PICK(false);
#undef MS1_PICK
#undef MS1_LAUNCH
  HB_CHECK_LAUNCH("hb_ms_single");
  return 0;
}
