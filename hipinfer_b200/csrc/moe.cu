// A routed feed-forward (mixture of experts): every token runs `top` of E small gated feed-forward layers.
//     z = Wr h (32-bit);  s = sigmoid(z);  the `top` largest s choose the experts (ties: the lower index)
//     out = sum over the chosen e of Wd_e (silu(Wg_e v) * (Wu_e v)),  v = s_e h
// The score multiplies the expert's INPUT. Experts have no biases, so Wg_e (s h) = s (Wg_e h): the products run on h and
// the score enters the activation in 32-bit, silu(s g) * (s u).
// A second form (route mode 1, `at_output`): z = Wr h + b; the `top` largest LOGITS choose; the weights are the softmax over
// the chosen logits alone and multiply the expert's RESULT, which, the down product being linear, is the activation times
// the weight, silu(g) * u * s, again in 32-bit.
// A third form (route mode 2): s = sigmoid(z); c = s + correction chooses, where the experts form equal groups of neighbours
// only among the groups that rank best by the sum of their two largest c; the weights are the chosen s (without the
// correction) divided by their sum, times a constant.
// A fourth form (route mode 3): s = softmax(z) over all E; c = s + correction chooses, within the groups that rank best by their
// largest c; the weights are the chosen s as they are.
// Identity experts (any form): the last of the E router rows name experts without weights, whose result is the row itself:
// their weights' sum goes to a number per token and what adds the results up adds the row times it. Beside the router's rows one more row may give a number per token,
// sigmoid(w . h), that a shared expert's result is multiplied by.
//
// moe_route_kernel          scores and the chosen experts of every row: expert [T][top], weight [T][top]
// Few rows (decoding): no sorting, nothing on the host
//   moe_gate_up_rows_kernel a block per ((row, choice), tile of the expert's hidden rows): act [T * top][F]
//   moe_down_rows_kernel    a block per (row, tile of output columns): the choices' results summed in their order
// Some rows (decoding in a batch): the pairs sorted by expert on the device, then
//   moe_grouped_kernel      a block per (expert, tile of output features): the expert's weights are read once for all of
//   moe_grouped_mma_kernel  its rows (a round of them at a time), for the gate/up product and for the down product;
//                           nothing on the host, so the step replays from a CUDA graph. The second is the bfloat16 form on
//                           warp MMAs, with the activation in the gate/up product; the first takes any element types and sizes
// Many rows (prompt portions): the (row, choice) pairs are sorted by expert, so that each expert's rows are one
// contiguous block that an ordinary product takes
//   moe_sort_kernel         offsets [E + 1], pos [pair] -> sorted row, src [sorted row] -> pair
//   moe_gather_kernel       the sorted copy of the input rows
//   moe_act_kernel          silu(s g) * (s u) on the sorted rows' 32-bit [g | u]
//   moe_combine_kernel      out[t] += sum over the choices, in their order, of the sorted results
#include "common.cuh"

constexpr int MR_THREADS = 512;

// Eight elements of two rows multiplied and added up: one 16-byte access a row where both are bfloat16.
__device__ __forceinline__ float mr_dot8(const __nv_bfloat16* a, const __nv_bfloat16* w, float acc) {
  const uint4 x = *(const uint4*)a, y = *(const uint4*)w;
  const __nv_bfloat162 *xp = (const __nv_bfloat162*)&x, *yp = (const __nv_bfloat162*)&y;
#pragma unroll
  for (int i = 0; i < 4; i++) {
    const float2 u = __bfloat1622float2(xp[i]), v = __bfloat1622float2(yp[i]);
    acc = fmaf(v.x, u.x, acc);
    acc = fmaf(v.y, u.y, acc);
  }
  return acc;
}
template <typename TA, typename TW>
__device__ __forceinline__ float mr_dot8(const TA* a, const TW* w, float acc) {
#pragma unroll
  for (int i = 0; i < 8; i += 4) {
    const float4 u = hb_load4(a + i), v = hb_load4(w + i);
    acc = fmaf(v.x, u.x, acc);
    acc = fmaf(v.y, u.y, acc);
    acc = fmaf(v.z, u.z, acc);
    acc = fmaf(v.w, u.w, acc);
  }
  return acc;
}

// A warp a router row (and the shared expert's gate), the token's row read beside it; then warp 0 ranks the groups, marks the
// experts of those that do not stay as taken (NaN), and picks the largest `top` times, ties to the lower index.
template <typename TA, typename TW>
__global__ void __launch_bounds__(MR_THREADS) moe_route_kernel(const TA* __restrict__ xn, long ldx, const TW* __restrict__ router,
                                                               const TW* __restrict__ bias, int* __restrict__ expert,
                                                               float* __restrict__ weight, int W, int E, int top, int mode,
                                                               const TW* __restrict__ correction, int groups, int keep, float scale,
                                                               const TW* __restrict__ shared_gate, float* __restrict__ shared_weight,
                                                               int vec, int n_real, float* __restrict__ identity_weight) {
  extern __shared__ float mr_sm[];     // [E] the scores, [E] those without the correction, [E] corrections, [groups] the groups' ranks, [top] weights
  float* sc = mr_sm;
  float* plain = sc + E;
  float* corr = plain + E;
  float* gs = corr + E;
  float* picked = gs + groups;
  hb_pdl_launch();
  hb_pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  const TA* row = xn + (size_t)t * ldx;
  for (int e = threadIdx.x; e < E; e += blockDim.x) corr[e] = correction ? hb_to_float(correction[e]) : 0.f;     // (asked for beside the rows)
  for (int e = warp; e < E + (shared_gate ? 1 : 0); e += nw) {
    const TW* wr = e < E ? router + (size_t)e * W : shared_gate;
    float acc = 0.f;
    if (vec) {
#pragma unroll 8
      for (int i = lane * 8; i < W; i += 256) acc = mr_dot8(row + i, wr + i, acc);
    } else {
      for (int i = lane; i < W; i += 32) acc = fmaf(hb_to_float(row[i]), hb_to_float(wr[i]), acc);
    }
    acc = hb_warp_sum(acc);
    if (lane != 0) continue;
    if (e == E) {
      shared_weight[t] = 1.f / (1.f + expf(-acc));
      continue;
    }
    if (bias) acc += hb_to_float(bias[e]);
    const float v = mode == 1 || mode == 3 ? acc : 1.f / (1.f + expf(-acc));
    sc[e] = v;
    plain[e] = v;
  }
  __syncthreads();
  if (warp != 0) return;
  if (mode == 2) {
    for (int e = lane; e < E; e += 32) sc[e] += corr[e];
    __syncwarp();
  }
  if (mode == 3) {                       // the softmax over all E, then the corrections
    float mx = -INFINITY, sum = 0.f;
    for (int e = lane; e < E; e += 32) mx = fmaxf(mx, plain[e]);
    mx = hb_warp_max(mx);
    for (int e = lane; e < E; e += 32) sum += expf(plain[e] - mx);
    sum = hb_warp_sum(sum);
    for (int e = lane; e < E; e += 32) {
      const float v = expf(plain[e] - mx) / sum;
      plain[e] = v;
      sc[e] = v + corr[e];
    }
    __syncwarp();
  }
  if (mode >= 2 && groups > 1) {
    const int span = E / groups;
    for (int q = lane; q < groups; q += 32) {
      float a = -INFINITY, b = -INFINITY;                  // the two largest
      for (int e = q * span; e < (q + 1) * span; e++) {
        const float v = sc[e];
        if (v > a) { b = a; a = v; } else if (v > b) b = v;
      }
      gs[q] = span > 1 && mode == 2 ? a + b : a;
    }
    __syncwarp();
    for (int q = lane; q < groups; q += 32) {
      const float v = gs[q];
      int ahead = 0;
      for (int p = 0; p < groups; p++) ahead += gs[p] > v || (gs[p] == v && p < q);
      if (ahead >= keep)
        for (int e = q * span; e < (q + 1) * span; e++) sc[e] = __int_as_float(0x7fc00000);
    }
    __syncwarp();
  }
  float first = 0.f, den = 0.f, idw = 0.f;
  for (int k = 0; k < top; k++) {
    float bs = -INFINITY;
    int best = E;
    for (int e = lane; e < E; e += 32) {
      const float v = sc[e];
      if (v == v && (best == E || v > bs)) { bs = v; best = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bs, o);
      const int oe = __shfl_xor_sync(0xffffffffu, best, o);
      if (oe < E && (best == E || ov > bs || (ov == bs && oe < best))) { bs = ov; best = oe; }
    }
    if (best == E) best = 0;             // every score NaN (bad weights or input): stay inside the tables
    // softmax over the chosen logits alone (mode 1): the first chosen one is the largest
    if (k == 0) first = bs;
    const float w = mode == 1 ? expf(bs - first) : plain[best];
    den += w;
    if (best >= n_real) idw += w;
    if (lane == 0) {
      expert[(size_t)t * top + k] = best;
      picked[k] = w;
      sc[best] = __int_as_float(0x7fc00000);
    }
    __syncwarp();
  }
  if (identity_weight && lane == 0) identity_weight[t] = idw;
  for (int k = lane; k < top; k += 32) {
    const float w = picked[k];
    weight[(size_t)t * top + k] = mode == 1 ? w / den : mode == 2 ? w / (den + 1e-20f) * scale : w;
  }
}

// mode 0: the scores are sigmoid(z) and the chosen scores are the weights; mode 1: the largest logits z choose and the
// weights are the softmax over the chosen logits alone; mode 2: sigmoid(z) + correction [E] chooses, within the `keep` best of
// `groups` groups, and the weights are the chosen sigmoid(z) over their sum, times scale. bias (the router's element type, or
// null) is added to z. mode 3: softmax(z) + correction (or null) chooses, within the groups whose largest is largest, and the
// weights are the chosen softmax(z). identity_weight [T] (or null; modes 0 and 3): the sum of the weights of the chosen experts
// from n_real on. shared_gate [W] (or null): shared_weight[t] = sigmoid(shared_gate . row).
HB_EXPORT int hb_moe_route(const void* xn, int x_dt, long ldx, const void* router, const void* bias, int w_dt, int* expert,
                           float* weight, int T, int W, int E, int top, int mode, const void* correction, int groups, int keep,
                           float scale, const void* shared_gate, float* shared_weight, int n_real, float* identity_weight, cudaStream_t s) {
  if (T <= 0) return 0;
  if (mode == 2 && !correction) HB_FAIL("hb_moe_route: the third form needs its corrections");
  if (mode < 0 || mode > 3) HB_FAIL("hb_moe_route: unknown form %d", mode);
  if (n_real < E && (!identity_weight || (mode != 0 && mode != 3)))
    HB_FAIL("hb_moe_route: identity experts need a place for their weight and weights that are not normalised");
  if (groups > 1 && (E % groups || keep < 1 || keep > groups || (long)keep * (E / groups) < top))
    HB_FAIL("hb_moe_route: %d experts in %d groups of which %d stay, %d chosen", E, groups, keep, top);
  if (shared_gate && !shared_weight) HB_FAIL("hb_moe_route: a shared expert's gate needs a place for its result");
  if (top < 1 || top > E) HB_FAIL("hb_moe_route: top %d of %d experts", top, E);
  const size_t smem = (size_t)(3 * E + groups + top) * sizeof(float);
  const int vec = W % 8 == 0 && ldx % 8 == 0 && !(((uintptr_t)router | (uintptr_t)shared_gate | (uintptr_t)xn) & 15);
  const int rows = E + (shared_gate ? 1 : 0), threads = 32 * (rows < MR_THREADS / 32 ? rows : MR_THREADS / 32);
  if (smem > 200 * 1024) HB_FAIL("hb_moe_route: %d experts in %d groups do not fit shared memory", E, groups);
  HB_DISPATCH_2(x_dt, w_dt, "hb_moe_route", do {
    auto kern = moe_route_kernel<TA, TB>;
    if (smem > 40 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    hb_launch(kern, dim3(T), dim3(threads), smem, s, (const TA*)xn, ldx, (const TB*)router, (const TB*)bias, expert, weight,
              W, E, top, mode, (const TB*)correction, groups, keep, scale, (const TB*)shared_gate, shared_weight, vec, n_real, identity_weight);
  } while (0));
  HB_CHECK_LAUNCH("hb_moe_route");
  return 0;
}

// A warp's dot product of a weight row with a 32-bit row in shared memory: lanes take groups of four columns (scalar
// columns where K is no multiple of four), the lanes' sums are joined in a fixed order.
template <typename TW>
__device__ __forceinline__ float moe_warp_dot(const TW* __restrict__ w, const float* __restrict__ a, int K, int lane, bool vec) {
  float acc = 0.f;
  if (vec) {
    for (int i = lane * 4; i < K; i += 128) {
      const float4 wv = hb_load4(w + i);
      const float4 av = *(const float4*)(a + i);
      acc = fmaf(wv.x, av.x, acc);
      acc = fmaf(wv.y, av.y, acc);
      acc = fmaf(wv.z, av.z, acc);
      acc = fmaf(wv.w, av.w, acc);
    }
  } else {
    for (int i = lane; i < K; i += 32) acc = fmaf(hb_to_float(w[i]), a[i], acc);
  }
  return hb_warp_sum(acc);
}

constexpr int MG_THREADS = 256, MG_ROWS = 32;

// An expert's gate and up rows take turns, grp of each (16: the layout of the gated epilogues; F: gate rows first): where hidden
// unit j's gate row lies; its up row is grp further.
__device__ __forceinline__ int moe_gate_row(int j, int grp) { return j / grp * 2 * grp + j % grp; }

template <typename TA, typename TW, typename TO>
__global__ void __launch_bounds__(MG_THREADS) moe_gate_up_rows_kernel(const TA* __restrict__ xn, long ldx,
                                                                      const TW* __restrict__ wgu, const int* __restrict__ expert,
                                                                      const float* __restrict__ weight, TO* __restrict__ act,
                                                                      int W, int F, int top, int vec, int at_output, int E, int grp) {
  extern __shared__ __align__(16) float mg_row[];      // [W]
  hb_pdl_launch();
  hb_pdl_wait();
  const int pair = blockIdx.y, t = pair / top, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if (expert[pair] >= E) return;                       // an identity expert has no hidden rows
  for (int i = threadIdx.x; i < W; i += MG_THREADS) mg_row[i] = hb_to_float(xn[(size_t)t * ldx + i]);
  __syncthreads();
  const int e = expert[pair];
  const float sw = weight[pair];
  const float s = at_output ? 1.f : sw, so = at_output ? sw : 1.f;     // the weight multiplies the input, or the result
  const TW* we = wgu + (size_t)e * 2 * F * W;          // gate and up rows in turn, grp of each
  const int j1 = min(F, (int)(blockIdx.x + 1) * MG_ROWS);
  for (int j = blockIdx.x * MG_ROWS + warp; j < j1; j += MG_THREADS / 32) {
    const int jg = moe_gate_row(j, grp);
    const float g = s * moe_warp_dot(we + (size_t)jg * W, mg_row, W, lane, vec);
    const float u = s * moe_warp_dot(we + (size_t)(jg + grp) * W, mg_row, W, lane, vec);
    if (lane == 0) act[(size_t)pair * F + j] = hb_from_float<TO>(g / (1.f + expf(-g)) * u * so);
  }
}

HB_EXPORT int hb_moe_gate_up_rows(const void* xn, int x_dt, long ldx, const void* wgu, int w_dt, const int* expert,
                                  const float* weight, void* act, int T, int W, int F, int top, int at_output, int E, int grp, cudaStream_t s) {
  if (T <= 0) return 0;
  if (grp < 1 || F % grp) HB_FAIL("hb_moe_gate_up_rows: %d hidden rows in groups of %d", F, grp);
  const size_t smem = (size_t)W * sizeof(float);
  if (smem > 200 * 1024) HB_FAIL("hb_moe_gate_up_rows: a row of %d does not fit shared memory", W);
  const int vec = (W % 4 == 0) ? 1 : 0;
  dim3 grid((F + MG_ROWS - 1) / MG_ROWS, T * top);
  if (grid.y > 65535) HB_FAIL("hb_moe_gate_up_rows: %d rows x %d choices are too many for this kernel", T, top);
  // the activation has the input's element type
  HB_DISPATCH_2(x_dt, w_dt, "hb_moe_gate_up_rows", do {
    auto kern = moe_gate_up_rows_kernel<TA, TB, TA>;
    if (smem > 40 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    hb_launch(kern, grid, dim3(MG_THREADS), smem, s, (const TA*)xn, ldx, (const TB*)wgu, expert, weight, (TA*)act, W, F, top, vec, at_output, E, grp);
  } while (0));
  HB_CHECK_LAUNCH("hb_moe_gate_up_rows");
  return 0;
}

template <typename TA, typename TW>
__global__ void __launch_bounds__(MG_THREADS) moe_down_rows_kernel(const TA* __restrict__ act, const TW* __restrict__ wd,
                                                                   const int* __restrict__ expert, float* __restrict__ y, long ldy,
                                                                   int W, int F, int top, int vec, int E, const TA* __restrict__ xn,
                                                                   long ldx, const float* __restrict__ identity_weight) {
  extern __shared__ __align__(16) float md_act[];      // [top][F4], F4 = F rounded up to four
  hb_pdl_launch();
  hb_pdl_wait();
  const int t = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int F4 = (F + 3) & ~3;
  for (int i = threadIdx.x; i < top * F; i += MG_THREADS) {
    const int k = i / F, j = i - k * F;
    md_act[k * F4 + j] = expert[(size_t)t * top + k] < E ? hb_to_float(act[((size_t)t * top + k) * F + j]) : 0.f;
  }
  __syncthreads();
  const int n1 = min(W, (int)(blockIdx.x + 1) * MG_ROWS);
  for (int n = blockIdx.x * MG_ROWS + warp; n < n1; n += MG_THREADS / 32) {
    float acc = 0.f;
    for (int k = 0; k < top; k++) {
      const int e = expert[(size_t)t * top + k];
      if (e >= E) continue;
      acc += moe_warp_dot(wd + ((size_t)e * W + n) * F, md_act + k * F4, F, lane, vec);
    }
    if (lane == 0) {
      if (identity_weight) acc = fmaf(identity_weight[t], hb_to_float(xn[(size_t)t * ldx + n]), acc);
      y[(size_t)t * ldy + n] += acc;
    }
  }
}

HB_EXPORT int hb_moe_down_rows(const void* act, int a_dt, const void* wd, int w_dt, const int* expert, float* y, long ldy, int T,
                               int W, int F, int top, int E, const void* xn, long ldx, const float* identity_weight, cudaStream_t s) {
  if (T <= 0) return 0;
  const size_t smem = (size_t)top * ((F + 3) & ~3) * sizeof(float);
  if (smem > 200 * 1024) HB_FAIL("hb_moe_down_rows: %d x %d activations do not fit shared memory", top, F);
  const int vec = (F % 4 == 0) ? 1 : 0;
  dim3 grid((W + MG_ROWS - 1) / MG_ROWS, T);
  if (grid.y > 65535) HB_FAIL("hb_moe_down_rows: %d rows are too many for this kernel", T);
  HB_DISPATCH_2(a_dt, w_dt, "hb_moe_down_rows", do {
    auto kern = moe_down_rows_kernel<TA, TB>;
    if (smem > 40 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    hb_launch(kern, grid, dim3(MG_THREADS), smem, s, (const TA*)act, (const TB*)wd, expert, y, ldy, W, F, top, vec, E,
              (const TA*)xn, ldx, identity_weight);
  } while (0));
  HB_CHECK_LAUNCH("hb_moe_down_rows");
  return 0;
}

// ---------------------------------------------------------------------------------------------------------------------
// Some rows: one product kernel over all experts' blocks of sorted rows.
//   out[r][n] = sum_k w[e][n][k] a[row(r)][k]   for offsets[e] <= r < offsets[e + 1], e = blockIdx.y
// row(r) = src[r] / top where src is given (the step's input rows, gathered on the fly), else r. A warp owns MX_NW output
// features and MX_RB rows at a time: a weight row comes from memory once a round of rows, the rows wait in shared memory in
// their own element type, K in segments of KS. A (row, feature) sum runs in the same order whatever else is in the round.
// ---------------------------------------------------------------------------------------------------------------------
constexpr int MX_THREADS = 256, MX_RB = 8, MX_NW = 4, MX_TILE = (MX_THREADS / 32) * MX_NW;

// 16 bytes of a weight: read once a step, so not kept in L1, which the rows share.
__device__ __forceinline__ uint4 hb_ldg_once(const uint4* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

template <typename T> struct MxVec4;
template <> struct MxVec4<float> { using type = float4; };
template <> struct MxVec4<__nv_bfloat16> { using type = uint2; };

// One round: R rows (the first nr of them live) against the block's MX_TILE output features.
template <typename TA, typename TW, int R>
__device__ __forceinline__ void mx_round(const TA* __restrict__ a, long lda, const int* mx_row, int nr, const TW* __restrict__ we,
                                         float* __restrict__ out, TA* rows, int g0, int n0, int Nout, int K, int KS, int vec) {
  using V4 = typename MxVec4<TA>::type;
  const int tid = threadIdx.x, lane = tid & 31;
  float acc[MX_NW][R];
#pragma unroll
  for (int q = 0; q < MX_NW; q++)
#pragma unroll
    for (int r = 0; r < R; r++) acc[q][r] = 0.f;
  for (int k0 = 0; k0 < K; k0 += KS) {
    const int kn = min(KS, K - k0);
    __syncthreads();                                        // the segment before has been read; mx_row is written
    if (vec) {
      const int per = kn >> 2;
      for (int r = 0; r < nr; r++) {
        const TA* ar = a + (size_t)mx_row[r] * lda + k0;
#pragma unroll 4
        for (int i = tid; i < per; i += MX_THREADS) *(V4*)(rows + (size_t)r * KS + 4 * i) = *(const V4*)(ar + 4 * i);
      }
    } else {
      for (int r = 0; r < nr; r++) {
        const TA* ar = a + (size_t)mx_row[r] * lda + k0;
        for (int i = tid; i < kn; i += MX_THREADS) rows[(size_t)r * KS + i] = ar[i];
      }
    }
    __syncthreads();
    if (vec) {
#pragma unroll 2
      for (int i = lane * 4; i < kn; i += 128) {
        float4 wv[MX_NW];
#pragma unroll
        for (int q = 0; q < MX_NW; q++)
          wv[q] = n0 + q < Nout ? hb_load4(we + (size_t)(n0 + q) * K + k0 + i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int r = 0; r < R; r++) {
          const float4 av = hb_load4(rows + (size_t)r * KS + i);
#pragma unroll
          for (int q = 0; q < MX_NW; q++) {
            acc[q][r] = fmaf(wv[q].x, av.x, acc[q][r]);
            acc[q][r] = fmaf(wv[q].y, av.y, acc[q][r]);
            acc[q][r] = fmaf(wv[q].z, av.z, acc[q][r]);
            acc[q][r] = fmaf(wv[q].w, av.w, acc[q][r]);
          }
        }
      }
    } else {
      for (int i = lane; i < kn; i += 32) {
        float wv[MX_NW];
#pragma unroll
        for (int q = 0; q < MX_NW; q++) wv[q] = n0 + q < Nout ? hb_to_float(we[(size_t)(n0 + q) * K + k0 + i]) : 0.f;
#pragma unroll
        for (int r = 0; r < R; r++) {
          const float av = hb_to_float(rows[(size_t)r * KS + i]);
#pragma unroll
          for (int q = 0; q < MX_NW; q++) acc[q][r] = fmaf(wv[q], av, acc[q][r]);
        }
      }
    }
  }
  // rows beyond nr hold whatever shared memory held: their sums are never stored
#pragma unroll
  for (int q = 0; q < MX_NW; q++)
#pragma unroll
    for (int r = 0; r < R; r++) {
      const float v = hb_warp_sum(acc[q][r]);
      if (lane == 0 && n0 + q < Nout && r < nr) out[(size_t)(g0 + r) * Nout + n0 + q] = v;
    }
}

template <typename TA, typename TW>
__global__ void __launch_bounds__(MX_THREADS) moe_grouped_kernel(const TA* __restrict__ a, long lda, const int* __restrict__ src,
                                                                 int top, const TW* __restrict__ w, const int* __restrict__ offsets,
                                                                 float* __restrict__ out, int Nout, int K, int KS, int vec) {
  extern __shared__ __align__(16) unsigned char mx_raw[];
  __shared__ int mx_row[MX_RB];
  TA* rows = (TA*)mx_raw;                                   // [MX_RB][KS]
  hb_pdl_launch();
  hb_pdl_wait();
  const int e = blockIdx.y, lo = offsets[e], hi = offsets[e + 1];
  if (lo >= hi) return;
  const int tid = threadIdx.x, warp = tid >> 5;
  const int n0 = blockIdx.x * MX_TILE + warp * MX_NW;
  const TW* we = w + (size_t)e * Nout * K;
  for (int g0 = lo; g0 < hi; g0 += MX_RB) {
    const int nr = min(MX_RB, hi - g0);
    __syncthreads();                                        // the round before has read its row numbers
    if (tid < nr) mx_row[tid] = src ? src[g0 + tid] / top : g0 + tid;
    // a round of few rows does the sums of few rows; which form a row meets changes nothing in its sums
    if (nr == 1) mx_round<TA, TW, 1>(a, lda, mx_row, nr, we, out, rows, g0, n0, Nout, K, KS, vec);
    else if (nr == 2) mx_round<TA, TW, 2>(a, lda, mx_row, nr, we, out, rows, g0, n0, Nout, K, KS, vec);
    else if (nr <= 4) mx_round<TA, TW, 4>(a, lda, mx_row, nr, we, out, rows, g0, n0, Nout, K, KS, vec);
    else mx_round<TA, TW, MX_RB>(a, lda, mx_row, nr, we, out, rows, g0, n0, Nout, K, KS, vec);
  }
}

// The same product on warp MMAs (bfloat16 rows and weights, K a multiple of 32), and the gate/up product with its activation. A
// warp owns 16 weight rows, the MMA's row operand, over one of KW equal parts of K; the rows are the column operand, 8 a tile, up
// to 4 tiles a round. Both come straight from memory (the rows from L1 and L2: every warp of a block reads the same ones): a lane
// reads 8 consecutive k (16 bytes) of weight rows g and g + 8 and of row g of every tile per block of 32 k. Inside a block of 32 k
// the lanes' k are dealt to the MMA's k slots in another order than memory's, the same for both operands, which a sum over k does
// not see. The loads of the next MU blocks are under way while this one's products run: no shared memory and no barrier between
// a warp and its weights. The parts of K are added in their order through shared memory. 32-bit accumulation; a (row, feature) sum
// does not depend on the other rows of the round.
// ACT: the 16 weight rows are 8 gate rows and the 8 up rows that go with them, so that a thread holds both halves of its hidden
// units: it applies the activation and the pair's weight and writes bfloat16.
constexpr int MM_THREADS = 128, MM_WARPS = MM_THREADS / 32, MM_ROWS = 32;

__device__ __forceinline__ void mm_mma(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

struct MmArgs {
  const __nv_bfloat16* a;      // the rows
  long lda;
  const int* src;              // sorted row -> pair, or null: the rows are sorted already
  int top;
  const __nv_bfloat16* w;      // [E][Nw][K]
  const int* offsets;          // [E + 1]
  const float* weight;         // ACT: [pairs]
  __nv_bfloat16* act;          // ACT: [sorted rows][Nout]
  float* out;                  // else: [sorted rows][Nout]
  int Nout, Nw, K, at_output, grp;
};

template <int NT, int KW, bool ACT>
__device__ __forceinline__ void mm_round(const MmArgs& A, const __nv_bfloat16* __restrict__ we, int g0, int nr, float* red) {
  constexpr int MU = NT == 4 ? 2 : 4, FT = ACT ? 8 : 16, TILES = MM_WARPS / KW;     // blocks of 32 k a stage; features and tiles
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int tile = warp / KW, part = warp % KW, n0 = (blockIdx.x * TILES + tile) * FT;
  const int nb = A.K >> 5, b0 = nb * part / KW, b1 = nb * (part + 1) / KW;
  // features past the end read the last one's weights, rows past the round's end its first row: their sums are not stored
  const int fa = min(n0 + g, A.Nout - 1), ra = ACT ? moe_gate_row(fa, A.grp) : fa, rb = ACT ? ra + A.grp : min(n0 + g + 8, A.Nout - 1);
  const uint4* wa = (const uint4*)(we + (size_t)ra * A.K) + t;
  const uint4* wb = (const uint4*)(we + (size_t)rb * A.K) + t;
  const uint4* row[NT];
#pragma unroll
  for (int nt = 0; nt < NT; nt++) {
    const int r = g0 + (nt * 8 + g < nr ? nt * 8 + g : 0);
    row[nt] = (const uint4*)(A.a + (size_t)(A.src ? A.src[r] / A.top : r) * A.lda) + t;
  }
  float acc[NT][4];
#pragma unroll
  for (int nt = 0; nt < NT; nt++)
#pragma unroll
    for (int i = 0; i < 4; i++) acc[nt][i] = 0.f;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  uint4 A0[MU], A1[MU], B[MU][NT];
  auto load = [&](int b, uint4 (&x0)[MU], uint4 (&x1)[MU], uint4 (&y)[MU][NT]) {
#pragma unroll
    for (int u = 0; u < MU; u++) {
      const bool in = b + u < b1;
      x0[u] = in ? hb_ldg_once(wa + (b + u) * 4) : zero;
      x1[u] = in ? hb_ldg_once(wb + (b + u) * 4) : zero;
    }
#pragma unroll
    for (int u = 0; u < MU; u++)
#pragma unroll
      for (int nt = 0; nt < NT; nt++) y[u][nt] = b + u < b1 ? row[nt][(b + u) * 4] : zero;
  };
  load(b0, A0, A1, B);
  for (int b = b0; b < b1; b += MU) {
    uint4 N0[MU], N1[MU], NB[MU][NT];
    load(b + MU, N0, N1, NB);
#pragma unroll
    for (int u = 0; u < MU; u++)
#pragma unroll
      for (int nt = 0; nt < NT; nt++) {
        mm_mma(acc[nt], A0[u].x, A1[u].x, A0[u].y, A1[u].y, B[u][nt].x, B[u][nt].y);
        mm_mma(acc[nt], A0[u].z, A1[u].z, A0[u].w, A1[u].w, B[u][nt].z, B[u][nt].w);
      }
#pragma unroll
    for (int u = 0; u < MU; u++) {
      A0[u] = N0[u];
      A1[u] = N1[u];
#pragma unroll
      for (int nt = 0; nt < NT; nt++) B[u][nt] = NB[u][nt];
    }
  }
  if constexpr (KW > 1) {
    __syncthreads();                                        // the round before has read its sums
    if (part > 0) {
#pragma unroll
      for (int nt = 0; nt < NT; nt++)
#pragma unroll
        for (int i = 0; i < 4; i++) red[((warp * NT + nt) * 4 + i) * 32 + lane] = acc[nt][i];
    }
    __syncthreads();
    if (part > 0) return;
#pragma unroll
    for (int q = 1; q < KW; q++)
#pragma unroll
      for (int nt = 0; nt < NT; nt++)
#pragma unroll
        for (int i = 0; i < 4; i++) acc[nt][i] += red[(((warp + q) * NT + nt) * 4 + i) * 32 + lane];
  }
#pragma unroll
  for (int nt = 0; nt < NT; nt++)
#pragma unroll
    for (int i = 0; i < 2; i++) {
      const int r = nt * 8 + 2 * t + i;
      if (r >= nr) continue;
      if constexpr (ACT) {
        if (n0 + g >= A.Nout) continue;
        const float sw = A.weight[A.src[g0 + r]], s = A.at_output ? 1.f : sw, so = A.at_output ? sw : 1.f;
        const float gt = s * acc[nt][i], up = s * acc[nt][2 + i];
        A.act[(size_t)(g0 + r) * A.Nout + n0 + g] = __float2bfloat16_rn(gt / (1.f + expf(-gt)) * up * so);
      } else {
        if (n0 + g < A.Nout) A.out[(size_t)(g0 + r) * A.Nout + n0 + g] = acc[nt][i];
        if (n0 + g + 8 < A.Nout) A.out[(size_t)(g0 + r) * A.Nout + n0 + g + 8] = acc[nt][2 + i];
      }
    }
}

template <int KW, bool ACT>
__global__ void __launch_bounds__(MM_THREADS, 3) moe_grouped_mma_kernel(MmArgs A) {
  __shared__ float red[KW > 1 ? MM_WARPS * 4 * 4 * 32 : 1];
  hb_pdl_launch();
  hb_pdl_wait();
  const int e = blockIdx.y, lo = A.offsets[e], hi = A.offsets[e + 1];
  const __nv_bfloat16* we = A.w + (size_t)e * A.Nw * A.K;
  for (int g0 = lo; g0 < hi; g0 += MM_ROWS) {
    const int nr = min(MM_ROWS, hi - g0);
    if (nr <= 8) mm_round<1, KW, ACT>(A, we, g0, nr, red);
    else if (nr <= 16) mm_round<2, KW, ACT>(A, we, g0, nr, red);
    else mm_round<4, KW, ACT>(A, we, g0, nr, red);
  }
}

static bool mm_ok(const void* a, int a_dt, long lda, const void* w, int w_dt, int K) {
  return a_dt == HB_BF16 && w_dt == HB_BF16 && K % 32 == 0 && lda % 8 == 0 && !(((uintptr_t)a | (uintptr_t)w) & 15);
}

template <bool ACT>
static void mm_launch(const MmArgs& A, int E, int parts, cudaStream_t s) {
  // the parts of K follow from K alone: short walks, and enough warps to fill the machine when only a few experts have rows
  constexpr int FT = ACT ? 8 : 16;
  const int tiles = (A.Nout + FT - 1) / FT, kw = parts ? parts : A.K >= 512 ? 4 : A.K >= 256 ? 2 : 1;
  const dim3 grid((tiles * kw + MM_WARPS - 1) / MM_WARPS, E);
  auto kern = kw == 1 ? moe_grouped_mma_kernel<1, ACT> : kw == 2 ? moe_grouped_mma_kernel<2, ACT> : moe_grouped_mma_kernel<4, ACT>;
  // The first of the two is an ordinary launch: started early beside a kernel that holds much shared memory, its blocks would find
  // the SM's memory split in that kernel's favour and little L1 for the rows (116 us instead of 69 us at 64 rows). The second
  // follows the first, which uses none.
  if (ACT) kern<<<grid, MM_THREADS, 0, s>>>(A);
  else hb_launch(kern, grid, dim3(MM_THREADS), 0, s, A);
}

// act[r] (bfloat16, sorted rows) = silu(s g) * (s u) times the rest of the pair's weight, [g | u] = w[e] row: the gate/up product
// with its activation in one kernel. parts: of K, 1, 2 or 4 (0: what suits the sizes). Returns 1 (nothing done) where the sizes or element types are not its.
HB_EXPORT int hb_moe_grouped_act(const void* a, int a_dt, long lda, const int* src, int top, const void* w, int w_dt, const int* offsets,
                                 const float* weight, void* act, int E, int F, int K, int at_output, int parts, int grp, cudaStream_t s) {
  if (grp < 1 || F % grp) HB_FAIL("hb_moe_grouped_act: %d hidden rows in groups of %d", F, grp);
  if (parts != 0 && parts != 1 && parts != 2 && parts != 4) HB_FAIL("hb_moe_grouped_act: %d parts of K", parts);
  if (E <= 0 || F <= 0 || K <= 0) return 0;
  if (!mm_ok(a, a_dt, lda, w, w_dt, K) || !src || E > 65535) return 1;
  mm_launch<true>(MmArgs{(const __nv_bfloat16*)a, lda, src, top, (const __nv_bfloat16*)w, offsets, weight, (__nv_bfloat16*)act, nullptr, F, 2 * F,
                         K, at_output, grp}, E, parts, s);
  HB_CHECK_LAUNCH("hb_moe_grouped_act");
  return 0;
}

HB_EXPORT int hb_moe_grouped(const void* a, int a_dt, long lda, const int* src, int top, const void* w, int w_dt,
                             const int* offsets, float* out, int E, int Nout, int K, int parts, cudaStream_t s) {
  if (parts != 0 && parts != 1 && parts != 2 && parts != 4) HB_FAIL("hb_moe_grouped: %d parts of K", parts);
  if (E <= 0 || Nout <= 0 || K <= 0) return 0;
  if (E > 65535) HB_FAIL("hb_moe_grouped: %d experts are too many for this kernel", E);
  if (mm_ok(a, a_dt, lda, w, w_dt, K)) {
    mm_launch<false>(MmArgs{(const __nv_bfloat16*)a, lda, src, top, (const __nv_bfloat16*)w, offsets, nullptr, nullptr, out, Nout, Nout, K, 0, 0}, E, parts, s);
    HB_CHECK_LAUNCH("hb_moe_grouped");
    return 0;
  }
  const int esz = a_dt == HB_F32 ? 4 : 2;
  const int vec = (K % 4 == 0 && lda % 4 == 0 && ((uintptr_t)a & 15) == 0 && ((uintptr_t)w & 15) == 0) ? 1 : 0;
  const int cap = (64 * 1024 / (MX_RB * esz)) & ~3;        // a segment's elements a row
  const int KS = K < cap ? ((K + 3) & ~3) : cap;
  const size_t smem = (size_t)MX_RB * KS * esz;
  dim3 grid((Nout + MX_TILE - 1) / MX_TILE, E);
  HB_DISPATCH_2(a_dt, w_dt, "hb_moe_grouped", do {
    auto kern = moe_grouped_kernel<TA, TB>;
    if (smem > 40 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    hb_launch(kern, grid, dim3(MX_THREADS), smem, s, (const TA*)a, lda, src, top, (const TB*)w, offsets, out, Nout, K, KS, vec);
  } while (0));
  HB_CHECK_LAUNCH("hb_moe_grouped");
  return 0;
}

// ---------------------------------------------------------------------------------------------------------------------
// Many rows: the pairs sorted by expert.
// ---------------------------------------------------------------------------------------------------------------------
constexpr int MS_THREADS = 1024;

// One block. Which sorted row a pair gets inside its expert's block depends on the order in which the threads arrive; a
// row's result does not depend on where it lies.
__global__ void __launch_bounds__(MS_THREADS) moe_sort_kernel(const int* __restrict__ expert, int* __restrict__ offsets,
                                                              int* __restrict__ pos, int* __restrict__ src, int pairs, int E) {
  extern __shared__ int ms_sm[];       // [E] counts, then cursors; [E] first sorted row of each expert
  int* count = ms_sm;
  int* base = ms_sm + E;
  hb_pdl_launch();
  hb_pdl_wait();
  for (int e = threadIdx.x; e < E; e += MS_THREADS) count[e] = 0;
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += MS_THREADS) atomicAdd(&count[expert[p]], 1);
  __syncthreads();
  if (threadIdx.x == 0) {
    int run = 0;
    for (int e = 0; e < E; e++) {
      base[e] = run;
      offsets[e] = run;
      run += count[e];
      count[e] = 0;
    }
    offsets[E] = run;
  }
  __syncthreads();
  for (int p = threadIdx.x; p < pairs; p += MS_THREADS) {
    const int e = expert[p];
    const int r = base[e] + atomicAdd(&count[e], 1);
    pos[p] = r;
    src[r] = p;
  }
}

HB_EXPORT int hb_moe_sort(const int* expert, int* offsets, int* pos, int* src, int pairs, int E, cudaStream_t s) {
  if (pairs <= 0) return 0;
  const size_t smem = (size_t)2 * E * sizeof(int);
  if (smem > 40 * 1024) HB_FAIL("hb_moe_sort: %d experts are too many", E);
  hb_launch(moe_sort_kernel, dim3(1), dim3(MS_THREADS), smem, s, expert, offsets, pos, src, pairs, E);
  HB_CHECK_LAUNCH("hb_moe_sort");
  return 0;
}

template <typename TA>
__global__ void __launch_bounds__(128) moe_gather_kernel(const TA* __restrict__ xn, long ldx, const int* __restrict__ src,
                                                         TA* __restrict__ xs, int W, int top, const int* __restrict__ limit) {
  hb_pdl_launch();
  hb_pdl_wait();
  if (limit && blockIdx.x >= *limit) return;
  const int r = blockIdx.x, t = src[r] / top;
  for (int i = threadIdx.x; i < W; i += 128) xs[(size_t)r * W + i] = xn[(size_t)t * ldx + i];
}

HB_EXPORT int hb_moe_gather(const void* xn, int x_dt, long ldx, const int* src, void* xs, int pairs, int W, int top,
                            const int* limit, cudaStream_t s) {
  if (pairs <= 0) return 0;
  HB_DISPATCH_1(x_dt, "hb_moe_gather",
                (hb_launch(moe_gather_kernel<TA>, dim3(pairs), dim3(128), 0, s, (const TA*)xn, ldx, src, (TA*)xs, W, top, limit)));
  HB_CHECK_LAUNCH("hb_moe_gather");
  return 0;
}

// gu [rows][g (F) | u (F)] 32-bit, sorted rows; the pair's score enters here
template <typename TO>
__global__ void __launch_bounds__(256) moe_act_kernel(const float* __restrict__ gu, const int* __restrict__ src,
                                                      const float* __restrict__ weight, TO* __restrict__ act, long n, int F,
                                                      int at_output, const int* __restrict__ limit, int grp) {
  hb_pdl_launch();
  hb_pdl_wait();
  if (limit) n = (long)*limit * F;
  for (long idx = (long)blockIdx.x * 256 + threadIdx.x; idx < n; idx += (long)gridDim.x * 256) {
    const long r = idx / F;
    const int j = (int)(idx - r * F);
    const float sw = weight[src[r]];
    const float s = at_output ? 1.f : sw, so = at_output ? sw : 1.f;
    const float* gr = gu + r * 2 * F + moe_gate_row(j, grp);
    const float g = s * gr[0], u = s * gr[grp];
    act[idx] = hb_from_float<TO>(g / (1.f + expf(-g)) * u * so);
  }
}

// Four columns a thread (F a multiple of four, aligned rows): the same values.
template <typename TO>
__global__ void __launch_bounds__(256) moe_act_vec_kernel(const float* __restrict__ gu, const int* __restrict__ src,
                                                          const float* __restrict__ weight, TO* __restrict__ act, long n4, int F,
                                                          int at_output, const int* __restrict__ limit, int grp) {
  hb_pdl_launch();
  hb_pdl_wait();
  const int F4 = F >> 2;
  if (limit) n4 = (long)*limit * F4;
  for (long idx = (long)blockIdx.x * 256 + threadIdx.x; idx < n4; idx += (long)gridDim.x * 256) {
    const long r = idx / F4;
    const int j = (int)(idx - r * F4) << 2;
    const float sw = weight[src[r]];
    const float s = at_output ? 1.f : sw, so = at_output ? sw : 1.f;
    const float* gr = gu + r * 2 * F + moe_gate_row(j, grp);
    const float4 gv = *(const float4*)gr, uv = *(const float4*)(gr + grp);
    const float g0 = s * gv.x, g1 = s * gv.y, g2 = s * gv.z, g3 = s * gv.w;
    hb_store4(act + r * F + j, make_float4(g0 / (1.f + expf(-g0)) * (s * uv.x) * so, g1 / (1.f + expf(-g1)) * (s * uv.y) * so,
                                           g2 / (1.f + expf(-g2)) * (s * uv.z) * so, g3 / (1.f + expf(-g3)) * (s * uv.w) * so));
  }
}

HB_EXPORT int hb_moe_act(const float* gu, const int* src, const float* weight, void* act, int o_dt, int pairs, int F,
                         int at_output, const int* limit, int grp, cudaStream_t s) {
  if (pairs <= 0) return 0;
  if (grp < 1 || F % grp) HB_FAIL("hb_moe_act: %d hidden rows in groups of %d", F, grp);
  if (F % 4 == 0 && grp % 4 == 0 && !(((uintptr_t)gu | (uintptr_t)act) & 15)) {
    const long n4 = (long)pairs * (F / 4);
    const int blocks4 = (int)((n4 + 255) / 256 < 148 * 16 ? (n4 + 255) / 256 : 148 * 16);
    HB_DISPATCH_1(o_dt, "hb_moe_act",
                  (hb_launch(moe_act_vec_kernel<TA>, dim3(blocks4), dim3(256), 0, s, gu, src, weight, (TA*)act, n4, F, at_output, limit, grp)));
    HB_CHECK_LAUNCH("hb_moe_act");
    return 0;
  }
  const long n = (long)pairs * F;
  const int blocks = (int)((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16);
  HB_DISPATCH_1(o_dt, "hb_moe_act", (hb_launch(moe_act_kernel<TA>, dim3(blocks), dim3(256), 0, s, gu, src, weight, (TA*)act, n, F, at_output, limit, grp)));
  HB_CHECK_LAUNCH("hb_moe_act");
  return 0;
}

template <typename TA>
__global__ void __launch_bounds__(256) moe_combine_kernel(const float* __restrict__ ys, const int* __restrict__ pos,
                                                          float* __restrict__ y, long ldy, long n, int W, int top,
                                                          const int* __restrict__ limit, const TA* __restrict__ xn, long ldx,
                                                          const float* __restrict__ identity_weight) {
  hb_pdl_launch();
  hb_pdl_wait();
  const int lim = limit ? *limit : 0x7fffffff;
  for (long idx = (long)blockIdx.x * 256 + threadIdx.x; idx < n; idx += (long)gridDim.x * 256) {
    const long t = idx / W;
    const int c = (int)(idx - t * W);
    float acc = 0.f;
    for (int k = 0; k < top; k++) {
      const int p = pos[t * top + k];
      if (p < lim) acc += ys[(size_t)p * W + c];
    }
    if (identity_weight) acc = fmaf(identity_weight[t], hb_to_float(xn[t * ldx + c]), acc);
    y[t * ldy + c] += acc;
  }
}

// Four columns a thread: the same sums.
template <typename TA>
__global__ void __launch_bounds__(256) moe_combine_vec_kernel(const float* __restrict__ ys, const int* __restrict__ pos,
                                                              float* __restrict__ y, long ldy, long n4, int W4, int top,
                                                              const int* __restrict__ limit, const TA* __restrict__ xn, long ldx,
                                                              const float* __restrict__ identity_weight) {
  hb_pdl_launch();
  hb_pdl_wait();
  const int lim = limit ? *limit : 0x7fffffff;
  for (long idx = (long)blockIdx.x * 256 + threadIdx.x; idx < n4; idx += (long)gridDim.x * 256) {
    const long t = idx / W4;
    const int c = (int)(idx - t * W4) * 4;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int k = 0; k < top; k++) {
      const int p = pos[t * top + k];
      if (p >= lim) continue;
      const float4 v = hb_load4(ys + (size_t)p * W4 * 4 + c);
      acc.x += v.x; acc.y += v.y; acc.z += v.z; acc.w += v.w;
    }
    if (identity_weight) {
      const float w = identity_weight[t];
      const float4 v = hb_load4(xn + t * ldx + c);
      acc.x = fmaf(w, v.x, acc.x); acc.y = fmaf(w, v.y, acc.y); acc.z = fmaf(w, v.z, acc.z); acc.w = fmaf(w, v.w, acc.w);
    }
    float4 o = hb_load4(y + t * ldy + c);
    o.x += acc.x; o.y += acc.y; o.z += acc.z; o.w += acc.w;
    hb_store4(y + t * ldy + c, o);
  }
}

// limit (or null): sorted rows from *limit on belong to identity experts and hold nothing; y also gets identity_weight[t] xn[t].
HB_EXPORT int hb_moe_combine(const float* ys, const int* pos, float* y, long ldy, int T, int W, int top, const int* limit,
                             const void* xn, int x_dt, long ldx, const float* identity_weight, cudaStream_t s) {
  if (T <= 0) return 0;
  if (identity_weight && !xn) HB_FAIL("hb_moe_combine: identity experts need their input rows");
  if (W % 4 == 0 && ldy % 4 == 0 && ldx % 4 == 0 && !(((uintptr_t)ys | (uintptr_t)y | (uintptr_t)xn) & 15)) {
    const long n4 = (long)T * (W / 4);
    const int blocks4 = (int)((n4 + 255) / 256 < 148 * 16 ? (n4 + 255) / 256 : 148 * 16);
    HB_DISPATCH_1(x_dt, "hb_moe_combine",
                  (hb_launch(moe_combine_vec_kernel<TA>, dim3(blocks4), dim3(256), 0, s, ys, pos, y, ldy, n4, W / 4, top, limit,
                             (const TA*)xn, ldx, identity_weight)));
    HB_CHECK_LAUNCH("hb_moe_combine");
    return 0;
  }
  const long n = (long)T * W;
  const int blocks = (int)((n + 255) / 256 < 148 * 16 ? (n + 255) / 256 : 148 * 16);
  HB_DISPATCH_1(x_dt, "hb_moe_combine",
                (hb_launch(moe_combine_kernel<TA>, dim3(blocks), dim3(256), 0, s, ys, pos, y, ldy, n, W, top, limit, (const TA*)xn, ldx,
                           identity_weight)));
  HB_CHECK_LAUNCH("hb_moe_combine");
  return 0;
}
