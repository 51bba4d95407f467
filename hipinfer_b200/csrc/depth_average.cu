// The residual row after a sublayer whose RESULT is normed, in one pass: with y (or ca ya + cb yb, two side-by-side results),
//     x' = x + (y - mean y) / sqrt(mean (y - mean y)^2 + eps) * w + bias        (an RMS norm: without the mean)
// and, at the end of a layer of a model that averages over its depth, what goes on to the next layer,
//     x'' = sum_j c[j] X_j + c[n] x',   X_0 .. X_(n-1) the kept states of earlier layers, x' kept as X_n.
// Everything is 32-bit; the rounded copy for the next products is made on the way out. A block a row.
#include "common.cuh"

struct DepthArgs {
  const float* x; const float* ya; const float* yb;      // yb null: y = ca ya
  float ca, cb;
  const void* w; const void* bias; float eps; int center; // bias null: none; center 0: an RMS norm
  float* x_out; void* rounded;                           // rounded null: none
  float* keep_in; float* keep;                           // copies of x and of x' (null: none)
  const float* states; long state_stride;                // X_0, X_1, ... [.][T][W] (null: no average)
  const float* coef; int n_states;                       // c[0 .. n_states]
  int W;
};

template <typename TW, typename TO>
__global__ void __launch_bounds__(256) output_norm_kernel(DepthArgs A) {
  extern __shared__ float on_row[];      // [W], then 32 floats for the sums
  hb_pdl_launch();
  hb_pdl_wait();
  float* red = on_row + A.W;
  const int W = A.W;
  const size_t base = (size_t)blockIdx.x * W;
  const TW* w = (const TW*)A.w;
  const TW* bi = (const TW*)A.bias;
  float s = 0.f;
  for (int i = threadIdx.x; i < W; i += 256) {
    const float v = A.yb ? fmaf(A.ca, A.ya[base + i], A.cb * A.yb[base + i]) : A.ca * A.ya[base + i];
    on_row[i] = v;
    s += v;
  }
  const float mean = A.center ? hb_block_sum(s, red) / (float)W : 0.f;
  float ss = 0.f;
  for (int i = threadIdx.x; i < W; i += 256) {
    const float d = on_row[i] - mean;
    ss = fmaf(d, d, ss);
  }
  const float f = rsqrtf(hb_block_sum(ss, red) / (float)W + A.eps);
  for (int i = threadIdx.x; i < W; i += 256) {
    const float xi = A.x[base + i];
    float v = xi + ((on_row[i] - mean) * f * hb_to_float(w[i]) + (bi ? hb_to_float(bi[i]) : 0.f));
    if (A.keep_in) A.keep_in[base + i] = xi;
    if (A.keep) A.keep[base + i] = v;
    if (A.states) {
      float acc = 0.f;
      for (int j = 0; j < A.n_states; j++) {
        const float sj = (A.keep_in && j == 0) ? xi : A.states[j * A.state_stride + base + i];
        acc = fmaf(A.coef[j], sj, acc);
      }
      v = fmaf(A.coef[A.n_states], v, acc);
    }
    A.x_out[base + i] = v;
    if (A.rounded) ((TO*)A.rounded)[base + i] = hb_from_float<TO>(v);
  }
}

__device__ __forceinline__ float4 dp_fma(float c, float4 a, float4 b) {
  return make_float4(fmaf(c, a.x, b.x), fmaf(c, a.y, b.y), fmaf(c, a.z, b.z), fmaf(c, a.w, b.w));
}

// Four columns a load, the row in registers; the kept states are summed before the norm's barriers, all loads in flight.
template <typename TW, typename TO, int NV>
__global__ void __launch_bounds__(256) output_norm_vec_kernel(DepthArgs A) {
  __shared__ float red[32];
  hb_pdl_launch();
  hb_pdl_wait();
  const int W = A.W;
  const size_t base = (size_t)blockIdx.x * W;
  const TW* w = (const TW*)A.w;
  const TW* bi = (const TW*)A.bias;
  float4 y[NV], x[NV], acc[NV];
  float s = 0.f;
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = (v * 256 + threadIdx.x) * 4;
    y[v] = x[v] = acc[v] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < W) {
      x[v] = hb_load4(A.x + base + c);
      const float4 ya = hb_load4(A.ya + base + c);
      y[v] = make_float4(A.ca * ya.x, A.ca * ya.y, A.ca * ya.z, A.ca * ya.w);
      if (A.yb) y[v] = dp_fma(A.cb, hb_load4(A.yb + base + c), y[v]);
      s += (y[v].x + y[v].y) + (y[v].z + y[v].w);
    }
  }
  if (A.states) {
    int j0 = 0;
    if (A.keep_in) {                     // X_0 is x itself
      j0 = 1;
      const float c0 = A.coef[0];
#pragma unroll
      for (int v = 0; v < NV; v++) acc[v] = dp_fma(c0, x[v], acc[v]);
    }
#pragma unroll 4
    for (int j = j0; j < A.n_states; j++) {
      const float cj = A.coef[j];
      const float* sj = A.states + j * A.state_stride + base;
#pragma unroll
      for (int v = 0; v < NV; v++) {
        const int c = (v * 256 + threadIdx.x) * 4;
        if (c < W) acc[v] = dp_fma(cj, hb_load4(sj + c), acc[v]);
      }
    }
  }
  const float mean = A.center ? hb_block_sum(s, red) / (float)W : 0.f;
  float ss = 0.f;
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = (v * 256 + threadIdx.x) * 4;
    if (c < W) {
      y[v].x -= mean; y[v].y -= mean; y[v].z -= mean; y[v].w -= mean;
      ss = fmaf(y[v].x, y[v].x, ss); ss = fmaf(y[v].y, y[v].y, ss); ss = fmaf(y[v].z, y[v].z, ss); ss = fmaf(y[v].w, y[v].w, ss);
    }
  }
  const float f = rsqrtf(hb_block_sum(ss, red) / (float)W + A.eps);
  const float cn = A.states ? A.coef[A.n_states] : 0.f;
#pragma unroll
  for (int v = 0; v < NV; v++) {
    const int c = (v * 256 + threadIdx.x) * 4;
    if (c < W) {
      const float4 wv = hb_load4(w + c), bv = bi ? hb_load4(bi + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      float4 o = make_float4(x[v].x + fmaf(y[v].x * f, wv.x, bv.x), x[v].y + fmaf(y[v].y * f, wv.y, bv.y),
                             x[v].z + fmaf(y[v].z * f, wv.z, bv.z), x[v].w + fmaf(y[v].w * f, wv.w, bv.w));
      if (A.keep_in) hb_store4(A.keep_in + base + c, x[v]);
      if (A.keep) hb_store4(A.keep + base + c, o);
      if (A.states) o = dp_fma(cn, o, acc[v]);
      hb_store4(A.x_out + base + c, o);
      if (A.rounded) hb_store4((TO*)A.rounded + base + c, o);
    }
  }
}

HB_EXPORT int hb_output_norm(const float* x, const float* ya, const float* yb, float ca, float cb, const void* w, const void* bias,
                             int w_dt, float eps, int center, float* x_out, void* rounded, int r_dt, float* keep_in, float* keep,
                             const float* states, long state_stride, const float* coef, int n_states, int T, int W, cudaStream_t s) {
  if (T <= 0) return 0;
  if (states && (!coef || n_states < 1)) HB_FAIL("hb_output_norm: an average over %d states", n_states);
  DepthArgs A;
  A.x = x; A.ya = ya; A.yb = yb; A.ca = ca; A.cb = cb; A.w = w; A.bias = bias; A.eps = eps; A.center = center; A.x_out = x_out; A.rounded = rounded;
  A.keep_in = keep_in; A.keep = keep; A.states = states; A.state_stride = state_stride; A.coef = coef; A.n_states = n_states; A.W = W;
  if (!rounded) r_dt = HB_F32;
  const uintptr_t all = (uintptr_t)x | (uintptr_t)ya | (uintptr_t)yb | (uintptr_t)w | (uintptr_t)bias | (uintptr_t)x_out |
                        (uintptr_t)rounded | (uintptr_t)keep_in | (uintptr_t)keep | (uintptr_t)states;
  if (W % 4 == 0 && W <= 8192 && !(all & 15) && (state_stride & 3) == 0) {
#define ON_LAUNCH(NV)                                                                                                    \
  HB_DISPATCH_2(w_dt, r_dt, "hb_output_norm", (hb_launch(output_norm_vec_kernel<TA, TB, NV>, dim3(T), dim3(256), 0, s, A)))
    if (W <= 1024) ON_LAUNCH(1);
    else if (W <= 2048) ON_LAUNCH(2);
    else if (W <= 4096) ON_LAUNCH(4);
    else ON_LAUNCH(8);
#undef ON_LAUNCH
  } else {
    const size_t smem = (size_t)(W + 32) * sizeof(float);
    if (smem > 200 * 1024) HB_FAIL("hb_output_norm: a row of %d does not fit shared memory", W);
    HB_DISPATCH_2(w_dt, r_dt, "hb_output_norm", do {
      auto kern = output_norm_kernel<TA, TB>;
      if (smem > 40 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      hb_launch(kern, dim3(T), dim3(256), smem, s, A);
    } while (0));
  }
  HB_CHECK_LAUNCH("hb_output_norm");
  return 0;
}
