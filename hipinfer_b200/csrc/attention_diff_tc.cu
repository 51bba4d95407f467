// Flash attention of prompt portions with TWO score maps per head (differential attention) on the 5th-generation tensor
// cores, causal or with a sliding window, over the paged bf16 cache.
//
// One CTA = 128 consecutive query rows of one request and one query head, BOTH maps: a key tile (128 ABSOLUTE positions, its
// two maps side by side in a key row) and its values are loaded once for both. Ten warps:
//   warps 0-3, 4-7       softmax of map 0 and of map 1: a thread owns one query row of its map. It reads its row of S from
//                        tensor memory in one go, masks on absolute positions, exponentiates in the exp2 domain in fp32 and
//                        writes P as bf16 into shared memory in the layout the tensor core reads. The map's output row stays
//                        in tensor memory over all the tiles, in units of 2^m, where m follows the row's maximum lazily (only
//                        a maximum that exceeds m by more than 8 raises it and has the row rescaled);
//   warp 8 (one thread a page)  TMA: the Q tile once, then per tile the K pages and the V pages (no multicast);
//   warp 9 (one thread)  tcgen05.mma: S_m = Q_m K_m^T of both maps, and, once the softmax warps have written P_m, O_m += P_m V.
// At the end o = O_0 / l_0 - lambda O_1 / l_1 per row, two threads a row (half of the columns each, the maps' sums and the
// halves' sums of squares exchanged through shared memory), divided by its root mean square, times `post`, times
// sigmoid(gate), rounded once. Tensor memory: S 2 x 128 columns, O 2 x E. The counterpart of attn_window_flash_kernel (warp
// MMAs), which takes other sizes and windows that keep the first tokens. Tiles are cut at absolute positions and a row's
// maximum and sum are its own: a row's result does not depend on how the prompt was cut or on the batch. Waits are bounded.
#include "tc_common.cuh"

constexpr int DT_BM = 128, DT_BN = 128, DT_TILE = 128 * 64 * 2, DT_THREADS = 320;

__device__ __forceinline__ uint64_t dt_desc_mn128(uint32_t smem_addr) {   // MN-major, 128-byte swizzle, the next 64 columns DT_TILE on
  return (uint64_t)((smem_addr & 0x3FFFFu) >> 4) | ((uint64_t)(DT_TILE >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) |
         ((uint64_t)1 << 46) | ((uint64_t)2 << 61);
}

struct DtBars {
  uint64_t q_full, k_full[2], k_free[2], v_full[2], v_free[2];
  uint64_t s_full[2], s_free[2], o_full[2], p_full[2], p_free[2];     // per map
  float part[2][128];            // per map the row sums' reciprocals, then per half the sums of squares
  uint32_t tmem_slot;
  int abort_flag;
};

struct DtArgs {
  const int* bt;
  int bt_stride;
  const int* q_start;
  const int* q_len;
  const int* ctx_len;
  const float* gate;         // [T][ld_gate] at column gate_off, or null
  long ld_gate;
  int gate_off;
  __nv_bfloat16* out;        // [T][H][E]
  int H, G, page_size, window, min_rows;
  float scale_log2, lambda, post, eps;
  int* status;
};

template <int D, int E>
__global__ void __launch_bounds__(DT_THREADS, 1) flash_diff_tc_kernel(const __grid_constant__ CUtensorMap map_q,
                                                                      const __grid_constant__ CUtensorMap map_k,
                                                                      const __grid_constant__ CUtensorMap map_v, DtArgs A) {
  constexpr int NQ = 2 * D / 64, NV = E / 64, KB = NQ * DT_TILE, VB = NV * DT_TILE;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t* sQ = smem;                  // [128][2 D]
  uint8_t* sK = sQ + KB;               // two stages of [128 keys][2 D]
  uint8_t* sV = sK + 2 * KB;           // two stages of [128 keys][E]
  uint8_t* sP = sV + 2 * VB;           // per map two K blocks of [128 rows][64 keys]
  DtBars* bar = (DtBars*)(sP + 4 * DT_TILE);
  volatile int* abort_flag = &bar->abort_flag;

  const int req = blockIdx.z, hq = blockIdx.x, qt = gridDim.y - 1 - blockIdx.y;     // heaviest query tiles first
  hb_pdl_launch();
  const int n_rows = A.q_len[req];
  if (n_rows < A.min_rows || qt * DT_BM >= n_rows) {
    if ((blockIdx.x | blockIdx.y | blockIdx.z) == 0) hb_pdl_wait();   // the grid never ends before the one ahead of it
    return;
  }
  if (hb_smem_u32(smem) & 1023) {   // never seen; the tiles would not be where the tensor core expects them
    if (threadIdx.x == 0) atomicExch(A.status, 1);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = hq / (A.H / A.G), ps = A.page_size, window = A.window;
  const int row0 = A.q_start[req] + qt * DT_BM, rows_here = min(DT_BM, n_rows - qt * DT_BM);
  const int p_first = A.ctx_len[req] + qt * DT_BM, p_last = p_first + rows_here - 1;
  const int lo = window > 0 ? max(0, p_first - window + 1) : 0;
  const int kt_lo = lo / DT_BN, n_tiles = p_last / DT_BN - kt_lo + 1;
  const int* table = A.bt + (size_t)req * A.bt_stride;

  if (threadIdx.x == 0) {
    hb_mbar_init(&bar->q_full, 1);
    for (int b = 0; b < 2; b++) {
      hb_mbar_init(&bar->k_full[b], 1); hb_mbar_init(&bar->k_free[b], 1);
      hb_mbar_init(&bar->v_full[b], 1); hb_mbar_init(&bar->v_free[b], 1);
      hb_mbar_init(&bar->s_full[b], 1); hb_mbar_init(&bar->s_free[b], 128);
      hb_mbar_init(&bar->o_full[b], 1);
      hb_mbar_init(&bar->p_full[b], 128); hb_mbar_init(&bar->p_free[b], 1);
    }
    bar->abort_flag = 0;
    hb_fence_barrier_init();
  }
  // keys of a ragged tile that are never loaded: what the tensor core reads in their place must be finite
  for (int i = threadIdx.x; i < 2 * (KB + VB) / 16; i += DT_THREADS) ((uint4*)sK)[i] = make_uint4(0, 0, 0, 0);
  if (warp == 8 && lane == 0) { hb_tma_prefetch_desc(&map_q); hb_tma_prefetch_desc(&map_k); hb_tma_prefetch_desc(&map_v); }
  hb_fence_proxy_async();
  hb_pdl_wait();   // barriers and shared memory were set up while the kernel ahead was still running
  // all of the tensor memory: taken only now that no kernel ahead can still be about to ask for some of it
  if (warp == 9) {
    hb_tmem_alloc(&bar->tmem_slot, 512);
    hb_tmem_relinquish();
  }
  hb_tc_fence_before();
  __syncthreads();
  hb_tc_fence_after();
  const uint32_t tmem = bar->tmem_slot;         // S of map m at column 128 m, O of map m at 256 + E m

  if (warp == 8) {  // ---------------- TMA: lane l brings page l of the tile
    if (lane == 0) {
      hb_mbar_expect_tx(&bar->q_full, KB);
#pragma unroll
      for (int t = 0; t < NQ; t++) hb_tma_load_2d(sQ + t * DT_TILE, &map_q, &bar->q_full, hq * 2 * D + t * 64, row0);
    }
    for (int i = 0; i < n_tiles; i++) {
      const int k_base = (kt_lo + i) * DT_BN, b = i & 1, free_phase = ((i >> 1) & 1) ^ 1;
      const int first_page = max(k_base, lo) / ps, np = min(k_base + DT_BN - 1, p_last) / ps - first_page + 1;
      const int pg = first_page + lane;
      const int row = lane < np ? (table[pg] * A.G + h) * ps : 0;
      const int off = (pg * ps - k_base) * 128;                    // rows of 128 bytes in each 64-column tile
      int ok = 1;
      if (lane == 0) {
        ok = hb_mbar_wait(&bar->k_free[b], free_phase, abort_flag);
        if (ok) hb_mbar_expect_tx(&bar->k_full[b], (uint32_t)(np * ps * 2 * D * 2));
      }
      if (!__shfl_sync(0xffffffffu, ok, 0)) break;
      if (lane < np) {
#pragma unroll
        for (int t = 0; t < NQ; t++) hb_tma_load_2d(sK + b * KB + t * DT_TILE + off, &map_k, &bar->k_full[b], t * 64, row);
      }
      if (lane == 0) {
        ok = hb_mbar_wait(&bar->v_free[b], free_phase, abort_flag);
        if (ok) hb_mbar_expect_tx(&bar->v_full[b], (uint32_t)(np * ps * E * 2));
      }
      if (!__shfl_sync(0xffffffffu, ok, 0)) break;
      if (lane < np) {
#pragma unroll
        for (int t = 0; t < NV; t++) hb_tma_load_2d(sV + b * VB + t * DT_TILE + off, &map_v, &bar->v_full[b], t * 64, row);
      }
    }
  } else if (warp == 9) {
    if (lane == 0) {  // ---------------- tensor cores: both S_i are issued before the O_{i-1}, so they overlap the softmax of tile i - 1
      constexpr uint32_t idesc_s = hb_umma_idesc_bf16(DT_BM, DT_BN), idesc_o = hb_umma_idesc_bf16(DT_BM, E) | (1u << 16);   // B of O MN-major
      bool ok = hb_mbar_wait(&bar->q_full, 0, abort_flag);
      for (int i = 0; i <= n_tiles && ok; i++) {
        if (i < n_tiles) {
          const int b = i & 1;
          if (!hb_mbar_wait(&bar->k_full[b], (i >> 1) & 1, abort_flag)) break;
          for (int m = 0; m < 2 && ok; m++) {
            ok = hb_mbar_wait(&bar->s_free[m], (i & 1) ^ 1, abort_flag);
            if (!ok) break;
            hb_tc_fence_after();
#pragma unroll
            for (int k = 0; k < D / 16; k++) {
              const int kk = m * (D / 16) + k;                     // 16 columns a step, four steps in each 64-column tile
              const uint64_t dq = hb_umma_desc_k128(hb_smem_u32(sQ + (kk >> 2) * DT_TILE)) + 2 * (kk & 3);
              const uint64_t dk = hb_umma_desc_k128(hb_smem_u32(sK + b * KB + (kk >> 2) * DT_TILE)) + 2 * (kk & 3);
              hb_umma_bf16(tmem + m * DT_BN, dq, dk, idesc_s, k != 0);
            }
            hb_umma_commit(&bar->s_full[m]);
          }
          if (!ok) break;
          hb_umma_commit(&bar->k_free[b]);
        }
        if (i > 0) {
          const int j = i - 1, b = j & 1;
          if (!hb_mbar_wait(&bar->v_full[b], (j >> 1) & 1, abort_flag)) break;
          for (int m = 0; m < 2 && ok; m++) {
            ok = hb_mbar_wait(&bar->p_full[m], j & 1, abort_flag);
            if (!ok) break;
            hb_tc_fence_after();
#pragma unroll
            for (int k = 0; k < DT_BN / 16; k++) {
              const uint64_t dp = hb_umma_desc_k128(hb_smem_u32(sP + (2 * m + (k >> 2)) * DT_TILE)) + 2 * (k & 3);
              const uint64_t dv = dt_desc_mn128(hb_smem_u32(sV + b * VB + k * 16 * 128));
              hb_umma_bf16(tmem + 2 * DT_BN + m * E, dp, dv, idesc_o, j != 0 || k != 0);
            }
            hb_umma_commit(&bar->o_full[m]);
            hb_umma_commit(&bar->p_free[m]);
          }
          if (!ok) break;
          hb_umma_commit(&bar->v_free[b]);
        }
      }
    }
  } else {  // ---------------- softmax: thread = (map, query row)
    const int m = warp >> 2, r = (warp & 3) * 32 + lane;
    const int qp = p_first + min(r, rows_here - 1);  // rows past the portion's end are computed, never stored
    const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
    const uint32_t tmem_s = tmem + m * DT_BN + lane_base, tmem_o = tmem + 2 * DT_BN + m * E + lane_base;
    const uint32_t p_row = hb_smem_u32(sP + 2 * m * DT_TILE) + r * 128;
    constexpr float SLACK = 8.f;
    const float scale_log2 = A.scale_log2;
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;   // every wait's outcome is made uniform over the warp: the tensor-memory accesses below are warp-wide
    for (int i = 0; i < n_tiles && ok; i++) {
      const int k_base = (kt_lo + i) * DT_BN;
      const bool need_mask = k_base + DT_BN - 1 > p_first || (window > 0 && k_base < p_last - window + 1);
      if (!__all_sync(0xffffffffu, hb_mbar_wait(&bar->s_full[m], i & 1, abort_flag))) { ok = false; break; }
      hb_tc_fence_after();
      uint32_t s[2][64];
      hb_tmem_ld64_nowait(tmem_s, s[0]);
      hb_tmem_ld64_nowait(tmem_s + 64, s[1]);
      hb_tmem_ld_wait();
      hb_tmem_ld_fence64(s[0]);
      hb_tmem_ld_fence64(s[1]);
      hb_tc_fence_before();
      hb_mbar_arrive(&bar->s_free[m]);       // the scores of the next tile may overwrite S
      const int hi_j = qp - k_base, lo_j = window > 0 ? qp - window - k_base : -1;  // key j of the tile is visible iff lo_j < j <= hi_j
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      if (need_mask) {
#pragma unroll
        for (int j = 0; j < 128; j++) {
          const float v = (j <= hi_j && j > lo_j) ? __uint_as_float(s[j >> 6][j & 63]) : -INFINITY;
          s[j >> 6][j & 63] = __float_as_uint(v);
          mx4[j & 3] = fmaxf(mx4[j & 3], v);
        }
      } else {
#pragma unroll
        for (int j = 0; j < 128; j++) mx4[j & 3] = fmaxf(mx4[j & 3], __uint_as_float(s[j >> 6][j & 63]));
      }
      const float m_tile = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * scale_log2;
      const bool grow = m_tile > m_run + SLACK;   // also the first tile with a visible key: m_run is -inf
      float corr = 1.f;
      if (grow) {
        corr = hb_exp2(m_run - m_tile);   // 0 while nothing has been summed
        m_run = m_tile;
      }
      const float sub = m_run == -INFINITY ? 0.f : m_run;
      float sum4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int hh = 0; hh < 2; hh++) {
#pragma unroll
        for (int j = 0; j < 64; j += 2) {  // masked scores are -inf: 2^-inf = 0
          const float p0 = hb_exp2(fmaf(__uint_as_float(s[hh][j]), scale_log2, -sub));
          const float p1 = hb_exp2(fmaf(__uint_as_float(s[hh][j + 1]), scale_log2, -sub));
          sum4[(j >> 1) & 3] += p0 + p1;
          s[hh][j >> 1] = hb_pack_bf16(p0, p1);
        }
        if (hh == 0 && !__all_sync(0xffffffffu, hb_mbar_wait(&bar->p_free[m], (i & 1) ^ 1, abort_flag))) { ok = false; break; }
#pragma unroll
        for (int cc = 0; cc < 8; cc++)   // 64 keys = eight 16-byte chunks of this row in K block hh of P
          asm volatile("st.shared.v4.u32 [%0], {%1, %2, %3, %4};" ::"r"(p_row + hh * DT_TILE + ((cc ^ (r & 7)) << 4)), "r"(s[hh][4 * cc]),
                       "r"(s[hh][4 * cc + 1]), "r"(s[hh][4 * cc + 2]), "r"(s[hh][4 * cc + 3]) : "memory");
      }
      if (!ok) break;
      l_run = l_run * corr + ((sum4[0] + sum4[1]) + (sum4[2] + sum4[3]));
      // a raised maximum: the rows of O so far, which the product of the tile before has to have finished writing
      if (i > 0 && __any_sync(0xffffffffu, grow)) {
        if (!__all_sync(0xffffffffu, hb_mbar_wait(&bar->o_full[m], (i - 1) & 1, abort_flag))) { ok = false; break; }
        hb_tc_fence_after();
#pragma unroll
        for (int t = 0; t < NV; t++) {
          uint32_t o[64];
          hb_tmem_ld64_nowait(tmem_o + t * 64, o);
          hb_tmem_ld_wait();
          hb_tmem_ld_fence64(o);
#pragma unroll
          for (int d = 0; d < 64; d++) o[d] = __float_as_uint(__uint_as_float(o[d]) * corr);
          hb_tmem_st64(tmem_o + t * 64, o);
        }
        hb_tmem_st_wait();
      }
      hb_tc_fence_before();
      hb_fence_proxy_async();
      hb_mbar_arrive(&bar->p_full[m]);
    }
    // the last product of this map; behind the barrier both maps' are done, and this thread combines half of its row's columns
    if (ok) ok = __all_sync(0xffffffffu, hb_mbar_wait(&bar->o_full[m], (n_tiles - 1) & 1, abort_flag));
    bar->part[m][r] = 1.f / l_run;
    hb_tc_fence_before();
    asm volatile("bar.sync 1, 256;" ::: "memory");          // (the softmax warps alone; all of them come here whatever their waits gave)
    const float i0 = bar->part[0][r], i1 = A.lambda * bar->part[1][r];
    asm volatile("bar.sync 1, 256;" ::: "memory");
    constexpr int EH = E / 2;
    float o[EH];
    float ss = 0.f;
    if (ok) {
      hb_tc_fence_after();
#pragma unroll
      for (int t = 0; t < EH / 32; t++) {
        float a[32], b[32];
        hb_tmem_ld32(tmem + 2 * DT_BN + m * EH + t * 32 + lane_base, a);
        hb_tmem_ld32(tmem + 2 * DT_BN + E + m * EH + t * 32 + lane_base, b);
#pragma unroll
        for (int d = 0; d < 32; d++) {
          const float v = a[d] * i0 - i1 * b[d];
          o[t * 32 + d] = v;
          ss = fmaf(v, v, ss);
        }
      }
    }
    bar->part[m][r] = ss;
    asm volatile("bar.sync 1, 256;" ::: "memory");
    if (ok && r < rows_here) {
      const float f = rsqrtf((bar->part[0][r] + bar->part[1][r]) / (float)E + A.eps) * A.post;
      __nv_bfloat16* dst = A.out + ((size_t)(row0 + r) * A.H + hq) * E + m * EH;
      const float* gp = A.gate ? A.gate + (size_t)(row0 + r) * A.ld_gate + A.gate_off + hq * E + m * EH : nullptr;
#pragma unroll
      for (int d = 0; d < EH; d += 8) {
        float y[8];
#pragma unroll
        for (int e = 0; e < 8; e++) y[e] = o[d + e] * f;
        if (gp) {
#pragma unroll
          for (int e = 0; e < 8; e += 2) {
            const float2 g = *(const float2*)(gp + d + e);
            y[e] *= 1.f / (1.f + expf(-g.x));
            y[e + 1] *= 1.f / (1.f + expf(-g.y));
          }
        }
        *(uint4*)(dst + d) = make_uint4(hb_pack_bf16(y[0], y[1]), hb_pack_bf16(y[2], y[3]), hb_pack_bf16(y[4], y[5]), hb_pack_bf16(y[6], y[7]));
      }
    }
  }

  hb_tc_fence_before();
  __syncthreads();
  if (*abort_flag) {
    if (threadIdx.x == 0) atomicExch(A.status, 1);
    __nanosleep(100000);
  }
  if (warp == 9) {
    __syncwarp();
    hb_tmem_dealloc(tmem, 512);
  }
}

HB_EXPORT int hb_flash_diff_tc_supported(int H, int G, int D, int E, int page_size) {
  return G > 0 && H % G == 0 && (D == 32 || D == 64) && (E == 64 || E == 128) && page_size >= 8 && page_size <= DT_BN &&
         (page_size & (page_size - 1)) == 0;
}

template <int D, int E>
static int dt_launch(const CUtensorMap& mq, const CUtensorMap& mk, const CUtensorMap& mv, const DtArgs& A, dim3 grid, cudaStream_t s) {
  const size_t smem = (size_t)DT_TILE * (3 * (2 * D / 64) + 2 * (E / 64) + 4) + sizeof(DtBars);
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(flash_diff_tc_kernel<D, E>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) HB_FAIL("hb_flash_diff_tc: %s", cudaGetErrorString(e));
    configured = true;
  }
  cudaError_t e = hb_launch(flash_diff_tc_kernel<D, E>, grid, DT_THREADS, smem, s, mq, mk, mv, A);
  if (e != cudaSuccess) HB_FAIL("hb_flash_diff_tc: %s", cudaGetErrorString(e));
  return 0;
}

// q [T, H, 2 D], out [T, H, E] bf16; planes [num_pages, G, page_size, 2 D] and [..., E] bf16; per request q_start, q_len, ctx_len
// and a block table row. window 0: every earlier key. Requests with fewer than min_rows rows are skipped. `status` is set to 1
// if a bounded wait ran out.
HB_EXPORT int hb_flash_diff_tc(const void* q, const void* kc, const void* vc, long num_pages, const int* bt, int bt_stride,
                               const int* q_start, const int* q_len, const int* ctx_len, const float* gate, long ld_gate, int gate_off,
                               void* out, int T, int R, int max_q_len, int H, int G, int D, int E, int page_size, int window, float scale,
                               float lambda, float post, float eps, int min_rows, int* status, cudaStream_t s) {
  if (R <= 0 || max_q_len <= 0 || T <= 0) return 0;
  if (!hb_flash_diff_tc_supported(H, G, D, E, page_size))
    HB_FAIL("hb_flash_diff_tc: %d/%d heads of %d/%d with pages of %d are not supported", H, G, D, E, page_size);
  if (R > 65535 || max_q_len > 65535 * DT_BM) HB_FAIL("hb_flash_diff_tc: %d requests / portions of %d rows are beyond the grid limit", R, max_q_len);
  if (!status) HB_FAIL("hb_flash_diff_tc: no status word");
  if (!(scale > 0.f)) HB_FAIL("hb_flash_diff_tc: scores are scaled by a positive number");
  if (((uintptr_t)out & 15) || (gate && (((uintptr_t)gate & 7) || (ld_gate & 1) || (gate_off & 1)))) HB_FAIL("hb_flash_diff_tc: out or gate is not aligned");
  CUtensorMap mq, mk, mv;
  if (hb_make_tensor_map_bf16(&mq, q, (uint64_t)T, (uint64_t)H * 2 * D, (uint64_t)H * 2 * D, DT_BM)) return -1;
  const uint64_t rows = (uint64_t)num_pages * G * page_size;
  if (hb_make_tensor_map_bf16(&mk, kc, rows, (uint64_t)2 * D, (uint64_t)2 * D, (uint32_t)page_size)) return -1;
  if (hb_make_tensor_map_bf16(&mv, vc, rows, (uint64_t)E, (uint64_t)E, (uint32_t)page_size)) return -1;
  DtArgs A{bt, bt_stride, q_start, q_len, ctx_len, gate, ld_gate, gate_off, (__nv_bfloat16*)out, H, G, page_size, window, min_rows,
           scale * 1.4426950408889634f, lambda, post, eps, status};
  const dim3 grid(H, (max_q_len + DT_BM - 1) / DT_BM, R);
  int r;
  if (D == 32 && E == 64) r = dt_launch<32, 64>(mq, mk, mv, A, grid, s);
  else if (D == 32) r = dt_launch<32, 128>(mq, mk, mv, A, grid, s);
  else if (E == 64) r = dt_launch<64, 64>(mq, mk, mv, A, grid, s);
  else r = dt_launch<64, 128>(mq, mk, mv, A, grid, s);
  if (r) return r;
  HB_CHECK_LAUNCH("hb_flash_diff_tc");
  return 0;
}
