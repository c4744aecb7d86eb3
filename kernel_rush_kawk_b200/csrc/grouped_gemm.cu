// The routed experts' products of many rows in one launch on the 5th-generation tensor cores, the rows of an expert
// wherever the routing put their number: C[r, :] = act(A[r, :] W_e^T) for the rows r of expert e, offsets[e] <= r <
// offsets[e + 1], W [E, N, K]. GATED: W [E, 2N, K] holds every expert's gate rows and then its up rows; a block streams 128
// of either, and the epilogue reads both halves of its accumulator: C = act(g, u) with g and u multiplied by the row's weight
// first where there is one (a router that weighs an expert's input). The offsets stay on the device: the grid holds as many row tiles as the routing could need
// at most, a block finds its expert and rows by a scan over the experts' tile counts, and blocks beyond the last tile leave
// at once.
//
// The tile engine is that of gemm_tcgen05.cu: warp 0 drives TMA (128 rows of A, BN rows of W, 64 elements of K a stage,
// 128-byte swizzle), warp 1 owns tensor memory and issues tcgen05.mma, warps 2..5 read the accumulator back. With MT = 2 a
// block takes up to 256 of an expert's rows: two tiles of A ride with every tile of W into two accumulators (all 512 columns
// of tensor memory), which warps 2..5 and 6..9 read back side by side. Where experts have more than one tile of rows, W is
// then fetched once instead of twice and half as many blocks pay for their start and their epilogue. A tile of A
// that reaches past its expert's rows reads the next expert's (or zeros beyond the matrix); what it makes of them is not
// stored. Every wait is bounded: one that runs out sets the error word and the block leaves, after freeing its tensor
// memory.
#include "tcgen05.cuh"

namespace {

using namespace tc;

constexpr int BM = 128, BK = 64, UMMA_K = 16;
constexpr uint32_t A_BYTES = BM * BK * 2;

// act 0: silu(g) u of the two products as they would have been stored; act 3: clamped inputs,
// g' = min(g, limit), u' = clamp(u, -limit, limit), g' sigmoid(slope g') (u' + 1), nothing rounded before the end
__device__ __forceinline__ float gated_act_of(float g, float u, int act, float limit, float slope) {
  if (act == 3) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return __fdividef(g, 1.0f + __expf(-slope * g)) * (u + 1.0f);
  }
  g = round_to<bf16>(g);
  return __fdividef(g, 1.0f + __expf(-g)) * round_to<bf16>(u);
}

template <int BN, int STAGES, bool GATED, int MT>
__global__ void __launch_bounds__(64 + 128 * MT)
grouped_gemm_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_w, bf16* __restrict__ C,
                    const int* __restrict__ offsets, int E, int N, int K, int act, const float* __restrict__ row_weights,
                    float limit, float slope, int* __restrict__ error) {
  constexpr int BC = GATED ? BN / 2 : BN;  // columns of C a block makes
  extern __shared__ __align__(1024) unsigned char smem_raw[];
  constexpr uint32_t B_BYTES = BN * BK * 2;
  constexpr uint32_t STAGE_BYTES = MT * A_BYTES + B_BYTES;
  constexpr uint32_t TMEM_COLS = MT * (BN <= 128 ? 128 : 256);
  unsigned char* tiles = reinterpret_cast<unsigned char*>(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(tiles + (size_t)STAGES * STAGE_BYTES);
  uint64_t* empty_bar = full_bar + STAGES;
  uint64_t* acc_bar = empty_bar + STAGES;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_bar + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  // which expert's which tile: every warp scans the experts' tile counts, 32 at a time
  int e = -1, m0 = 0, row_end = 0;
  for (int e0 = 0, before = 0; e0 < E && e < 0; e0 += 32) {
    const int mine = e0 + lane;
    const int lo = mine < E ? offsets[mine] : 0, hi = mine < E ? offsets[mine + 1] : 0;
    const int tiles_here = (hi - lo + MT * BM - 1) / (MT * BM);
    int incl = tiles_here;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int p = __shfl_up_sync(0xffffffffu, incl, o);
      if (lane >= o) incl += p;
    }
    const int t = (int)blockIdx.y - before;
    const unsigned hit = __ballot_sync(0xffffffffu, t < incl && t >= incl - tiles_here);
    if (hit) {
      const int src = __ffs(hit) - 1;
      e = e0 + src;
      m0 = __shfl_sync(0xffffffffu, lo + (t - (incl - tiles_here)) * (MT * BM), src);
      row_end = __shfl_sync(0xffffffffu, hi, src);
    }
    before += __shfl_sync(0xffffffffu, incl, 31);
  }
  if (e < 0) return;  // the same for the whole block
  const int n0 = blockIdx.x * BC;
  const int k_blocks = (K + BK - 1) / BK;
  const int live = (MT == 2 && row_end - m0 > BM) ? 2 : 1;  // tiles of A that hold rows of this expert

  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) {
      mbar_init(full_bar + s, 1);
      mbar_init(empty_bar + s, 1);
    }
    mbar_init(acc_bar, 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(TMEM_COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;

  if (warp == 0 && lane == 0) {
    for (int kb = 0; kb < k_blocks; ++kb) {
      const int s = kb % STAGES;
      if (kb >= STAGES && !mbar_wait(empty_bar + s, ((kb / STAGES) - 1) & 1)) { atomicExch(error, 3); break; }
      unsigned char* stage = tiles + (size_t)s * STAGE_BYTES;
      mbar_expect_tx(full_bar + s, live * A_BYTES + B_BYTES);
#pragma unroll
      for (int t = 0; t < MT; ++t)
        if (t < live) tma_load_2d(stage + t * A_BYTES, &map_a, full_bar + s, kb * BK, m0 + t * BM);
#pragma unroll
      for (int h = 0; h < BN / 128; ++h)
        tma_load_2d(stage + MT * A_BYTES + h * (128 * BK * 2), &map_w, full_bar + s, kb * BK,
                    GATED ? (2 * e + h) * N + n0 : e * N + n0 + 128 * h);
    }
  } else if (warp == 1 && lane == 0) {
    constexpr uint32_t idesc = umma_idesc(BM, BN);
    for (int kb = 0; kb < k_blocks; ++kb) {
      const int s = kb % STAGES;
      if (!mbar_wait(full_bar + s, (kb / STAGES) & 1)) { atomicExch(error, 4); break; }
      tc_fence_after();
      unsigned char* stage = tiles + (size_t)s * STAGE_BYTES;
      const uint64_t b_desc = umma_desc(stage + MT * A_BYTES);
#pragma unroll
      for (int t = 0; t < MT; ++t) {
        if (t >= live) break;
        const uint64_t a_desc = umma_desc(stage + t * A_BYTES);
#pragma unroll
        for (int k = 0; k < BK / UMMA_K; ++k) {
          const uint64_t adv = (uint64_t)((k * UMMA_K * 2) >> 4);
          umma_bf16(tmem_base + (uint32_t)(t * BN), a_desc + adv, b_desc + adv, idesc, (kb > 0 || k > 0) ? 1u : 0u);
        }
      }
      umma_commit(empty_bar + s);
    }
    umma_commit(acc_bar);  // arrives even after a failed wait, so the epilogue moves on
  } else if (warp >= 2) {
    const int quarter = warp & 3, tile = (warp - 2) >> 2;
    const int row = m0 + tile * BM + quarter * 32 + lane;
    const uint32_t acc = tmem_base + ((uint32_t)(quarter * 32) << 16) + (uint32_t)(tile * BN);
    const bool ok = mbar_wait(acc_bar, 0);
    if (!ok && lane == 0) atomicExch(error, 5);
    tc_fence_after();
    if (ok && tile < live) {
      const float a = (GATED && row_weights && row < row_end) ? row_weights[row] : 1.f;
#pragma unroll 1
      for (int c0 = 0; c0 < BC; c0 += 32) {
        if (n0 + c0 >= N) break;  // the same for the whole block
        uint32_t g[32], u[GATED ? 32 : 1];
        tmem_ld_32x32(acc + (uint32_t)c0, g);
        if constexpr (GATED) tmem_ld_32x32(acc + (uint32_t)(BC + c0), u);
        tmem_wait_ld();
        if (row < row_end) {
          bf16* dst = C + (size_t)row * N + n0 + c0;
          float v[32];
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            v[j] = __uint_as_float(g[j]);
            if constexpr (GATED) {
              v[j] = gated_act_of(a * v[j], a * __uint_as_float(u[j]), act, limit, slope);
            } else if (act == 5) {  // squared relu of the product as it would have been stored
              const float z = round_to<bf16>(v[j]);
              v[j] = z > 0.f ? z * z : 0.f;
            }
          }
          if (n0 + c0 + 32 <= N) {  // N is a multiple of 8: 16-byte stores
#pragma unroll
            for (int j = 0; j < 32; j += 8) {
              uint4 pk;
              __nv_bfloat162* pp = reinterpret_cast<__nv_bfloat162*>(&pk);
#pragma unroll
              for (int q = 0; q < 4; ++q) pp[q] = __floats2bfloat162_rn(v[j + 2 * q], v[j + 2 * q + 1]);
              *reinterpret_cast<uint4*>(dst + j) = pk;
            }
          } else {
#pragma unroll
            for (int j = 0; j < 32; ++j)
              if (n0 + c0 + j < N) dst[j] = from_float<bf16>(v[j]);
          }
        }
      }
    }
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(TMEM_COLS) : "memory");
  }
}

template <int BN, int STAGES, bool GATED, int MT>
int launch_grouped(bf16* C, const bf16* A, const bf16* W, const int* offsets, int rows, int E, int N, int K, int act,
                   const float* row_weights, float limit, float slope, int* error, cudaStream_t stream) {
  static_assert(!GATED || BN == 256, "a gate tile and an up tile of 128 rows each");
  constexpr size_t SMEM = (size_t)STAGES * (MT * A_BYTES + BN * BK * 2) + 1024 + (2 * STAGES + 1) * 8 + 16;
  CUtensorMap map_a, map_w;
  int rc = make_map_bf16(&map_a, A, rows, K, K, BM);
  if (rc) return rc;
  rc = make_map_bf16(&map_w, W, (long long)E * N * (GATED ? 2 : 1), K, K, 128);
  if (rc) return rc;
  auto kern = grouped_gemm_kernel<BN, STAGES, GATED, MT>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)SMEM);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const long long row_tiles = rows / (MT * BM) + (rows < E ? rows : E);  // an expert leaves at most one tile partly filled
  if (row_tiles > 65535) return -3;
  constexpr int BC = GATED ? BN / 2 : BN;
  kern<<<dim3((N + BC - 1) / BC, (unsigned)row_tiles), 64 + 128 * MT, SMEM, stream>>>(map_a, map_w, C, offsets, E, N, K, act, row_weights,
                                                                                limit, slope, error);
  KRK_CHECK_LAUNCH();
  return 0;
}

}  // namespace

// C [rows, N] = act(A [rows, K] W_e^T) over the experts' rows (offsets int32 [E + 1] on the device; rows is the most there
// can be). act: -1 none, 5 squared relu. N and K multiples of 8, K at least 64, 16-byte aligned bases. `gated`: W [E, 2N, K],
// act 0 (silu) or 3 (clamped swish with its limit and slope), row_weights [rows] or null. `tall`: blocks of up to 256 rows
// (N above 128), for experts of more than 128 rows.
KRK_API int krk_grouped_gemm(void* C, const void* A, const void* W, const int* offsets, int rows, int E, int N, int K, int act,
                             int gated, int tall, const float* row_weights, float limit, float slope, int* error,
                             cudaStream_t stream) {
  if (rows == 0 || N == 0 || E == 0) return 0;
  if (N % 8 || K % 8 || K < 64 || (((uintptr_t)A | (uintptr_t)W | (uintptr_t)C) & 15) || 2LL * E * N > 0x7fffffffLL) return -2;
  if (gated ? (act != 0 && act != 3) : ((act != -1 && act != 5) || row_weights)) return -2;
  auto go = gated ? (tall ? launch_grouped<256, 3, true, 2> : launch_grouped<256, 4, true, 1>)
                  : N <= 128 ? launch_grouped<128, 4, false, 1>
                             : (tall ? launch_grouped<256, 3, false, 2> : launch_grouped<256, 4, false, 1>);
  return go((bf16*)C, (const bf16*)A, (const bf16*)W, offsets, rows, E, N, K, act, row_weights, limit, slope, error, stream);
}
