// Single-token attention over cached latent rows on the tensor cores (mma.sync m16n8k16, bfloat16 in, float32 accumulate).
//
// Every head reads the same row of W = R + E elements per position as its key and the row's first R as its value, so sixteen
// heads are the sixteen rows of a tile: S [16 x 64] = Q [16 x W] rows^T, O [16 x R] += P rows[:, :R]. A block takes sixteen
// heads of one sequence and every `splits`-th page of its positions; a page is brought to shared memory once (cp.async, two
// stages) and serves as keys and as values. Warp w scores the page's keys 8w .. 8w + 7, then softens two heads' rows of
// scores (float32, online), then adds its share of the value columns; a weight reaches P.V as two bfloat16 halves. Each
// block leaves (output, maximum, sum) per head in scratch, and krk_latent_decode's second kernel adds the shares in block
// order. The number of splits depends on the step's shape alone, so a captured step stays valid as sequences grow.
#include "mma.cuh"

namespace {

constexpr int WARPS = 8, HEADS = 16, KEYS = KRK_PAGE;
constexpr int SP = KEYS + 4, PP = KEYS + 8;  // row pitches of scores (float) and weights (bfloat16)
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// NT: 8-wide value tiles per warp (a multiple of 2)
template <int NT>
__global__ void __launch_bounds__(WARPS * 32)
latent_decode_kernel(float* __restrict__ scratch, const bf16* __restrict__ q, int q_stride, int H, int R, int W,
                     const int* __restrict__ seq_slot, const int* __restrict__ seq_start, const int* __restrict__ table,
                     int width, const bf16* __restrict__ cache, float scale_log2) {
  extern __shared__ __align__(16) bf16 sm[];
  const int WP = W + 8;
  bf16* qs = sm;                                    // [HEADS][WP]
  bf16* rows = qs + HEADS * WP;                     // [2][KEYS][WP]
  bf16* ps = rows + 2 * KEYS * WP;                  // [2 halves][HEADS][PP]
  float* ss = reinterpret_cast<float*>(ps + 2 * HEADS * PP);  // [HEADS][SP]
  float* alpha_s = ss + HEADS * SP;                 // [HEADS]
  const int split = blockIdx.x, splits = gridDim.x, h0 = blockIdx.y * HEADS, seq = blockIdx.z;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = lane >> 2, t4 = lane & 3;
  grid_launch_dependents();
  grid_dependency_wait();
  const int pos = seq_start[seq], slot = seq_slot[seq];  // the new token sits at the length before the step
  const int pages = pos / KEYS + 1;
  const int nh = min(HEADS, H - h0);

  auto issue = [&](int j, int stage) {
    const bf16* src = cache + (size_t)table[(size_t)slot * width + j % width] * KEYS * W;
    bf16* dst = rows + stage * KEYS * WP;
    const int pieces = W / 8;
    for (int i = threadIdx.x; i < KEYS * pieces; i += WARPS * 32) {
      const int key = i / pieces, c = i - key * pieces;
      cp_async_16(dst + key * WP + c * 8, src + key * W + c * 8);
    }
    cp_async_commit();
  };
  if (split < pages) issue(split, 0);
  for (int i = threadIdx.x; i < HEADS * (W / 8); i += WARPS * 32) {
    const int r = i / (W / 8), c = i % (W / 8);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < nh) v = *reinterpret_cast<const uint4*>(q + (size_t)seq * q_stride + (size_t)(h0 + r) * W + c * 8);
    *reinterpret_cast<uint4*>(qs + r * WP + c * 8) = v;
  }

  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};  // of heads 2 * warp and 2 * warp + 1
  float o[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int c = 0; c < 4; ++c) o[n][c] = 0.f;
  const int tile0 = warp * NT, tiles = R / 8;

  int stage = 0;
  for (int j = split; j < pages; j += splits, stage ^= 1) {
    if (j + splits < pages) {
      issue(j + splits, stage ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const bf16* kr = rows + stage * KEYS * WP;
    {
      float s[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int c = 0; c < 4; ++c) s[i][c] = 0.f;
      for (int k0 = 0; k0 < W; k0 += 32) {  // two k-steps at a time; W is a multiple of 16
        uint32_t b0, b1, b2, b3;
        const int col = min(k0 + (lane >> 3) * 8, W - 8);
        ldmatrix_x4(b0, b1, b2, b3, kr + (warp * 8 + (lane & 7)) * WP + col);
        uint32_t a0, a1, a2, a3;
        ldmatrix_x4(a0, a1, a2, a3, qs + (lane & 15) * WP + k0 + (lane >> 4) * 8);
        mma_bf16_16816(s[0], a0, a1, a2, a3, b0, b1);
        if (k0 + 16 < W) {
          ldmatrix_x4(a0, a1, a2, a3, qs + (lane & 15) * WP + k0 + 16 + (lane >> 4) * 8);
          mma_bf16_16816(s[1], a0, a1, a2, a3, b2, b3);
        }
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int key = warp * 8 + 2 * t4 + (c & 1);
        ss[(g + 8 * (c >> 1)) * SP + key] = j * KEYS + key <= pos ? (s[0][c] + s[1][c]) * scale_log2 : -INFINITY;
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = 2 * warp + i;
      const float2 x = *reinterpret_cast<const float2*>(ss + r * SP + 2 * lane);
      const float m_new = fmaxf(m[i], warp_max(fmaxf(x.x, x.y)));  // a page's first key is visible
      const float alpha = fast_exp2(m[i] - m_new);
      const float p0 = fast_exp2(x.x - m_new), p1 = fast_exp2(x.y - m_new);
      l[i] = l[i] * alpha + warp_sum(p0 + p1);
      m[i] = m_new;
      const float q0 = __bfloat162float(__float2bfloat16_rn(p0)), q1 = __bfloat162float(__float2bfloat16_rn(p1));
      *reinterpret_cast<uint32_t*>(ps + r * PP + 2 * lane) = pack_bf16x2(q0, q1);
      *reinterpret_cast<uint32_t*>(ps + (HEADS + r) * PP + 2 * lane) = pack_bf16x2(p0 - q0, p1 - q1);
      if (lane == 0) alpha_s[r] = alpha;
    }
    __syncthreads();
    if (tile0 < tiles) {
      const float f0 = alpha_s[g], f1 = alpha_s[g + 8];
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        o[n][0] *= f0; o[n][1] *= f0;
        o[n][2] *= f1; o[n][3] *= f1;
      }
#pragma unroll
      for (int kk = 0; kk < KEYS / 16; ++kk) {
        uint32_t hi[4], lo[4];
        ldmatrix_x4(hi[0], hi[1], hi[2], hi[3], ps + (lane & 15) * PP + kk * 16 + (lane >> 4) * 8);
        ldmatrix_x4(lo[0], lo[1], lo[2], lo[3], ps + (HEADS + (lane & 15)) * PP + kk * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int n = 0; n < NT; n += 2) {
          if (tile0 + n >= tiles) break;
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(b0, b1, b2, b3, kr + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * WP + (tile0 + n + (lane >> 4)) * 8);
          mma_bf16_16816(o[n], hi[0], hi[1], hi[2], hi[3], b0, b1);
          mma_bf16_16816(o[n], lo[0], lo[1], lo[2], lo[3], b0, b1);
          mma_bf16_16816(o[n + 1], hi[0], hi[1], hi[2], hi[3], b2, b3);
          mma_bf16_16816(o[n + 1], lo[0], lo[1], lo[2], lo[3], b2, b3);
        }
      }
    }
    __syncthreads();  // the stage, the scores and the weights are free
  }
  // this block's share of every head: R outputs, the maximum (log2 units), the sum
  const int PS = R + 2;
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    const int r = g + 8 * hh;
    if (r >= nh) continue;
    float* dst = scratch + (((size_t)seq * H + h0 + r) * splits + split) * PS;
#pragma unroll
    for (int n = 0; n < NT; ++n)
      if (tile0 + n < tiles) *reinterpret_cast<float2*>(dst + (tile0 + n) * 8 + 2 * t4) = make_float2(o[n][2 * hh], o[n][2 * hh + 1]);
  }
  if (lane < 2 && 2 * warp + lane < nh) {
    float* dst = scratch + (((size_t)seq * H + h0 + 2 * warp + lane) * splits + split) * PS;
    dst[R] = lane ? m[1] : m[0];
    dst[R + 1] = lane ? l[1] : l[0];
  }
}

// The shares of one (sequence, head), added in block order: 64 columns a warp, a lane per share for the factors (up to 32)
__global__ void latent_decode_merge_kernel(bf16* __restrict__ out, const float* __restrict__ scratch, int R, int splits,
                                           int items) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int lane = threadIdx.x & 31;
  const int chunks = (R + 63) / 64, PS = R + 2;
  const long long w = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int item = (int)(w / chunks), c = (int)(w % chunks) * 64 + 2 * lane;
  if (item >= items) return;
  const float* base = scratch + (size_t)item * splits * PS;
  const float m = lane < splits ? base[(size_t)lane * PS + R] : -INFINITY;
  const float top = warp_max(m);
  const float f = m == -INFINITY ? 0.f : fast_exp2(m - top);
  const float total = warp_sum(lane < splits ? f * base[(size_t)lane * PS + R + 1] : 0.f);
  float2 acc = make_float2(0.f, 0.f);
  const bool on = c < R;
  for (int s0 = 0; s0 < splits; s0 += 8) {
    float2 v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i)
      v[i] = (on && s0 + i < splits) ? *reinterpret_cast<const float2*>(base + (size_t)(s0 + i) * PS + c) : make_float2(0.f, 0.f);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float fi = __shfl_sync(0xffffffffu, f, (s0 + i) & 31);
      acc.x = fmaf(v[i].x, fi, acc.x);
      acc.y = fmaf(v[i].y, fi, acc.y);
    }
  }
  if (on) *reinterpret_cast<uint32_t*>(out + (size_t)item * R + c) = pack_bf16x2(acc.x / total, acc.y / total);
}

size_t decode_smem(int W) {
  return (size_t)(HEADS + 2 * KEYS) * (W + 8) * sizeof(bf16) + 2 * HEADS * PP * sizeof(bf16) + (HEADS * SP + HEADS) * sizeof(float);
}

}  // namespace

// out [n_seqs, H * R] bfloat16: per head, the softmax of q . row over the sequence's positions times the rows' first R
// elements. q [n_seqs, H * W] (16-byte aligned rows), cache [pages, 64, W]; R and W multiples of 16, R up to 512. scratch:
// n_seqs * H * splits * (R + 2) floats, up to 32 splits. -2: sizes it does not take.
KRK_API int krk_latent_decode(void* out, float* scratch, const void* q, int q_stride, int H, int R, int W, const int* seq_slot,
                              const int* seq_start, const int* table, int width, const void* cache, float scale, int splits,
                              int n_seqs, cudaStream_t stream) {
  if (n_seqs == 0) return 0;
  const size_t smem = decode_smem(W);
  if (R % 16 || W % 16 || R > 512 || R > W || q_stride % 8 || (((uintptr_t)q | (uintptr_t)cache) & 15) || ((uintptr_t)out & 3) ||
      ((uintptr_t)scratch & 7) || splits < 1 || splits > 32 || smem > 220 * 1024 || n_seqs > 65535)
    return -2;
  auto kern = R <= 128 ? latent_decode_kernel<2> : R <= 256 ? latent_decode_kernel<4> : latent_decode_kernel<8>;
  cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  int rc = (int)launch_pdl(kern, dim3((unsigned)splits, (unsigned)((H + HEADS - 1) / HEADS), (unsigned)n_seqs), dim3(WARPS * 32),
                           smem, stream, scratch, (const bf16*)q, q_stride, H, R, W, seq_slot, seq_start, table, width,
                           (const bf16*)cache, scale * LOG2E);
  if (rc) return rc;
  const long long warps = (long long)n_seqs * H * ((R + 63) / 64);
  return (int)launch_pdl(latent_decode_merge_kernel, dim3((unsigned)((warps + 3) / 4)), dim3(128), 0, stream, (bf16*)out,
                         (const float*)scratch, R, splits, n_seqs * H);
}
