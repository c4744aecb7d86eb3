// Kernels of attention over one cached low-rank row per token.
//
// krk_latent_norm_write: one warp per row. The row's `rank` projected elements are divided by their root
// mean square (eps under the root), multiplied by a float32 gain and written, rounded once, to the
// position's place in a cache of one "kv head" of `rank` elements (and, if asked, to a plain row buffer as well).
//
// krk_latent_rows: the same for rows with a rotated part behind them, and beside it the RMS norm of a low-rank query row of
// the same input row, written to a buffer: a warp per (row, which of the two).
//
// krk_latent_gather: the cached rows of every sequence of a step, positions 0 .. its new length - 1, as one dense
// matrix.
//
// krk_head_linear: out[r, h, :] = scale * W_h x[r, h, :] for every head h, W [heads, N, K] contiguous;
// x and out are rows with strides, a head's slice of x starting x_head elements after the one before (out: out_head).
// With rot > 0 the rot elements behind a head's K are rotated (neighbours together, cosine and sine times a factor) and
// placed behind its N results: what carries a query with a rotated part into the latent space. With a gate, results are
// multiplied by sigmoid of the gate's element of the same place (heads * N columns). One block per (tile of output elements, head, tile of 8 rows): the
// rows' slices sit in shared memory as float32, each warp owns output elements, its lanes split K
// (coalesced reads of W's rows), sums are float32 and their order does not depend on the other rows.
#include "mma.cuh"

namespace {

template <typename T>
__global__ void latent_norm_write_kernel(const T* __restrict__ proj, int stride, int c_col, int R,
                                         const float* __restrict__ gain, float eps, const int* __restrict__ row_seq,
                                         const int* __restrict__ row_pos, const int* __restrict__ seq_slot,
                                         const int* __restrict__ table, int width, int keep_pages, T* cache, int rows,
                                         T* __restrict__ rows_out) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int lane = threadIdx.x & 31;
  const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (row >= rows) return;
  const T* c = proj + (size_t)row * stride + c_col;
  float sq = 0.f;
  for (int i = lane; i < R; i += 32) {
    const float f = to_float<T>(c[i]);
    sq += f * f;
  }
  const float rstd = rsqrtf(warp_sum(sq) / (float)R + eps);
  const int pos = row_pos[row];
  const int page = page_of(table, width, seq_slot[row_seq[row]], pos, keep_pages);
  T* dst = cache + ((size_t)page * KRK_PAGE + (pos % KRK_PAGE)) * R;
  for (int i = lane; i < R; i += 32) {
    const T v = from_float<T>(to_float<T>(c[i]) * rstd * gain[i]);
    dst[i] = v;
    if (rows_out) rows_out[(size_t)row * R + i] = v;
  }
}

// sine and cosine of p * (f_hi + f_lo): the product's float32 value through sincosf, its rounding error and the rest of
// the frequency as a first-order correction
__device__ __forceinline__ void pair_sincos(float p, float f_hi, float f_lo, float* s, float* c) {
  const float a = __fmul_rn(p, f_hi);
  const float e = fmaf(p, f_hi, -a) + p * f_lo;
  float s0, c0;
  sincosf(a, &s0, &c0);
  *s = fmaf(e, c0, s0);
  *c = fmaf(-e, s0, c0);
}

// dst and src [rot]: neighbours rotated together by a warp
template <typename T>
__device__ __forceinline__ void rotate_pairs_warp(T* dst, const T* src, int rot, float p, const float* __restrict__ inv_freq,
                                                  float factor, int lane) {
  const int half = rot >> 1;
  for (int i = lane; i < half; i += 32) {
    float s, c;
    pair_sincos(p, inv_freq[i], inv_freq[half + i], &s, &c);
    s *= factor;
    c *= factor;
    const float u = to_float<T>(src[2 * i]), v = to_float<T>(src[2 * i + 1]);
    dst[2 * i] = from_float<T>(u * c - v * s);
    dst[2 * i + 1] = from_float<T>(v * c + u * s);
  }
}

template <typename T>
__device__ __forceinline__ void rms_row_warp(T* dst, const T* __restrict__ src, int n, const float* __restrict__ gain, float eps,
                                             int lane) {
  float sq = 0.f;
  if (sizeof(T) == 2 && (n & 7) == 0 &&
      ((reinterpret_cast<uintptr_t>(src) | reinterpret_cast<uintptr_t>(dst) | reinterpret_cast<uintptr_t>(gain)) & 15) == 0) {
    // 16-byte pieces, the first eight a lane kept in registers between the sum and the result (rows of up to 2,048)
    constexpr int KEEP = 8;
    uint4 raw[KEEP];
    auto squares = [](const uint4& r) {
      const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&r);
      float t = 0.f;
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float a = __low2float(p[q]), b = __high2float(p[q]);
        t += a * a + b * b;
      }
      return t;
    };
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
      const int i = 8 * (lane + 32 * j);
      raw[j] = i < n ? *reinterpret_cast<const uint4*>(src + i) : make_uint4(0u, 0u, 0u, 0u);
    }
#pragma unroll
    for (int j = 0; j < KEEP; ++j) sq += squares(raw[j]);
    for (int i = 8 * (lane + 32 * KEEP); i < n; i += 256) sq += squares(*reinterpret_cast<const uint4*>(src + i));
    const float rstd = rsqrtf(warp_sum(sq) / (float)n + eps);
    auto store = [&](int i, const uint4& r) {
      const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&r);
      uint4 o;
      __nv_bfloat162* po = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
      for (int q = 0; q < 4; ++q)
        po[q] = __floats2bfloat162_rn(__low2float(p[q]) * rstd * gain[i + 2 * q], __high2float(p[q]) * rstd * gain[i + 2 * q + 1]);
      *reinterpret_cast<uint4*>(dst + i) = o;
    };
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
      const int i = 8 * (lane + 32 * j);
      if (i < n) store(i, raw[j]);
    }
    for (int i = 8 * (lane + 32 * KEEP); i < n; i += 256) store(i, *reinterpret_cast<const uint4*>(src + i));
    return;
  }
  for (int i = lane; i < n; i += 32) {
    const float f = to_float<T>(src[i]);
    sq += f * f;
  }
  const float rstd = rsqrtf(warp_sum(sq) / (float)n + eps);
  for (int i = lane; i < n; i += 32) dst[i] = from_float<T>(to_float<T>(src[i]) * rstd * gain[i]);
}

template <typename T>
__global__ void latent_rows_kernel(T* __restrict__ q_out, const T* __restrict__ proj, int stride, int q_col, int QR,
                                   const float* __restrict__ q_gain, int c_col, int R, const float* __restrict__ c_gain, int rot,
                                   const float* __restrict__ inv_freq, float factor, float eps,
                                   const int* __restrict__ row_seq, const int* __restrict__ row_pos,
                                   const int* __restrict__ seq_slot, const int* __restrict__ table, int width, T* cache,
                                   int rows) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int lane = threadIdx.x & 31;
  const int item = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int kinds = cache ? 2 : 1;
  if (item >= rows * kinds) return;
  const int row = item / kinds;
  const T* src = proj + (size_t)row * stride;
  if (item % kinds == 0) {
    rms_row_warp<T>(q_out + (size_t)row * QR, src + q_col, QR, q_gain, eps, lane);
    return;
  }
  const int pos = row_pos[row];
  const int page = page_of(table, width, seq_slot[row_seq[row]], pos);
  T* dst = cache + ((size_t)page * KRK_PAGE + (pos % KRK_PAGE)) * (R + rot);
  rms_row_warp<T>(dst, src + c_col, R, c_gain, eps, lane);
  rotate_pairs_warp<T>(dst + R, src + c_col + R, rot, (float)pos, inv_freq, factor, lane);
}

// out [sum of lengths, W]: a block per 8 positions of a sequence (blockIdx.y); offsets[s] is where sequence s starts
template <typename T>
__global__ void latent_gather_kernel(T* __restrict__ out, const T* __restrict__ cache, int W, const int* __restrict__ seq_slot,
                                     const int* __restrict__ seq_start, const int* __restrict__ seq_qlen,
                                     const int* __restrict__ offsets, const int* __restrict__ table, int width) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int seq = blockIdx.y;
  const int n = seq_start[seq] + seq_qlen[seq];
  const int pos = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (pos >= n) return;
  const T* src = cache + ((size_t)page_of(table, width, seq_slot[seq], pos) * KRK_PAGE + (pos % KRK_PAGE)) * W;
  T* dst = out + ((size_t)offsets[seq] + pos) * W;
  if ((W * sizeof(T)) % 16 == 0) {
    for (int i = lane; i < W * (int)sizeof(T) / 16; i += 32) reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
    return;
  }
  for (int i = lane; i < W; i += 32) dst[i] = src[i];
}

constexpr int HL_ROWS = 8;
constexpr int HL_WARPS = 8;

template <typename T>
__global__ void __launch_bounds__(HL_WARPS * 32)
head_linear_kernel(T* __restrict__ out, int out_stride, int out_col, int out_head, float out_scale, const T* __restrict__ x,
                   int x_stride, int x_head, const T* __restrict__ w, int N, int K, int rows, int rot,
                   const float* __restrict__ inv_freq, float factor, const int* __restrict__ row_pos,
                   const T* __restrict__ gate, int gate_stride) {
  extern __shared__ __align__(16) float xs[];  // [HL_ROWS][K4], K4 = K rounded up to a multiple of 4
  const int K4 = (K + 3) & ~3;
  grid_launch_dependents();
  grid_dependency_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int h = blockIdx.y, r0 = blockIdx.z * HL_ROWS;
  const int nr = min(HL_ROWS, rows - r0);
  for (int i = threadIdx.x; i < HL_ROWS * K; i += blockDim.x) {
    const int r = i / K, k = i - r * K;
    xs[r * K4 + k] = r < nr ? to_float<T>(x[(size_t)(r0 + r) * x_stride + (size_t)h * x_head + k]) : 0.f;
  }
  __syncthreads();
  for (int n = blockIdx.x * HL_WARPS + warp; n < N; n += gridDim.x * HL_WARPS) {
    const T* wr = w + ((size_t)h * N + n) * K;
    float mine = 0.f;
#pragma unroll
    for (int r = 0; r < HL_ROWS; ++r) {
      if (r >= nr) break;
      const float t = warp_sum(lane_dot<T>(wr, xs + r * K4, K, lane));  // the weight row comes from L1 after the first
      if (lane == r) mine = t;
    }
    if (lane < nr) {
      mine *= out_scale;
      if (gate) mine *= 1.0f / (1.0f + expf(-to_float<T>(gate[(size_t)(r0 + lane) * gate_stride + (size_t)h * N + n])));
      out[(size_t)(r0 + lane) * out_stride + out_col + (size_t)h * out_head + n] = from_float<T>(mine);
    }
  }
  if (rot > 0 && blockIdx.x == 0 && warp < nr) {
    const int r = r0 + warp;  // HL_WARPS >= HL_ROWS
    rotate_pairs_warp<T>(out + (size_t)r * out_stride + out_col + (size_t)h * out_head + N,
                         x + (size_t)r * x_stride + (size_t)h * x_head + K, rot, (float)row_pos[r], inv_freq, factor, lane);
  }
}

// The same on the tensor cores for bfloat16 and K a multiple of 8: a warp takes 8 output elements of one head for up to 16
// rows. A lane loads 16 bytes of its output element's weight row and of its two input rows: along K a lane's eight elements
// stand for elements 2t, 2t + 1, 2t + 8, 2t + 9 of two m16n8k16 products, the same places in both operands, so no operand
// passes through shared memory. A row's sums depend on its own elements alone.
__global__ void __launch_bounds__(HL_WARPS * 32)
head_linear_mma_kernel(bf16* __restrict__ out, int out_stride, int out_col, int out_head, float out_scale,
                       const bf16* __restrict__ x, int x_stride, int x_head, const bf16* __restrict__ w, int N, int K, int rows,
                       int rot, const float* __restrict__ inv_freq, float factor, const int* __restrict__ row_pos,
                       const bf16* __restrict__ gate, int gate_stride) {
  grid_launch_dependents();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.y, r0 = blockIdx.z * 16;
  const int n0 = (blockIdx.x * HL_WARPS + warp) * 8;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  const bool w_on = n0 + g < N, a_on = r0 + g < rows, b_on = r0 + g + 8 < rows;
  const bf16* wr = w + ((size_t)h * N + (w_on ? n0 + g : 0)) * K + 8 * t4;
  const bf16* xa = x + (size_t)(r0 + g) * x_stride + (size_t)h * x_head + 8 * t4;
  const bf16* xb = xa + (size_t)8 * x_stride;
  constexpr int FLY = 4;
  uint4 wv[FLY];
#pragma unroll
  for (int i = 0; i < FLY; ++i) wv[i] = (w_on && 32 * i + 8 * t4 < K) ? *reinterpret_cast<const uint4*>(wr + 32 * i) : zero;
  grid_dependency_wait();  // no kernel writes the weights
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  if (n0 < N) {
    for (int k0 = 0; k0 < K; k0 += 32 * FLY) {
      uint4 next[FLY], av[FLY], bv[FLY];
#pragma unroll
      for (int i = 0; i < FLY; ++i) {
        const int k = k0 + 32 * i, kn = k + 32 * FLY;
        next[i] = (w_on && kn + 8 * t4 < K) ? *reinterpret_cast<const uint4*>(wr + kn) : zero;
        av[i] = (a_on && k + 8 * t4 < K) ? *reinterpret_cast<const uint4*>(xa + k) : zero;
        bv[i] = (b_on && k + 8 * t4 < K) ? *reinterpret_cast<const uint4*>(xb + k) : zero;
      }
#pragma unroll
      for (int i = 0; i < FLY; ++i) {
        if (k0 + 32 * i >= K) break;
        mma_bf16_16816(acc, av[i].x, bv[i].x, av[i].y, bv[i].y, wv[i].x, wv[i].y);
        mma_bf16_16816(acc, av[i].z, bv[i].z, av[i].w, bv[i].w, wv[i].z, wv[i].w);
        wv[i] = next[i];
      }
    }
#pragma unroll
    for (int c = 0; c < 4; ++c) {
      const int r = r0 + g + 8 * (c >> 1), n = n0 + 2 * t4 + (c & 1);
      if (r >= rows || n >= N) continue;
      float v = acc[c] * out_scale;
      if (gate) v *= 1.0f / (1.0f + expf(-__bfloat162float(gate[(size_t)r * gate_stride + (size_t)h * N + n])));
      out[(size_t)r * out_stride + out_col + (size_t)h * out_head + n] = __float2bfloat16_rn(v);
    }
  }
  if (rot > 0 && blockIdx.x == 0)
    for (int r = r0 + warp; r < min(rows, r0 + 16); r += HL_WARPS)
      rotate_pairs_warp<bf16>(out + (size_t)r * out_stride + out_col + (size_t)h * out_head + N,
                              x + (size_t)r * x_stride + (size_t)h * x_head + K, rot, (float)row_pos[r], inv_freq, factor, lane);
}

}  // namespace

KRK_API int krk_latent_norm_write(const void* proj, int stride, int c_col, int R, const float* gain, float eps,
                                  const int* row_seq, const int* row_pos, const int* seq_slot, const int* table, int width,
                                  int keep_pages, void* cache, int rows, void* rows_out, int dtype, cudaStream_t stream) {
  if (rows == 0) return 0;
  const int warps = 4;
  const unsigned blocks = (unsigned)((rows + warps - 1) / warps);
  if (dtype == KRK_DTYPE_F32)
    return (int)launch_pdl(latent_norm_write_kernel<float>, dim3(blocks), dim3(warps * 32), 0, stream, (const float*)proj,
                           stride, c_col, R, gain, eps, row_seq, row_pos, seq_slot, table, width, keep_pages,
                           (float*)cache, rows, (float*)rows_out);
  return (int)launch_pdl(latent_norm_write_kernel<bf16>, dim3(blocks), dim3(warps * 32), 0, stream, (const bf16*)proj,
                         stride, c_col, R, gain, eps, row_seq, row_pos, seq_slot, table, width, keep_pages, (bf16*)cache,
                         rows, (bf16*)rows_out);
}

KRK_API int krk_latent_rows(void* q_out, const void* proj, int stride, int q_col, int QR, const float* q_gain, int c_col, int R,
                            const float* c_gain, int rot, const float* inv_freq, float factor, float eps, const int* row_seq,
                            const int* row_pos, const int* seq_slot, const int* table, int width, void* cache, int rows,
                            int dtype, cudaStream_t stream) {
  if (rows == 0) return 0;
  if (rot < 0 || (rot & 1)) return -2;
  const int warps = 4;
  const long long items = (long long)rows * (cache ? 2 : 1);
  if (items > 0x7fffffffLL) return -3;
  const unsigned blocks = (unsigned)((items + warps - 1) / warps);
  if (dtype == KRK_DTYPE_F32)
    return (int)launch_pdl(latent_rows_kernel<float>, dim3(blocks), dim3(warps * 32), 0, stream, (float*)q_out,
                           (const float*)proj, stride, q_col, QR, q_gain, c_col, R, c_gain, rot, inv_freq, factor, eps, row_seq,
                           row_pos, seq_slot, table, width, (float*)cache, rows);
  return (int)launch_pdl(latent_rows_kernel<bf16>, dim3(blocks), dim3(warps * 32), 0, stream, (bf16*)q_out, (const bf16*)proj,
                         stride, q_col, QR, q_gain, c_col, R, c_gain, rot, inv_freq, factor, eps, row_seq, row_pos, seq_slot,
                         table, width, (bf16*)cache, rows);
}

KRK_API int krk_latent_gather(void* out, const void* cache, int W, int n_seqs, int max_kv_len, const int* seq_slot,
                              const int* seq_start, const int* seq_qlen, const int* offsets, const int* table, int width,
                              int dtype, cudaStream_t stream) {
  if (n_seqs == 0 || max_kv_len == 0) return 0;
  if (n_seqs > 65535) return -3;
  const dim3 grid((unsigned)((max_kv_len + 7) / 8), (unsigned)n_seqs);
  if (dtype == KRK_DTYPE_F32)
    return (int)launch_pdl(latent_gather_kernel<float>, grid, dim3(256), 0, stream, (float*)out, (const float*)cache, W,
                           seq_slot, seq_start, seq_qlen, offsets, table, width);
  return (int)launch_pdl(latent_gather_kernel<bf16>, grid, dim3(256), 0, stream, (bf16*)out, (const bf16*)cache, W, seq_slot,
                         seq_start, seq_qlen, offsets, table, width);
}

KRK_API int krk_head_linear(void* out, int out_stride, int out_col, int out_head, float out_scale, const void* x, int x_stride,
                            int x_head, const void* w, int heads, int N, int K, int rows, int rot, const float* inv_freq,
                            float factor, const int* row_pos, const void* gate, int gate_stride, int dtype,
                            cudaStream_t stream) {
  if (rows == 0 || heads == 0 || N == 0) return 0;
  if (rot < 0 || (rot & 1) || (rot > 0 && (!inv_freq || !row_pos))) return -2;
  if (dtype == KRK_DTYPE_BF16 && K % 8 == 0 && x_stride % 8 == 0 && x_head % 8 == 0 &&
      (((uintptr_t)x | (uintptr_t)w) & 15) == 0) {
    const int tiles = (rows + 15) / 16;
    if (heads > 65535 || tiles > 65535) return -3;
    const dim3 grid((unsigned)((N + 8 * HL_WARPS - 1) / (8 * HL_WARPS)), (unsigned)heads, (unsigned)tiles);
    return (int)launch_pdl(head_linear_mma_kernel, grid, dim3(HL_WARPS * 32), 0, stream, (bf16*)out, out_stride, out_col, out_head,
                           out_scale, (const bf16*)x, x_stride, x_head, (const bf16*)w, N, K, rows, rot, inv_freq, factor, row_pos,
                           (const bf16*)gate, gate_stride);
  }
  const size_t smem = (size_t)HL_ROWS * ((K + 3) & ~3) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  if (smem > 48 * 1024) {
    cudaFuncSetAttribute(head_linear_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    cudaFuncSetAttribute(head_linear_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  }
  const int row_tiles = (rows + HL_ROWS - 1) / HL_ROWS;
  if (heads > 65535 || row_tiles > 65535) return -3;
  const dim3 grid((unsigned)((N + HL_WARPS - 1) / HL_WARPS), (unsigned)heads, (unsigned)row_tiles);
  if (dtype == KRK_DTYPE_F32)
    return (int)launch_pdl(head_linear_kernel<float>, grid, dim3(HL_WARPS * 32), smem, stream, (float*)out, out_stride,
                           out_col, out_head, out_scale, (const float*)x, x_stride, x_head, (const float*)w, N, K, rows, rot,
                           inv_freq, factor, row_pos, (const float*)gate, gate_stride);
  return (int)launch_pdl(head_linear_kernel<bf16>, grid, dim3(HL_WARPS * 32), smem, stream, (bf16*)out, out_stride, out_col,
                         out_head, out_scale, (const bf16*)x, x_stride, x_head, (const bf16*)w, N, K, rows, rot, inv_freq,
                         factor, row_pos, (const bf16*)gate, gate_stride);
}
