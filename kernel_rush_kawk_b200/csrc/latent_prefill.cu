// Causal attention of a step's rows over keys and values that were made from latent rows, for steps that bring many
// tokens per sequence, in bfloat16 (mma.sync m16n8k16, float32 accumulate).
//
// A key of head h is two pieces: `plain` elements of its own, row j of the dense product kv = [Wuk; Wuv] c (all heads'
// keys, then all heads' values), and the rotated part that all heads share, which sits behind the latent in the row the
// product was made from. The pieces meet in shared memory; no key is ever written out whole. Queries are rotated on
// their way into shared memory (neighbours together; see latent.cu), so a head's row is rotated by the one block that
// reads it.
//
// Block = (64 query rows, head, sequence), four warps of 16 rows; keys come 64 positions at a time by cp.async in two
// stages. Scores, maxima and sums are float32; a weight reaches P.V as two bfloat16 halves (about 16 bits of mantissa). The
// result is multiplied by sigmoid of the gate's element of the same place and by out_scale. A query at position p sees
// positions 0..p.
//
// Compiled once per pair of sizes: -DKRK_KEY_DIM=<plain + rotated> -DKRK_VALUE_DIM=<value head>, multiples of 16.
#include "mma.cuh"

#if !defined(KRK_KEY_DIM) || !defined(KRK_VALUE_DIM)
#error "compile with -DKRK_KEY_DIM=<key size> -DKRK_VALUE_DIM=<value size>"
#endif

namespace {

constexpr int D = KRK_KEY_DIM, DV = KRK_VALUE_DIM;
static_assert(D % 16 == 0 && DV % 16 == 0, "multiples of 16");
constexpr int KP = D + 8, VP = DV + 8;  // row pitches in shared memory: an odd number of 16-byte pieces
constexpr int KSTEPS = D / 16, VTILES = DV / 8;
constexpr int KEYS = 64, ROWS = 64, THREADS = 128;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct Args {
  bf16* out;
  int out_stride;
  float out_scale;
  const bf16* q;  // [rows, H * D]
  int q_stride, H, plain;
  const bf16* kv;  // [sum of lengths, H * (plain + DV)]
  const bf16* rows;  // [sum of lengths, rank + rot]
  int row_width, rank;
  const float* inv_freq;
  float factor, scale_log2;
  const int *seq_start, *seq_qlen, *cu_q, *offsets;
  const bf16* gate;
  int gate_stride;
};

__global__ void __launch_bounds__(THREADS) latent_prefill_kernel(Args a) {
  extern __shared__ __align__(16) bf16 smem[];  // [2 stages][K [KEYS][KP], V [KEYS][VP]]; the query tile uses stage 1's K first
  constexpr int STAGE = KEYS * (KP + VP);
  const int seq = blockIdx.z, h = blockIdx.y;
  const int tile = gridDim.x - 1 - blockIdx.x;  // long tiles first
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int g = lane >> 2, t4 = lane & 3;
  grid_launch_dependents();
  grid_dependency_wait();
  const int q_len = a.seq_qlen[seq];
  if (tile * ROWS >= q_len) return;
  const int start = a.seq_start[seq], row0 = a.cu_q[seq], base = a.offsets[seq];
  const int plain = a.plain, rot = D - plain, plain_pieces = plain / 8;
  const int kv_width = a.H * (plain + DV);
  const int last_pos = start + min(q_len, tile * ROWS + ROWS) - 1;  // of the tile
  const int total = start + q_len;
  const int steps = last_pos / KEYS + 1;

  auto issue = [&](int j, int stage) {
    bf16* ks = smem + stage * STAGE;
    bf16* vs = ks + KEYS * KP;
    for (int i = threadIdx.x; i < KEYS * (D / 8); i += THREADS) {
      const int key = i / (D / 8), c = i % (D / 8);
      const size_t r = (size_t)base + min(j * KEYS + key, total - 1);  // beyond the last position: any row, never seen
      const bf16* src = c < plain_pieces ? a.kv + r * kv_width + (size_t)h * plain + c * 8
                                         : a.rows + r * a.row_width + a.rank + (c - plain_pieces) * 8;
      cp_async_16(ks + key * KP + c * 8, src);
    }
    for (int i = threadIdx.x; i < KEYS * (DV / 8); i += THREADS) {
      const int key = i / (DV / 8), c = i % (DV / 8);
      const size_t r = (size_t)base + min(j * KEYS + key, total - 1);
      cp_async_16(vs + key * VP + c * 8, a.kv + r * kv_width + (size_t)a.H * plain + (size_t)h * DV + c * 8);
    }
    cp_async_commit();
  };
  issue(0, 0);

  // the query tile: the plain part as it is, the rotated part rotated; rows beyond the end are zero
  bf16* qs = smem + STAGE;
  for (int i = threadIdx.x; i < ROWS * plain_pieces; i += THREADS) {
    const int r = i / plain_pieces, c = i % plain_pieces;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (tile * ROWS + r < q_len)
      v = *reinterpret_cast<const uint4*>(a.q + (size_t)(row0 + tile * ROWS + r) * a.q_stride + (size_t)h * D + c * 8);
    *reinterpret_cast<uint4*>(qs + r * KP + c * 8) = v;
  }
  const int half = rot / 2;
  for (int i = threadIdx.x; i < ROWS * half; i += THREADS) {
    const int r = i / half, c = i % half;
    uint32_t out = 0u;
    if (tile * ROWS + r < q_len) {
      const __nv_bfloat162 uv = *reinterpret_cast<const __nv_bfloat162*>(
          a.q + (size_t)(row0 + tile * ROWS + r) * a.q_stride + (size_t)h * D + plain + 2 * c);
      const float p = (float)(start + tile * ROWS + r), fh = a.inv_freq[c], fl = a.inv_freq[half + c];
      const float ang = __fmul_rn(p, fh);
      const float e = fmaf(p, fh, -ang) + p * fl;  // what the float32 product leaves of the angle
      float s0, c0;
      sincosf(ang, &s0, &c0);
      const float sn = fmaf(e, c0, s0) * a.factor, cs = fmaf(-e, s0, c0) * a.factor;
      const float u = __low2float(uv), v = __high2float(uv);
      out = pack_bf16x2(u * cs - v * sn, v * cs + u * sn);
    }
    *reinterpret_cast<uint32_t*>(qs + r * KP + plain + 2 * c) = out;
  }
  __syncthreads();
  uint32_t qf[KSTEPS][4];
#pragma unroll
  for (int kk = 0; kk < KSTEPS; ++kk)
    ldmatrix_x4(qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3],
                qs + (warp * 16 + (lane & 15)) * KP + kk * 16 + (lane >> 4) * 8);
  __syncthreads();  // the query tile gives its place to stage 1

  int pos[2];
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    const int r = tile * ROWS + warp * 16 + g + 8 * hh;
    pos[hh] = r < q_len ? start + r : -1;
  }
  const int warp_first = start + tile * ROWS + warp * 16;  // the warp's least position (if its rows exist)
  float o[VTILES][4];
#pragma unroll
  for (int n = 0; n < VTILES; ++n)
#pragma unroll
    for (int c = 0; c < 4; ++c) o[n][c] = 0.f;

  for (int j = 0; j < steps; ++j) {
    const int stage = j & 1;
    if (j + 1 < steps) {
      issue(j + 1, stage ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const bf16* ks = smem + stage * STAGE;
    const bf16* vs = ks + KEYS * KP;
    const int key0 = j * KEYS;
    if (key0 <= warp_first + 15) {  // a warp whose rows see none of these keys has nothing to do
      float s[8][4];
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c) s[n][c] = 0.f;
#pragma unroll
      for (int kk = 0; kk < KSTEPS; ++kk)
#pragma unroll
        for (int n = 0; n < 8; n += 2) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(b0, b1, b2, b3, ks + (n * 8 + ((lane >> 4) << 3) + (lane & 7)) * KP + kk * 16 + ((lane >> 3) & 1) * 8);
          mma_bf16_16816(s[n], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], b0, b1);
          mma_bf16_16816(s[n + 1], qf[kk][0], qf[kk][1], qf[kk][2], qf[kk][3], b2, b3);
        }
      const bool whole = key0 + KEYS - 1 <= warp_first && warp_first + 15 < total;
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int c = 0; c < 4; ++c)
          s[n][c] = (whole || key0 + n * 8 + 2 * t4 + (c & 1) <= pos[c >> 1]) ? s[n][c] * a.scale_log2 : -INFINITY;
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        float mx = -INFINITY;
#pragma unroll
        for (int n = 0; n < 8; ++n) mx = fmaxf(mx, fmaxf(s[n][2 * hh], s[n][2 * hh + 1]));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
        mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
        const float m_new = fmaxf(m[hh], mx);
        const float m_safe = m_new == -INFINITY ? 0.f : m_new;
        const float alpha = fast_exp2(m[hh] - m_safe);
        float sum = 0.f;
#pragma unroll
        for (int n = 0; n < 8; ++n) {
          s[n][2 * hh] = fast_exp2(s[n][2 * hh] - m_safe);
          s[n][2 * hh + 1] = fast_exp2(s[n][2 * hh + 1] - m_safe);
          sum += s[n][2 * hh] + s[n][2 * hh + 1];
        }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        sum += __shfl_xor_sync(0xffffffffu, sum, 2);
        l[hh] = l[hh] * alpha + sum;
        m[hh] = m_new;
#pragma unroll
        for (int n = 0; n < VTILES; ++n) {
          o[n][2 * hh] *= alpha;
          o[n][2 * hh + 1] *= alpha;
        }
      }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {  // 16 keys a step; weights as two halves
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int f = 0; f < 4; ++f) {
          const float x = s[2 * kk + (f >> 1)][2 * (f & 1)], y = s[2 * kk + (f >> 1)][2 * (f & 1) + 1];
          const float xh = __bfloat162float(__float2bfloat16_rn(x)), yh = __bfloat162float(__float2bfloat16_rn(y));
          hi[f] = pack_bf16x2(xh, yh);
          lo[f] = pack_bf16x2(x - xh, y - yh);
        }
#pragma unroll
        for (int n = 0; n < VTILES; n += 2) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(b0, b1, b2, b3, vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VP + (n + (lane >> 4)) * 8);
          mma_bf16_16816(o[n], hi[0], hi[1], hi[2], hi[3], b0, b1);
          mma_bf16_16816(o[n], lo[0], lo[1], lo[2], lo[3], b0, b1);
          mma_bf16_16816(o[n + 1], hi[0], hi[1], hi[2], hi[3], b2, b3);
          mma_bf16_16816(o[n + 1], lo[0], lo[1], lo[2], lo[3], b2, b3);
        }
      }
    }
    __syncthreads();  // the stage is free for the load after next
  }
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    if (pos[hh] < 0) continue;
    const size_t r = (size_t)row0 + tile * ROWS + warp * 16 + g + 8 * hh;
    const float inv = a.out_scale / l[hh];
    const bf16* gp = a.gate + r * a.gate_stride + (size_t)h * DV;
    bf16* op = a.out + r * a.out_stride + (size_t)h * DV;
#pragma unroll
    for (int n = 0; n < VTILES; ++n) {
      const int c = n * 8 + 2 * t4;
      const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gp + c));
      *reinterpret_cast<uint32_t*>(op + c) =
          pack_bf16x2(o[n][2 * hh] * inv / (1.0f + expf(-z.x)), o[n][2 * hh + 1] * inv / (1.0f + expf(-z.y)));
    }
  }
}

}  // namespace

// out, gate: first column of the result and of the gate (4-byte aligned rows); q, kv, rows: 16-byte aligned rows; plain,
// rot = D - plain, rank multiples of 8
KRK_API int krk_latent_prefill(void* out, int out_stride, float out_scale, const void* q, int q_stride, int H, int plain,
                               const void* kv, const void* rows, int row_width, int rank, const float* inv_freq, float factor,
                               float scale, int n_seqs, int max_q_len, const int* seq_start, const int* seq_qlen,
                               const int* cu_q, const int* offsets, const void* gate, int gate_stride, cudaStream_t stream) {
  if (n_seqs == 0 || max_q_len == 0) return 0;
  if (plain % 8 || (D - plain) % 8 || plain > D || rank % 8 || row_width % 8 || q_stride % 8 || (out_stride & 1) ||
      (gate_stride & 1) || (((uintptr_t)q | (uintptr_t)kv | (uintptr_t)rows) & 15) || (((uintptr_t)out | (uintptr_t)gate) & 3))
    return -2;
  if (H > 65535 || n_seqs > 65535) return -3;
  Args a;
  a.out = (bf16*)out; a.out_stride = out_stride; a.out_scale = out_scale; a.q = (const bf16*)q; a.q_stride = q_stride; a.H = H;
  a.plain = plain; a.kv = (const bf16*)kv; a.rows = (const bf16*)rows; a.row_width = row_width; a.rank = rank;
  a.inv_freq = inv_freq; a.factor = factor; a.scale_log2 = scale * LOG2E; a.seq_start = seq_start; a.seq_qlen = seq_qlen;
  a.cu_q = cu_q; a.offsets = offsets; a.gate = (const bf16*)gate; a.gate_stride = gate_stride;
  constexpr size_t smem = 2 * (size_t)KEYS * (KP + VP) * sizeof(bf16);
  static_assert(smem <= 220 * 1024, "two stages of keys and values fit a block's shared memory");
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(latent_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const dim3 grid((unsigned)((max_q_len + ROWS - 1) / ROWS), (unsigned)H, (unsigned)n_seqs);
  return (int)launch_pdl(latent_prefill_kernel, grid, dim3(THREADS), smem, stream, a);
}
