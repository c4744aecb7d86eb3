// The recurrences of matrix_memory.cu over a step's many tokens in chunks of 64, on the tensor cores (mma.sync m16n8k16,
// bfloat16 in, float32 accumulate). Within a chunk, with the state S before it,
//
//   y_t = r_t (q_t . S) + sum_{s <= t} A_ts v_s ,   S' = R S + sum_s (w_s k_s) v_s^T
//
// Per-channel decays (c_t: the log decays summed from the chunk's first token to t): A_ts = (q_t e^{c_t}) . (k_s e^{-c_s}),
// q_t . S is (q_t e^{c_t}) . S, w_s = e^{c_last - c_s}, R = e^{c_last} per key channel. Gated by a running maximum (F_t: the
// log forget gates summed likewise, i_s the log input gates, m the maximum): A_ts = (q_t . k_s) e^{F_t - F_s + i_s - m_t},
// r_t = e^{F_t + m_before - m_t}, w_s = e^{F_last - F_s + i_s - m_last}, R = e^{F_last + m_before - m_last}; the vector n
// beside S is one more value column whose v is 1, and its y is what the gated kind divides by.
//
// q, k and v are bfloat16 already, so a product of two of them is exact. Every operand that is not (decayed queries and
// keys, A, the state) is handed to the tensor cores as three bfloat16 terms that add up to it (24 bits of mantissa); where
// both sides are such sums, the six products that matter in 32-bit are formed. So the arithmetic is that of float32 with the
// sums grouped by chunks.
//
// e^{-c_s} overflows where a chunk forgets everything: where a channel's decay over the chunk passes e^-40 the chunk's A is
// formed pair by pair from e^{c_t - c_s} on the CUDA cores instead (right for any decay, and slow).
//
// Three passes: (1) every chunk's own sum_s (w_s k_s) v_s^T; (2) the walk over a sequence's chunks, which leaves every
// chunk its starting state and the sequence its final one; (3) the outputs. A block takes some slices of 64 value
// columns of one (sequence, chunk, head).
#include "mma.cuh"

namespace {

constexpr int L = 64;        // tokens per chunk
constexpr int PB = 64;       // value columns per block
constexpr int VPITCH = PB + 8;
constexpr int APITCH = L + 8;
constexpr int THREADS = 256;
constexpr float SAFE = 40.f;

__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

struct ChunkArgs {
  const bf16 *q, *k, *v;
  int q_stride, k_stride, v_stride;
  float q_scale;
  const float* cum;     // [rows, H * N]: log decays summed within the chunk (per-channel kind); or null
  const float4* gates;  // [rows, H]: (f, i, m before, m after) (gated kind); or null
  float *state, *nm;    // [slots, H, N, P], [slots, H, N + 1]
  float* y;             // [rows, H, P]
  float* den;           // [rows, H]: n . q (gated kind)
  float* cs;            // [n_seqs, max_chunks, H, N * P + (gated ? N : 0)]: chunk sums, then chunk starts
  float* cd;            // [n_seqs, max_chunks, H, N]: a chunk's decays
  int H, N, P, max_chunks;
  int slices;  // column slices a block walks
  const int *cu_q, *seq_qlen, *seq_slot;
};

// x and y as three pairs of bfloat16 terms each
__device__ __forceinline__ void split3_pair(float x, float y, uint32_t (&t)[3]) {
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    const float xa = __bfloat162float(__float2bfloat16_rn(x)), ya = __bfloat162float(__float2bfloat16_rn(y));
    t[i] = pack_bf16x2(xa, ya);
    x -= xa;
    y -= ya;
  }
}
// eight consecutive floats as three terms of eight bfloat16 each, 16 bytes a term
__device__ __forceinline__ void split3_store8(const float (&f)[8], bf16* dst, size_t apart) {
  uint32_t t[4][3];
#pragma unroll
  for (int j = 0; j < 4; ++j) split3_pair(f[2 * j], f[2 * j + 1], t[j]);
#pragma unroll
  for (int i = 0; i < 3; ++i) *reinterpret_cast<uint4*>(dst + i * apart) = make_uint4(t[0][i], t[1][i], t[2][i], t[3][i]);
}
__device__ __forceinline__ void widen8(const bf16* p, float (&f)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int j = 0; j < 4; ++j) { f[2 * j] = __low2float(h[j]); f[2 * j + 1] = __high2float(h[j]); }
}

// F[t] = sum of f over the chunk's tokens 0..t (64 of them, zero beyond the last), by one warp
__device__ __forceinline__ void chunk_sums(float* F, const float* f, int lane) {
  const float a = f[2 * lane], b = a + f[2 * lane + 1];
  float run = b;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const float p = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run += p;
  }
  const float before = run - b;  // exact enough: log gates of one chunk
  F[2 * lane] = before + a;
  F[2 * lane + 1] = before + b;
}

__device__ __forceinline__ void load_values(bf16* vs, const ChunkArgs& a, size_t row0, int h, int p0, int nt) {
  for (int i = threadIdx.x; i < L * (PB / 8); i += THREADS) {
    const int s = i / (PB / 8), c = (i % (PB / 8)) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (s < nt && p0 + c < a.P) v = *reinterpret_cast<const uint4*>(a.v + (row0 + s) * a.v_stride + (size_t)h * a.P + p0 + c);
    *reinterpret_cast<uint4*>(vs + s * VPITCH + c) = v;
  }
}

// ---- pass 1: the chunk's own sum of (w k) v^T, and its decays ------------------------------------------------
template <bool GATED>
__global__ void __launch_bounds__(THREADS) chunk_sum_kernel(ChunkArgs a) {
  extern __shared__ __align__(16) bf16 sm[];
  __shared__ float fs[L], is_[L], Fs[L], ws[L];
  const int N = a.N, P = a.P, H = a.H, NP = N + 8;
  bf16* kt = sm;                          // [3][L][NP]
  bf16* vs = kt + 3 * (size_t)L * NP;     // [L][VPITCH]
  const int h = blockIdx.y % H, chunk = blockIdx.y / H, seq = blockIdx.z;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  grid_launch_dependents();
  grid_dependency_wait();
  const int nt = min(L, a.seq_qlen[seq] - chunk * L);
  if (nt <= 0) return;
  const size_t row0 = (size_t)a.cu_q[seq] + chunk * L;
  float m_before = 0.f, m_last = 0.f;
  if (GATED) {
    if (threadIdx.x < L) {
      const float4 g = threadIdx.x < nt ? a.gates[(row0 + threadIdx.x) * H + h] : make_float4(0.f, -INFINITY, 0.f, 0.f);
      fs[threadIdx.x] = g.x;
      is_[threadIdx.x] = g.y;
    }
    m_before = a.gates[row0 * H + h].z;
    m_last = a.gates[(row0 + nt - 1) * H + h].w;
    __syncthreads();
    if (warp == 0) {
      chunk_sums(Fs, fs, lane);
      __syncwarp();
      for (int s = lane; s < L; s += 32) ws[s] = s < nt ? expf(Fs[L - 1] - Fs[s] + is_[s] - m_last) : 0.f;
    }
    __syncthreads();
  }
  const float* cum_last = GATED ? nullptr : a.cum + (row0 + nt - 1) * H * N + (size_t)h * N;
  for (int i = threadIdx.x; i < L * (N / 8); i += THREADS) {
    const int s = i / (N / 8), n = (i % (N / 8)) * 8;
    float f[8];
    if (s < nt) {
      widen8(a.k + (row0 + s) * a.k_stride + (size_t)h * N + n, f);
      if (GATED) {
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] *= ws[s];
      } else {
        const float* c = a.cum + (row0 + s) * H * N + (size_t)h * N + n;
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] *= expf(cum_last[n + j] - c[j]);
      }
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = 0.f;
    }
    split3_store8(f, kt + s * NP + n, (size_t)L * NP);
  }
  __syncthreads();
  const size_t at = ((size_t)seq * a.max_chunks + chunk) * H + h;
  float* cs = a.cs + at * ((size_t)N * P + (GATED ? N : 0));
  if (blockIdx.x == 0) {
    for (int n = threadIdx.x; n < N; n += THREADS) {
      a.cd[at * N + n] = GATED ? expf(Fs[L - 1] + m_before - m_last) : expf(cum_last[n]);
      if (GATED) {
        float d = 0.f;
        for (int s = 0; s < nt; ++s) {
          const bf16* t = kt + s * NP + n;
          d += (__bfloat162float(t[2 * (size_t)L * NP]) + __bfloat162float(t[(size_t)L * NP])) + __bfloat162float(t[0]);
        }
        cs[(size_t)N * P + n] = d;
      }
    }
  }
  for (int slice = blockIdx.x * a.slices; slice < (int)(blockIdx.x + 1) * a.slices && slice * PB < P; ++slice) {
  const int p0 = slice * PB;
  __syncthreads();  // the values of the slice before are no longer read
  load_values(vs, a, row0, h, p0, nt);
  __syncthreads();
  for (int m0 = warp * 16; m0 < N; m0 += 16 * (THREADS / 32)) {
    float acc[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) acc[n][c] = 0.f;
#pragma unroll
    for (int ks = 0; ks < L / 16; ++ks) {
      uint32_t af[3][4];
#pragma unroll
      for (int t = 0; t < 3; ++t)  // the transpose of k's rows
        ldmatrix_x4_trans(af[t][0], af[t][1], af[t][2], af[t][3],
                          kt + t * (size_t)L * NP + (ks * 16 + (lane & 7) + ((lane >> 4) & 1) * 8) * NP + m0 + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int n = 0; n < 8; n += 2) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(b0, b1, b2, b3, vs + (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VPITCH + (n + (lane >> 4)) * 8);
#pragma unroll
        for (int t = 2; t >= 0; --t) {
          mma_bf16_16816(acc[n], af[t][0], af[t][1], af[t][2], af[t][3], b0, b1);
          mma_bf16_16816(acc[n + 1], af[t][0], af[t][1], af[t][2], af[t][3], b2, b3);
        }
      }
    }
    const int g = lane >> 2, t4 = lane & 3;
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const int p = p0 + n * 8 + 2 * t4;
      if (p < P) {
        *reinterpret_cast<float2*>(cs + (size_t)(m0 + g) * P + p) = make_float2(acc[n][0], acc[n][1]);
        *reinterpret_cast<float2*>(cs + (size_t)(m0 + g + 8) * P + p) = make_float2(acc[n][2], acc[n][3]);
      }
    }
  }
  }
}

// ---- pass 2: a sequence's chunks in order, four neighbouring elements of the state a thread ------------------
template <bool GATED>
__global__ void chunk_walk_kernel(ChunkArgs a) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int h = blockIdx.y, seq = blockIdx.z;
  const int qlen = a.seq_qlen[seq];
  if (qlen <= 0) return;
  const int n_chunks = (qlen + L - 1) / L;
  const size_t NP = (size_t)a.N * a.P, all = NP + (GATED ? a.N : 0);
  const size_t e = 4 * ((size_t)blockIdx.x * blockDim.x + threadIdx.x);
  if (e >= all) return;
  const bool matrix = e < NP;
  const int n = (int)(matrix ? e / a.P : e - NP);  // the gated kind's decay is one number for all n
  const size_t head = (size_t)a.seq_slot[seq] * a.H + h;
  float* st = matrix ? a.state + head * NP + e : a.nm + head * (a.N + 1) + n;
  float4 run = matrix ? *reinterpret_cast<const float4*>(st) : make_float4(st[0], st[1], st[2], st[3]);
  float4* cs = reinterpret_cast<float4*>(a.cs + ((size_t)seq * a.max_chunks * a.H + h) * all + e);
  const float* cd = a.cd + ((size_t)seq * a.max_chunks * a.H + h) * a.N + n;
  const size_t step = (size_t)a.H * all / 4, dstep = (size_t)a.H * a.N;
  for (int c0 = 0; c0 < n_chunks; c0 += 8) {
    float4 own[8];
    float decay[8];
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (c0 + i < n_chunks) {
        own[i] = __ldcg(cs + (size_t)(c0 + i) * step);
        decay[i] = __ldcg(cd + (size_t)(c0 + i) * dstep);
      }
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (c0 + i < n_chunks) {
        cs[(size_t)(c0 + i) * step] = run;
        run.x = fmaf(decay[i], run.x, own[i].x);
        run.y = fmaf(decay[i], run.y, own[i].y);
        run.z = fmaf(decay[i], run.z, own[i].z);
        run.w = fmaf(decay[i], run.w, own[i].w);
      }
  }
  if (matrix) {
    *reinterpret_cast<float4*>(st) = run;
  } else {
    st[0] = run.x; st[1] = run.y; st[2] = run.z; st[3] = run.w;
  }
}

// ---- pass 3: the outputs -------------------------------------------------------------------------------------
// A is formed once per block, each warp one quarter of the tokens against one half of the earlier ones, and left in shared
// memory; then the block walks its column slices.
template <bool GATED>
__global__ void __launch_bounds__(THREADS) chunk_output_kernel(ChunkArgs a) {
  extern __shared__ __align__(16) bf16 sm[];
  __shared__ float fs[L], is_[L], Fs[L], ms[L], den[2][L];
  const int N = a.N, P = a.P, H = a.H, NP = N + 8;
  constexpr int TERMS = GATED ? 1 : 3;  // of a query's and a key's row in shared memory
  const size_t q_apart = (size_t)L * NP, s_apart = (size_t)N * VPITCH;
  bf16* qs = sm;                       // [TERMS][L][NP]
  bf16* as = qs + TERMS * q_apart;     // [3][L][APITCH]: A
  bf16* vs = as + 3 * L * APITCH;      // [L][VPITCH]
  bf16* ks = vs + L * VPITCH;          // [TERMS][L][NP]; the state takes its place
  bf16* ss = ks;                       // [3][N][VPITCH]
  const int h = blockIdx.y % H, chunk = blockIdx.y / H, seq = blockIdx.z;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int mt = warp & 3, half = warp >> 2;  // 16 tokens; 32 earlier tokens, later 32 of a slice's columns
  const int g = lane >> 2, t4 = lane & 3;
  grid_launch_dependents();
  grid_dependency_wait();
  const int nt = min(L, a.seq_qlen[seq] - chunk * L);
  if (nt <= 0) return;
  const size_t row0 = (size_t)a.cu_q[seq] + chunk * L;
  const float* start = a.cs + (((size_t)seq * a.max_chunks + chunk) * H + h) * ((size_t)N * P + (GATED ? N : 0));
  float m_before = 0.f;
  bool safe = true;

  if (GATED) {
    if (threadIdx.x < L) {
      const float4 gt = threadIdx.x < nt ? a.gates[(row0 + threadIdx.x) * H + h] : make_float4(0.f, -INFINITY, 0.f, 0.f);
      fs[threadIdx.x] = gt.x;
      is_[threadIdx.x] = gt.y;
      ms[threadIdx.x] = gt.w;
    }
    m_before = a.gates[row0 * H + h].z;
    for (int i = threadIdx.x; i < 2 * L * (N / 8); i += THREADS) {
      const int s = (i / (N / 8)) % L, n = (i % (N / 8)) * 8;
      const bool is_k = i >= L * (N / 8);
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (s < nt) v = *reinterpret_cast<const uint4*>((is_k ? a.k + (row0 + s) * a.k_stride : a.q + (row0 + s) * a.q_stride) + (size_t)h * N + n);
      *reinterpret_cast<uint4*>((is_k ? ks : qs) + s * NP + n) = v;
    }
    __syncthreads();
    if (warp == 0) chunk_sums(Fs, fs, lane);
  } else {
    const float* cl = a.cum + (row0 + nt - 1) * H * N + (size_t)h * N;
    int over = 0;
    for (int n = threadIdx.x; n < N; n += THREADS) over |= !(cl[n] > -SAFE);
    safe = !__syncthreads_or(over);
    for (int i = threadIdx.x; i < L * (N / 8); i += THREADS) {
      const int s = i / (N / 8), n = (i % (N / 8)) * 8;
      float f[8], k8[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = k8[j] = 0.f;
      if (s < nt) {
        const float4* c4 = reinterpret_cast<const float4*>(a.cum + (row0 + s) * H * N + (size_t)h * N + n);
        const float4 c0 = c4[0], c1 = c4[1];
        const float e[8] = {c0.x, c0.y, c0.z, c0.w, c1.x, c1.y, c1.z, c1.w};
        widen8(a.q + (row0 + s) * a.q_stride + (size_t)h * N + n, f);
        if (safe) widen8(a.k + (row0 + s) * a.k_stride + (size_t)h * N + n, k8);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] *= expf(e[j]);
        if (safe) {
#pragma unroll
          for (int j = 0; j < 8; ++j) k8[j] *= expf(-e[j]);
        }
      }
      split3_store8(f, qs + s * NP + n, q_apart);
      if (safe) split3_store8(k8, ks + s * NP + n, q_apart);
    }
  }
  __syncthreads();

  // A: the warp's 16 tokens against 32 of the chunk's (a tile of later tokens stays zero and is not read)
  float s[4][4];
#pragma unroll
  for (int n = 0; n < 4; ++n)
#pragma unroll
    for (int c = 0; c < 4; ++c) s[n][c] = 0.f;
  const int u0 = half * 32;
  if (safe) {
    for (int kk = 0; kk < N / 16; ++kk) {
      if (u0 >= mt * 16 + 16) break;
      uint32_t af[TERMS][4];
#pragma unroll
      for (int t = 0; t < TERMS; ++t)
        ldmatrix_x4(af[t][0], af[t][1], af[t][2], af[t][3], qs + t * q_apart + (mt * 16 + (lane & 15)) * NP + kk * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int n = 0; n < 4; n += 2) {
        if (u0 + n * 8 >= mt * 16 + 16) break;  // later tokens
        uint32_t b[TERMS][4];
#pragma unroll
        for (int t = 0; t < TERMS; ++t)
          ldmatrix_x4(b[t][0], b[t][1], b[t][2], b[t][3],
                      ks + t * q_apart + (u0 + n * 8 + ((lane >> 4) << 3) + (lane & 7)) * NP + kk * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int sum = TERMS == 1 ? 0 : 2; sum >= 0; --sum)  // small terms first
#pragma unroll
          for (int t = 0; t <= sum; ++t) {
            mma_bf16_16816(s[n], af[t][0], af[t][1], af[t][2], af[t][3], b[sum - t][0], b[sum - t][1]);
            mma_bf16_16816(s[n + 1], af[t][0], af[t][1], af[t][2], af[t][3], b[sum - t][2], b[sum - t][3]);
          }
      }
    }
  } else {
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        const int t = mt * 16 + g + 8 * (c >> 1), u = u0 + n * 8 + 2 * t4 + (c & 1);
        if (u > t || t >= nt) continue;
        const bf16* qr = a.q + (row0 + t) * a.q_stride + (size_t)h * N;
        const bf16* kr = a.k + (row0 + u) * a.k_stride + (size_t)h * N;
        const float* ct = a.cum + (row0 + t) * H * N + (size_t)h * N;
        const float* cu = a.cum + (row0 + u) * H * N + (size_t)h * N;
        float d = 0.f;
        for (int j = 0; j < N; ++j) d += __bfloat162float(qr[j]) * __bfloat162float(kr[j]) * expf(ct[j] - cu[j]);
        s[n][c] = d;
      }
  }
  float rows[2] = {a.q_scale, a.q_scale};  // what q . S is multiplied by
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    const int t = mt * 16 + g + 8 * hh;
    float sum = 0.f;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      float v[2];
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const int u = u0 + n * 8 + 2 * t4 + c;
        v[c] = 0.f;
        if (u <= t && t < nt) {
          v[c] = s[n][2 * hh + c] * a.q_scale;
          if (GATED) v[c] *= expf(Fs[t] - Fs[u] + is_[u] - ms[t]);
        }
        sum += v[c];
      }
      uint32_t p[3];
      split3_pair(v[0], v[1], p);
#pragma unroll
      for (int i = 0; i < 3; ++i)
        *reinterpret_cast<uint32_t*>(as + (i * L + t) * APITCH + u0 + n * 8 + 2 * t4) = p[i];
    }
    if (GATED) {
      rows[hh] *= t < nt ? expf(Fs[t] + m_before - ms[t]) : 0.f;
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      if (t4 == 0) den[half][t] = sum;
    }
  }
  __syncthreads();  // A is complete, and the keys are no longer read
  if (GATED && blockIdx.x == 0) {
    const float* n0 = start + (size_t)N * P;
    for (int t = warp; t < nt; t += THREADS / 32) {
      float d = 0.f;
      for (int n = lane; n < N; n += 32) d += __bfloat162float(qs[t * NP + n]) * n0[n];
      d = warp_sum(d);
      if (lane == 0)
        a.den[(row0 + t) * H + h] = den[0][t] + den[1][t] + a.q_scale * expf(Fs[t] + m_before - ms[t]) * d;
    }
  }

  for (int slice = blockIdx.x * a.slices; slice < (int)(blockIdx.x + 1) * a.slices && slice * PB < P; ++slice) {
    const int p0 = slice * PB;
    load_values(vs, a, row0, h, p0, nt);
    for (int i = threadIdx.x; i < N * (PB / 8); i += THREADS) {
      const int n = i / (PB / 8), c = (i % (PB / 8)) * 8;
      float f[8];
      if (p0 + c < P) {
        const float4 x = __ldcg(reinterpret_cast<const float4*>(start + (size_t)n * P + p0 + c));
        const float4 y = __ldcg(reinterpret_cast<const float4*>(start + (size_t)n * P + p0 + c + 4));
        f[0] = x.x; f[1] = x.y; f[2] = x.z; f[3] = x.w; f[4] = y.x; f[5] = y.y; f[6] = y.z; f[7] = y.w;
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = 0.f;
      }
      split3_store8(f, ss + n * VPITCH + c, s_apart);
    }
    __syncthreads();
    float acc[4][4];
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) acc[n][c] = 0.f;
    for (int kk = 0; kk < N / 16; ++kk) {
      uint32_t af[TERMS][4];
#pragma unroll
      for (int t = 0; t < TERMS; ++t)
        ldmatrix_x4(af[t][0], af[t][1], af[t][2], af[t][3], qs + t * q_apart + (mt * 16 + (lane & 15)) * NP + kk * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int n = 0; n < 4; n += 2) {
        uint32_t b[3][4];
#pragma unroll
        for (int t = 0; t < 3; ++t)
          ldmatrix_x4_trans(b[t][0], b[t][1], b[t][2], b[t][3],
                            ss + t * s_apart + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VPITCH + (half * 4 + n + (lane >> 4)) * 8);
#pragma unroll
        for (int sum = 2; sum >= 0; --sum)
#pragma unroll
          for (int t = 0; t < TERMS; ++t) {
            if (sum - t < 0) continue;
            mma_bf16_16816(acc[n], af[t][0], af[t][1], af[t][2], af[t][3], b[sum - t][0], b[sum - t][1]);
            mma_bf16_16816(acc[n + 1], af[t][0], af[t][1], af[t][2], af[t][3], b[sum - t][2], b[sum - t][3]);
          }
      }
    }
#pragma unroll
    for (int n = 0; n < 4; ++n)
#pragma unroll
      for (int c = 0; c < 4; ++c) acc[n][c] *= rows[c >> 1];
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      if (kk > mt) break;  // later tokens
      uint32_t af[3][4];
#pragma unroll
      for (int t = 0; t < 3; ++t)
        ldmatrix_x4(af[t][0], af[t][1], af[t][2], af[t][3], as + (t * L + mt * 16 + (lane & 15)) * APITCH + kk * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int n = 0; n < 4; n += 2) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(b0, b1, b2, b3, vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VPITCH + (half * 4 + n + (lane >> 4)) * 8);
#pragma unroll
        for (int t = 2; t >= 0; --t) {
          mma_bf16_16816(acc[n], af[t][0], af[t][1], af[t][2], af[t][3], b0, b1);
          mma_bf16_16816(acc[n + 1], af[t][0], af[t][1], af[t][2], af[t][3], b2, b3);
        }
      }
    }
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int t = mt * 16 + g + 8 * hh;
      if (t >= nt) continue;
      float* yr = a.y + ((row0 + t) * H + h) * P;
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        const int p = p0 + half * 32 + n * 8 + 2 * t4;
        if (p < P) *reinterpret_cast<float2*>(yr + p) = make_float2(acc[n][2 * hh], acc[n][2 * hh + 1]);
      }
    }
    __syncthreads();  // the state and the values make room for the next slice's
  }
}

// ---- log decays summed within chunks -------------------------------------------------------------------------
// cum[row, c]: sum over the chunk's tokens up to the row's of logsigmoid(z) / tau, z = W2 lora + bias
__global__ void chunk_decays_kernel(float* __restrict__ cum, const bf16* __restrict__ lora, int lora_stride,
                                    const bf16* __restrict__ w2, const float* __restrict__ bias, float inv_tau, int channels,
                                    int R, const int* __restrict__ cu_q, const int* __restrict__ seq_qlen) {
  extern __shared__ __align__(16) float ls[];  // [L][R]
  grid_launch_dependents();
  grid_dependency_wait();
  const int chunk = blockIdx.y, seq = blockIdx.z;
  const int nt = min(L, seq_qlen[seq] - chunk * L);
  if (nt <= 0) return;
  const size_t row0 = (size_t)cu_q[seq] + chunk * L;
  for (int i = threadIdx.x; i < nt * R; i += blockDim.x) ls[i] = __bfloat162float(lora[(row0 + i / R) * lora_stride + i % R]);
  __syncthreads();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= channels) return;
  const float b = bias[c];
  float run = 0.f;
  for (int t0 = 0; t0 < nt; t0 += 16) {
    float z[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) z[t] = b;
    for (int m = 0; m < R; ++m) {
      const float w = __bfloat162float(w2[(size_t)c * R + m]);
#pragma unroll
      for (int t = 0; t < 16; ++t) z[t] += w * ls[min(t0 + t, nt - 1) * R + m];
    }
#pragma unroll
    for (int t = 0; t < 16; ++t)
      if (t0 + t < nt) {
        run += log_sigmoid_f(z[t]) * inv_tau;
        cum[(row0 + t0 + t) * channels + c] = run;
      }
  }
}

size_t sum_smem(int N) { return (3 * (size_t)L * (N + 8) + (size_t)L * VPITCH) * sizeof(bf16); }
size_t output_smem(int N, bool gated) {
  const size_t terms = gated ? 1 : 3, rows = terms * L * (N + 8), state = 3 * (size_t)N * VPITCH;
  return (rows + 3 * (size_t)L * APITCH + (size_t)L * VPITCH + (state > rows ? state : rows)) * sizeof(bf16);
}

template <bool GATED>
int launch_chunks(ChunkArgs a, int n_seqs, cudaStream_t stream) {
  const size_t s1 = sum_smem(a.N), s3 = output_smem(a.N, GATED);
  const long long heads = (long long)a.H * a.max_chunks;
  if (heads > 65535 || n_seqs > 65535) return -2;
  // what a block does before its first slice is done once per block: as many slices a block as leave every SM three
  const int all_slices = (a.P + PB - 1) / PB;
  const long long most = heads * n_seqs * all_slices;
  a.slices = (int)(most / 444 < 1 ? 1 : most / 444 > all_slices ? all_slices : most / 444);
  const dim3 grid((unsigned)((all_slices + a.slices - 1) / a.slices), (unsigned)heads, (unsigned)n_seqs);
  cudaFuncSetAttribute(chunk_sum_kernel<GATED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
  cudaFuncSetAttribute(chunk_output_kernel<GATED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s3);
  int rc = (int)launch_pdl(chunk_sum_kernel<GATED>, grid, dim3(THREADS), s1, stream, a);
  if (rc) return rc;
  const size_t all = (size_t)a.N * a.P + (GATED ? a.N : 0);
  rc = (int)launch_pdl(chunk_walk_kernel<GATED>, dim3((unsigned)((all / 4 + 63) / 64), (unsigned)a.H, (unsigned)n_seqs), dim3(64),
                       0, stream, a);
  if (rc) return rc;
  return (int)launch_pdl(chunk_output_kernel<GATED>, grid, dim3(THREADS), s3, stream, a);
}

}  // namespace

// Tokens per chunk, and whether head sizes are ones that the chunked passes take.
KRK_API int krk_memory_chunk_tokens(int N, int P, int gated) {
  return N % 16 == 0 && P % 16 == 0 && N >= 16 && sum_smem(N) <= 220 * 1024 && output_smem(N, gated != 0) <= 220 * 1024 ? L : 0;
}

KRK_API int krk_memory_chunk_decays(float* cum, const void* lora, int lora_stride, const void* w2, const float* bias, float tau,
                                    int channels, int R, int n_seqs, int max_q_len, const int* cu_q, const int* seq_qlen,
                                    cudaStream_t stream) {
  if (n_seqs == 0 || max_q_len == 0) return 0;
  const size_t smem = (size_t)L * R * sizeof(float);
  const int chunks = (max_q_len + L - 1) / L;
  if (smem > 48 * 1024 || chunks > 65535 || n_seqs > 65535) return -2;
  const dim3 grid((unsigned)((channels + 127) / 128), (unsigned)chunks, (unsigned)n_seqs);
  return (int)launch_pdl(chunk_decays_kernel, grid, dim3(128), smem, stream, cum, (const bf16*)lora, lora_stride, (const bf16*)w2,
                         bias, 1.0f / tau, channels, R, cu_q, seq_qlen);
}

// The scan of krk_memory_scan in chunks, bfloat16. cum (per-channel kind) or gates and nm (gated kind); scratch cs and cd
// for ceil(max_q_len / 64) chunks a sequence. Row starts of q, k and v on 16-byte boundaries.
KRK_API int krk_memory_chunks(float* y, float* den, const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride,
                              float q_scale, const float* cum, const float* gates, float* state, float* nm, float* cs, float* cd,
                              int H, int N, int P, int n_seqs, int max_q_len, const int* cu_q, const int* seq_qlen,
                              const int* seq_slot, cudaStream_t stream) {
  if (n_seqs == 0 || max_q_len == 0) return 0;
  if ((cum == nullptr) == (gates == nullptr) || (gates && (!nm || !den)) || !krk_memory_chunk_tokens(N, P, gates != nullptr) ||
      q_stride % 8 || k_stride % 8 || v_stride % 8 || (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)state | (uintptr_t)cs | (uintptr_t)cum) & 15))
    return -2;
  ChunkArgs a;
  a.q = (const bf16*)q; a.k = (const bf16*)k; a.v = (const bf16*)v; a.q_stride = q_stride; a.k_stride = k_stride;
  a.v_stride = v_stride; a.q_scale = q_scale; a.cum = cum; a.gates = (const float4*)gates; a.state = state; a.nm = nm; a.y = y; a.den = den;
  a.cs = cs; a.cd = cd; a.H = H; a.N = N; a.P = P; a.max_chunks = (max_q_len + L - 1) / L; a.slices = 1;
  a.cu_q = cu_q; a.seq_qlen = seq_qlen; a.seq_slot = seq_slot;
  return gates ? launch_chunks<true>(a, n_seqs, stream) : launch_chunks<false>(a, n_seqs, stream);
}
