// Mixers with a matrix state per head, S [N key channels, P value channels], written without a removal term.
//
//   S <- a S + b k v^T ;  y = S^T q
//
// in two kinds. Per-channel decays (gated linear attention): a = exp(logsigmoid(z) / tau) per key channel with
// z = W2 lora + bias, b = 1. Gated by a running maximum (mLSTM): per token and head i and f are log gates,
// m' = max(f + m, i), a = exp(f + m - m'), b = exp(i - m'), and beside S a vector n <- a n + b k whose product with
// q divides y: y / (max(|n . q|, exp(-m')) + 1e-6). n is treated as one more value column whose v is 1.
//
// krk_memory_gates / krk_memory_decays: what does not depend on the state, for all rows of a step: the gates with the
// running maximum before and after every token (a block per (sequence, head), tokens side by side, composed as
// max-plus maps), or the log decays.
// krk_memory_scan: the state over a step's tokens, one after the other, for any sizes and both element types. A
// block takes a slice of the value columns of one (sequence, head); NS lanes of a warp share a column, each with NPT
// consecutive key channels in registers; q, k and the decays are staged in shared memory sixteen tokens at a time. A
// token's y is each lane's ordered partial sum followed by a fixed exchange, so it depends on (N, P) alone.
// krk_memory_finish: y -> the rows the output projection reads: each head's part divided by its root mean square, times a
// weight, times a gate.
#include "common.cuh"

namespace {

constexpr int TOK = 16;  // tokens staged at a time

__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

struct GateArgs {
  const void* z;  // [rows, 2H]: input gates, then forget gates, before bias and cap
  int z_stride;
  const float* bias;  // [2H]
  float cap;
  float* nm;  // [slots, H, N + 1]: m sits behind n
  int H, N;
  const int *cu_q, *seq_qlen, *seq_slot;
};

template <typename T> __device__ __forceinline__ void gates_of(const GateArgs& a, int row, int h, float* f, float* i) {
  const T* z = reinterpret_cast<const T*>(a.z) + (size_t)row * a.z_stride;
  *i = a.cap * tanhf((to_float<T>(z[h]) + a.bias[h]) / a.cap);
  *f = log_sigmoid_f(a.cap * tanhf((to_float<T>(z[a.H + h]) + a.bias[a.H + h]) / a.cap));
}

// gates [rows, H]: (f, i, m before the token, m after it). A token is the map m -> max(F + m, M); maps compose to maps.
template <typename T>
__global__ void memory_gates_kernel(float4* __restrict__ gates, GateArgs a) {
  __shared__ float wf[32], wm[32];
  grid_launch_dependents();
  grid_dependency_wait();
  const int h = blockIdx.x, seq = blockIdx.y;
  const int n = a.seq_qlen[seq], row0 = a.cu_q[seq];
  if (n <= 0) return;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  float* m_state = a.nm + ((size_t)a.seq_slot[seq] * a.H + h) * (a.N + 1) + a.N;
  float carry = *m_state;
  for (int t0 = 0; t0 < n; t0 += blockDim.x) {
    const int t = t0 + threadIdx.x;
    float f = 0.f, i = -INFINITY;
    if (t < n) gates_of<T>(a, row0 + t, h, &f, &i);
    float F = f, M = i;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float pf = __shfl_up_sync(0xffffffffu, F, o), pm = __shfl_up_sync(0xffffffffu, M, o);
      if (lane >= o) { M = fmaxf(pm + F, M); F += pf; }
    }
    if (lane == 31) { wf[warp] = F; wm[warp] = M; }
    __syncthreads();
    float m = carry;  // before this warp's first token
    for (int w = 0; w < warp; ++w) m = fmaxf(wf[w] + m, wm[w]);
    float next = m;
    for (int w = warp; w < n_warps; ++w) next = fmaxf(wf[w] + next, wm[w]);
    float pf = __shfl_up_sync(0xffffffffu, F, 1), pm = __shfl_up_sync(0xffffffffu, M, 1);
    const float before = lane == 0 ? m : fmaxf(pf + m, pm);
    const float after = fmaxf(f + before, i);
    if (t < n) {
      gates[(size_t)(row0 + t) * a.H + h] = make_float4(f, i, before, after);
      if (t == n - 1) *m_state = after;
    }
    carry = next;
    __syncthreads();
  }
}

constexpr int DECAY_ROWS = 16;

// log decays [rows, channels] of gated linear attention
template <typename T>
__global__ void memory_decays_kernel(float* __restrict__ out, const T* __restrict__ lora, int lora_stride,
                                     const T* __restrict__ w2, const float* __restrict__ bias, float inv_tau, int rows,
                                     int channels, int R) {
  extern __shared__ __align__(16) float ls[];  // [DECAY_ROWS][R]
  grid_launch_dependents();
  grid_dependency_wait();
  const int r0 = blockIdx.x * DECAY_ROWS, nr = min(DECAY_ROWS, rows - r0);
  for (int i = threadIdx.x; i < DECAY_ROWS * R; i += blockDim.x) {
    const int r = i / R, m = i - r * R;
    ls[i] = r < nr ? to_float<T>(lora[(size_t)(r0 + r) * lora_stride + m]) : 0.f;
  }
  __syncthreads();
  const int c = blockIdx.y * blockDim.x + threadIdx.x;
  if (c >= channels) return;
  float z[DECAY_ROWS];
  const float b = bias[c];
#pragma unroll
  for (int r = 0; r < DECAY_ROWS; ++r) z[r] = 0.f;
  for (int m = 0; m < R; ++m) {
    const float w = to_float<T>(w2[(size_t)c * R + m]);
#pragma unroll
    for (int r = 0; r < DECAY_ROWS; ++r) z[r] += w * ls[r * R + m];
  }
#pragma unroll
  for (int r = 0; r < DECAY_ROWS; ++r)
    if (r < nr) out[(size_t)(r0 + r) * channels + c] = log_sigmoid_f(z[r] + b) * inv_tau;
}

struct MemArgs {
  const void *q, *k, *v;
  int q_stride, k_stride, v_stride;
  float q_scale;
  const float* log_decay;  // [rows, H * N]: per-channel decays; or null
  const float4* gates;     // [rows, H]: the gated kind; or null
  float* state;            // [slots, H, N, P]
  float* nm;               // [slots, H, N + 1] (gated kind)
  float* y;                // [rows, H, P]
  float* den;              // [rows, H]: n . q (gated kind)
  int H, N, P;
  const int *cu_q, *seq_qlen, *seq_slot;
};

template <typename T, int NPT, bool GATED>
__global__ void __launch_bounds__(128) memory_scan_kernel(MemArgs a, int NS) {
  extern __shared__ __align__(16) float sm[];
  constexpr int SL = NPT + 4;  // a lane's slice starts this many floats after its neighbour's: other banks
  grid_launch_dependents();
  const int h = blockIdx.y, seq = blockIdx.z;
  const int N = a.N, P = a.P, PT = P + (GATED ? 1 : 0);
  const int VS = NS * SL;
  const int PW = 32 / NS, PB = 4 * PW;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int ns = lane / PW, pl = warp * PW + lane % PW;  // key slice, column within the block
  const int p = blockIdx.x * PB + pl;
  const int n0 = ns * NPT;
  float* qs = sm;                              // [TOK][VS]
  float* ks = qs + TOK * VS;                   // [TOK][VS]
  float* as = ks + TOK * VS;                   // [TOK][VS] (per channel) or [TOK] (gated)
  float* vs = as + (GATED ? TOK : TOK * VS);   // [TOK][PB]
  for (int i = threadIdx.x; i < (GATED ? 2 : 3) * TOK * VS; i += blockDim.x) sm[i] = 0.f;  // beyond N: zero for good
  grid_dependency_wait();
  const int qlen = a.seq_qlen[seq], row0 = a.cu_q[seq];
  if (qlen <= 0) return;
  const size_t head = (size_t)a.seq_slot[seq] * a.H + h;
  float* st = p < P ? a.state + head * N * P + p : (GATED && p == P ? a.nm + head * (N + 1) : nullptr);
  const size_t step = p < P ? P : 1;
  float s[NPT];
#pragma unroll
  for (int j = 0; j < NPT; ++j) s[j] = (st && n0 + j < N) ? st[(size_t)(n0 + j) * step] : 0.f;

  for (int t0 = 0; t0 < qlen; t0 += TOK) {
    const int nt = min(TOK, qlen - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * N; i += blockDim.x) {
      const int t = i / N, n = i - t * N;
      const size_t r = (size_t)(row0 + t0 + t);
      const int at = t * VS + (n / NPT) * SL + (n % NPT);
      qs[at] = to_float<T>(reinterpret_cast<const T*>(a.q)[r * a.q_stride + h * N + n]) * a.q_scale;
      ks[at] = to_float<T>(reinterpret_cast<const T*>(a.k)[r * a.k_stride + h * N + n]);
      if (!GATED) as[at] = expf(a.log_decay[r * a.H * N + h * N + n]);
    }
    for (int i = threadIdx.x; i < nt * PB; i += blockDim.x) {
      const int t = i / PB, c = blockIdx.x * PB + i % PB;
      const size_t r = (size_t)(row0 + t0 + t);
      float v = c < P ? to_float<T>(reinterpret_cast<const T*>(a.v)[r * a.v_stride + h * P + c]) : (c == P ? 1.f : 0.f);
      if (GATED) {
        const float4 g = a.gates[r * a.H + h];
        v *= expf(g.y - g.w);
        if (i % PB == 0) as[t] = expf(g.x + g.z - g.w);
      }
      vs[i] = v;
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float4* q4 = reinterpret_cast<const float4*>(qs + t * VS + ns * SL);
      const float4* k4 = reinterpret_cast<const float4*>(ks + t * VS + ns * SL);
      const float4* a4 = reinterpret_cast<const float4*>(as + t * VS + ns * SL);
      const float v = vs[t * PB + pl];
      const float at = GATED ? as[t] : 0.f;
      float y0 = 0.f, y1 = 0.f;
#pragma unroll
      for (int j = 0; j < NPT / 4; ++j) {
        const float4 q = q4[j], k = k4[j];
        const float4 d = GATED ? make_float4(at, at, at, at) : a4[j];
        s[4 * j] = fmaf(d.x, s[4 * j], k.x * v);
        s[4 * j + 1] = fmaf(d.y, s[4 * j + 1], k.y * v);
        s[4 * j + 2] = fmaf(d.z, s[4 * j + 2], k.z * v);
        s[4 * j + 3] = fmaf(d.w, s[4 * j + 3], k.w * v);
        y0 = fmaf(q.x, s[4 * j], y0);
        y1 = fmaf(q.y, s[4 * j + 1], y1);
        y0 = fmaf(q.z, s[4 * j + 2], y0);
        y1 = fmaf(q.w, s[4 * j + 3], y1);
      }
      float y = y0 + y1;
      for (int o = PW; o < 32; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (ns == 0 && p < PT) {
        const size_t at = (size_t)(row0 + t0 + t) * a.H + h;
        if (p < P) a.y[at * P + p] = y;
        else a.den[at] = y;
      }
    }
  }
#pragma unroll
  for (int j = 0; j < NPT; ++j)
    if (st && n0 + j < N) st[(size_t)(n0 + j) * step] = s[j];
}

// one warp per (row, head), V columns a lane. Gated: y / den, weight [H * P], gate sigmoid; else weight [P], gate silu.
template <typename T, int V> struct alignas(V * sizeof(T)) Cols { T v[V]; };

template <typename T, bool GATED, int V>
__global__ void memory_finish_kernel(T* __restrict__ out, int out_stride, int out_col, float out_scale,
                                     const float* __restrict__ y, const float* __restrict__ den,
                                     const float4* __restrict__ gates, const T* __restrict__ g, int g_stride,
                                     const float* __restrict__ weight, int H, int P, float eps, int rows) {
  grid_launch_dependents();
  grid_dependency_wait();
  const int lane = threadIdx.x & 31;
  const long long w = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (w >= (long long)rows * H) return;
  const size_t row = (size_t)(w / H);
  const int h = (int)(w % H);
  const float* yr = y + (size_t)w * P;
  float inv = 1.f;
  if (GATED) inv = 1.0f / (fmaxf(fabsf(den[w]), expf(-gates[w].w)) + 1e-6f);
  float sq = 0.f;
  for (int p = V * lane; p < P; p += V * 32) {
    const Cols<float, V> c = *reinterpret_cast<const Cols<float, V>*>(yr + p);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const float o = c.v[i] * inv;
      sq += o * o;
    }
  }
  const float factor = rsqrtf(warp_sum(sq) / (float)P + eps) * inv;
  const T* gr = g + row * g_stride + (size_t)h * P;
  const float* wr = weight + (GATED ? (size_t)h * P : 0);
  T* o = out + row * out_stride + out_col + (size_t)h * P;
  for (int p = V * lane; p < P; p += V * 32) {
    const Cols<float, V> c = *reinterpret_cast<const Cols<float, V>*>(yr + p), wt = *reinterpret_cast<const Cols<float, V>*>(wr + p);
    const Cols<T, V> zz = *reinterpret_cast<const Cols<T, V>*>(gr + p);
    Cols<T, V> res;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const float z = to_float<T>(zz.v[i]);
      const float gate = GATED ? sigmoid_f(z) : z * sigmoid_f(z);
      res.v[i] = from_float<T>(c.v[i] * factor * wt.v[i] * gate * out_scale);
    }
    *reinterpret_cast<Cols<T, V>*>(o + p) = res;
  }
}

template <typename T>
int launch_memory_finish(void* out, int out_stride, int out_col, float out_scale, const float* y, const float* den,
                         const float* gates, const void* g, int g_stride, const float* weight, int H, int P, float eps, int rows,
                         cudaStream_t stream) {
  const dim3 grid((unsigned)(((long long)rows * H + 3) / 4));
  const uintptr_t mask = 4 * sizeof(T) - 1;
  const bool vec = P % 4 == 0 && ((out_stride | out_col | g_stride) & 3) == 0 && (((uintptr_t)out | (uintptr_t)g) & mask) == 0 &&
                   (((uintptr_t)y | (uintptr_t)weight) & 15) == 0;
  auto kern = gates ? (vec ? memory_finish_kernel<T, true, 4> : memory_finish_kernel<T, true, 1>)
                    : (vec ? memory_finish_kernel<T, false, 4> : memory_finish_kernel<T, false, 1>);
  return (int)launch_pdl(kern, grid, dim3(128), 0, stream, (T*)out, out_stride, out_col, out_scale, y, den, (const float4*)gates,
                         (const T*)g, g_stride, weight, H, P, eps, rows);
}

template <typename T, bool GATED>
int launch_memory_scan(const MemArgs& a, int n_seqs, cudaStream_t stream) {
  const int N = a.N;
  const int npt = N <= 64 ? 8 : N <= 512 ? 16 : 32;
  int NS = 1;
  while (NS * npt < N) NS <<= 1;
  if (NS > 32) return -2;
  const int PB = 4 * (32 / NS), PT = a.P + (GATED ? 1 : 0);
  const int VS = NS * (npt + 4);
  const size_t smem = ((size_t)(GATED ? 2 : 3) * TOK * VS + (GATED ? TOK : 0) + (size_t)TOK * PB) * sizeof(float);
  if (smem > 200 * 1024 || a.H > 65535 || n_seqs > 65535) return -2;
  const dim3 grid((unsigned)((PT + PB - 1) / PB), (unsigned)a.H, (unsigned)n_seqs);
  auto kern = npt == 8 ? memory_scan_kernel<T, 8, GATED> : npt == 16 ? memory_scan_kernel<T, 16, GATED> : memory_scan_kernel<T, 32, GATED>;
  if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  return (int)launch_pdl(kern, grid, dim3(128), smem, stream, a, NS);
}

}  // namespace

KRK_API int krk_memory_gates(float* gates, const void* z, int z_stride, const float* bias, float cap, float* nm, int H, int N,
                             int n_seqs, int max_q_len, const int* cu_q, const int* seq_qlen, const int* seq_slot, int dtype,
                             cudaStream_t stream) {
  if (n_seqs == 0) return 0;
  GateArgs a;
  a.z = z; a.z_stride = z_stride; a.bias = bias; a.cap = cap; a.nm = nm; a.H = H; a.N = N;
  a.cu_q = cu_q; a.seq_qlen = seq_qlen; a.seq_slot = seq_slot;
  const int threads = min(1024, (max(max_q_len, 1) + 31) / 32 * 32);
  if (n_seqs > 65535) return -3;
  if (dtype == KRK_DTYPE_F32)
    return (int)launch_pdl(memory_gates_kernel<float>, dim3(H, n_seqs), dim3(threads), 0, stream, (float4*)gates, a);
  return (int)launch_pdl(memory_gates_kernel<bf16>, dim3(H, n_seqs), dim3(threads), 0, stream, (float4*)gates, a);
}

KRK_API int krk_memory_decays(float* out, const void* lora, int lora_stride, const void* w2, const float* bias, float tau,
                              int rows, int channels, int R, int dtype, cudaStream_t stream) {
  if (rows == 0) return 0;
  const size_t smem = (size_t)DECAY_ROWS * R * sizeof(float);
  if (smem > 48 * 1024) return -2;
  const dim3 grid((unsigned)((rows + DECAY_ROWS - 1) / DECAY_ROWS), (unsigned)((channels + 127) / 128));
  if (dtype == KRK_DTYPE_F32)
    return (int)launch_pdl(memory_decays_kernel<float>, grid, dim3(128), smem, stream, out, (const float*)lora, lora_stride,
                           (const float*)w2, bias, 1.0f / tau, rows, channels, R);
  return (int)launch_pdl(memory_decays_kernel<bf16>, grid, dim3(128), smem, stream, out, (const bf16*)lora, lora_stride,
                         (const bf16*)w2, bias, 1.0f / tau, rows, channels, R);
}

// gates given: the gated kind (nm too); log_decay given: per-channel decays
KRK_API int krk_memory_scan(float* y, float* den, const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride,
                            float q_scale, const float* log_decay, const float* gates, float* state, float* nm, int H, int N,
                            int P, int n_seqs, const int* cu_q, const int* seq_qlen, const int* seq_slot, int dtype,
                            cudaStream_t stream) {
  if (n_seqs == 0) return 0;
  if ((log_decay == nullptr) == (gates == nullptr) || (gates && (!nm || !den))) return -2;
  MemArgs a;
  a.q = q; a.k = k; a.v = v; a.q_stride = q_stride; a.k_stride = k_stride; a.v_stride = v_stride; a.q_scale = q_scale;
  a.log_decay = log_decay; a.gates = (const float4*)gates; a.state = state; a.nm = nm; a.y = y; a.den = den; a.H = H; a.N = N; a.P = P;
  a.cu_q = cu_q; a.seq_qlen = seq_qlen; a.seq_slot = seq_slot;
  if (dtype == KRK_DTYPE_F32)
    return gates ? launch_memory_scan<float, true>(a, n_seqs, stream) : launch_memory_scan<float, false>(a, n_seqs, stream);
  return gates ? launch_memory_scan<bf16, true>(a, n_seqs, stream) : launch_memory_scan<bf16, false>(a, n_seqs, stream);
}

KRK_API int krk_memory_finish(void* out, int out_stride, int out_col, float out_scale, const float* y, const float* den,
                              const float* gates, const void* g, int g_stride, const float* weight, int H, int P, float eps,
                              int rows, int dtype, cudaStream_t stream) {
  if (rows == 0) return 0;
  if (gates && !den) return -2;
  return dtype == KRK_DTYPE_F32
             ? launch_memory_finish<float>(out, out_stride, out_col, out_scale, y, den, gates, g, g_stride, weight, H, P, eps, rows, stream)
             : launch_memory_finish<bf16>(out, out_stride, out_col, out_scale, y, den, gates, g, g_stride, weight, H, P, eps, rows, stream);
}
