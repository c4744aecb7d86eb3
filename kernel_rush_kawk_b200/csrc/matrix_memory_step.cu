// One token of every sequence through the recurrences of matrix_memory.cu, all of it in one launch: gates or decays, the
// update of the state, the readout, the division, the head's norm, weight and gate.
//
// A cluster of `CS` blocks serves one (sequence, head), each block a slice of the value columns: the state is read and written
// once, a thread taking V neighbouring columns of every R-th row with eight rows in flight. What concerns the whole head (its
// gates, n . q) every block works out for itself; the sum of squares over all columns crosses the blocks through distributed
// shared memory. n and the running maximum are written by the first block after all have read them. A result depends on
// the head's own inputs alone, with the sums' order fixed by the sizes and CS.
#include <cooperative_groups.h>

#include "common.cuh"

namespace cg = cooperative_groups;

namespace {

constexpr int THREADS = 256;
constexpr int FLY = 8;  // rows of the state in flight per thread

__device__ __forceinline__ float log_sigmoid_f(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.0f / (1.0f + expf(-z)); }

struct StepArgs {
  const void *q, *k, *v, *g;
  int q_stride, k_stride, v_stride, g_stride;
  float q_scale;
  const void* z;  // gated: [rows, 2H] gate inputs; per-channel: [rows, R] low-rank decay inputs
  int z_stride;
  const void* w2;     // per-channel: [H * N, R]
  const float* bias;  // gated: [2H]; per-channel: [H * N]
  float cap_or_inv_tau;
  int R;
  float *state, *nm;
  const float* weight;  // gated: [H * P]; per-channel: [P]
  float eps;
  void* out;
  int out_stride, out_col;
  float out_scale;
  int H, N, P, PB;  // PB: value columns per block
  const int* seq_slot;
};

template <int V> struct alignas(4 * V) Cols { float v[V]; };

template <typename T, bool GATED, int V>
__global__ void __launch_bounds__(THREADS) memory_step_kernel(StepArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float scratch[32];
  __shared__ float squares;
  const int N = a.N, P = a.P, H = a.H, PB = a.PB;
  float* qs = sm;             // [N]
  float* ks = qs + N;         // [N]: k, times the input gate
  float* as = ks + N;         // [N]: decays, or the new n
  float* part = as + N;       // [RW][PB]
  cg::cluster_group cluster = cg::this_cluster();
  grid_launch_dependents();
  grid_dependency_wait();
  const int h = blockIdx.y, seq = blockIdx.z;
  const int p0 = blockIdx.x * PB, cols = max(0, min(PB, P - p0));
  const size_t head = (size_t)a.seq_slot[seq] * H + h;
  const T* qr = reinterpret_cast<const T*>(a.q) + (size_t)seq * a.q_stride + (size_t)h * N;
  const T* kr = reinterpret_cast<const T*>(a.k) + (size_t)seq * a.k_stride + (size_t)h * N;
  const T* zr = reinterpret_cast<const T*>(a.z) + (size_t)seq * a.z_stride;
  float* nm = GATED ? a.nm + head * (N + 1) : nullptr;

  // this thread's columns, and its first rows of the state on their way
  const int GW = PB / V, RW = THREADS / GW;
  const int gc = threadIdx.x % GW, r0 = threadIdx.x / GW;
  const bool live = r0 < RW && gc * V < cols;  // with V > 1, P and PB are multiples of V
  float* st = a.state + head * N * P + p0 + gc * V;
  Cols<V> s[FLY];
#pragma unroll
  for (int i = 0; i < FLY; ++i)
    if (live && r0 + i * RW < N) s[i] = *reinterpret_cast<const Cols<V>*>(st + (size_t)(r0 + i * RW) * P);

  float keep = 1.f, take = 1.f, m = 0.f;
  if (GATED) {
    const float i = a.cap_or_inv_tau * tanhf((to_float<T>(zr[h]) + a.bias[h]) / a.cap_or_inv_tau);
    const float f = log_sigmoid_f(a.cap_or_inv_tau * tanhf((to_float<T>(zr[H + h]) + a.bias[H + h]) / a.cap_or_inv_tau));
    const float before = nm[N];
    m = fmaxf(f + before, i);
    keep = expf(f + before - m);
    take = expf(i - m);
  }
  float dot = 0.f;
  for (int n = threadIdx.x; n < N; n += THREADS) {
    const float q = to_float<T>(qr[n]) * a.q_scale, k = to_float<T>(kr[n]) * take;
    qs[n] = q;
    ks[n] = k;
    if (GATED) {
      const float nn = fmaf(keep, nm[n], k);
      as[n] = nn;
      dot += nn * q;
    } else {
      const T* w = reinterpret_cast<const T*>(a.w2) + (size_t)(h * N + n) * a.R;
      float z = 0.f;
      for (int j = 0; j < a.R; ++j) z += to_float<T>(w[j]) * to_float<T>(zr[j]);
      as[n] = expf(log_sigmoid_f(z + a.bias[h * N + n]) * a.cap_or_inv_tau);
    }
  }
  float inv = 1.f;
  if (GATED) inv = 1.0f / (fmaxf(fabsf(block_sum(dot, scratch)), expf(-m)) + 1e-6f);
  float v[V], acc[V];
#pragma unroll
  for (int c = 0; c < V; ++c) {
    v[c] = live ? to_float<T>(reinterpret_cast<const T*>(a.v)[(size_t)seq * a.v_stride + (size_t)h * P + p0 + gc * V + c]) : 0.f;
    acc[c] = 0.f;
  }
  __syncthreads();
  if (live) {
    for (int n0 = r0; n0 < N; n0 += FLY * RW) {
      Cols<V> next[FLY];
#pragma unroll
      for (int i = 0; i < FLY; ++i) {
        const int n = n0 + (FLY + i) * RW;
        if (n < N) next[i] = *reinterpret_cast<const Cols<V>*>(st + (size_t)n * P);
      }
#pragma unroll
      for (int i = 0; i < FLY; ++i) {
        const int n = n0 + i * RW;
        if (n < N) {
          const float d = GATED ? keep : as[n], k = ks[n], q = qs[n];
#pragma unroll
          for (int c = 0; c < V; ++c) {
            s[i].v[c] = fmaf(d, s[i].v[c], k * v[c]);
            acc[c] = fmaf(q, s[i].v[c], acc[c]);
          }
          *reinterpret_cast<Cols<V>*>(st + (size_t)n * P) = s[i];
        }
      }
#pragma unroll
      for (int i = 0; i < FLY; ++i) s[i] = next[i];
    }
#pragma unroll
    for (int c = 0; c < V; ++c) part[r0 * PB + gc * V + c] = acc[c];
  }
  __syncthreads();
  float sq = 0.f;
  for (int c = threadIdx.x; c < cols; c += THREADS) {
    float o = 0.f;
    for (int r = 0; r < RW; ++r) o += part[r * PB + c];
    o *= inv;
    part[c] = o;
    sq += o * o;
  }
  sq = block_sum(sq, scratch);
  const int CS = gridDim.x;
  if (CS > 1) {
    if (threadIdx.x == 0) squares = sq;
    cluster.sync();
    sq = 0.f;
    for (int b = 0; b < CS; ++b) sq += *cluster.map_shared_rank(&squares, b);
  }
  const float rstd = rsqrtf(sq / (float)P + a.eps);
  const T* gr = reinterpret_cast<const T*>(a.g) + (size_t)seq * a.g_stride + (size_t)h * P + p0;
  T* out = reinterpret_cast<T*>(a.out) + (size_t)seq * a.out_stride + a.out_col + (size_t)h * P + p0;
  for (int c = threadIdx.x; c < cols; c += THREADS) {
    const float z = to_float<T>(gr[c]);
    const float gate = GATED ? sigmoid_f(z) : z * sigmoid_f(z);
    out[c] = from_float<T>(part[c] * rstd * a.weight[GATED ? h * P + p0 + c : p0 + c] * gate * a.out_scale);
  }
  if (GATED && blockIdx.x == 0) {  // every block of the cluster has read the old ones: they met at the barrier above
    for (int n = threadIdx.x; n < N; n += THREADS) nm[n] = as[n];
    if (threadIdx.x == 0) nm[N] = m;
  }
  if (CS > 1) cluster.sync();  // a block's shared memory stays until its last reader is done
}

template <typename T, bool GATED>
int launch_step(StepArgs a, int n_seqs, int CS, cudaStream_t stream) {
  const bool vec = a.P % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
  const int V = vec ? 4 : 1;
  a.PB = ((a.P + CS - 1) / CS + V - 1) / V * V;
  if (a.PB / V > THREADS) return -2;
  const int RW = THREADS / (a.PB / V);
  const size_t smem = ((size_t)3 * a.N + (size_t)RW * a.PB) * sizeof(float);
  if (smem > 200 * 1024 || a.H > 65535 || n_seqs > 65535) return -2;
  auto kern = vec ? memory_step_kernel<T, GATED, 4> : memory_step_kernel<T, GATED, 1>;
  if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)CS, (unsigned)a.H, (unsigned)n_seqs);
  cfg.blockDim = dim3(THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = (unsigned)CS;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  static const bool plain = getenv("KRK_NO_PDL") != nullptr;
  cfg.attrs = attr;
  cfg.numAttrs = plain ? 1 : 2;
  return (int)cudaLaunchKernelEx(&cfg, kern, a);
}

}  // namespace

// One token per sequence (row s of the inputs is sequence s). Gated (nm given): z [rows, 2H], bias [2H], cap; per channel: z
// [rows, R], w2 [H * N, R], bias [H * N], tau. CS: blocks (a cluster) per (sequence, head), 1, 2, 4 or 8.
KRK_API int krk_memory_step(void* out, int out_stride, int out_col, float out_scale, const void* q, int q_stride, const void* k,
                            int k_stride, const void* v, int v_stride, const void* g, int g_stride, float q_scale,
                            const void* z, int z_stride, const void* w2, const float* bias, float cap_or_tau, int R,
                            float* state, float* nm, const float* weight, float eps, int H, int N, int P, int n_seqs, int CS,
                            const int* seq_slot, int dtype, cudaStream_t stream) {
  if (n_seqs == 0) return 0;
  if (CS != 1 && CS != 2 && CS != 4 && CS != 8) return -2;
  StepArgs a;
  a.q = q; a.k = k; a.v = v; a.g = g; a.q_stride = q_stride; a.k_stride = k_stride; a.v_stride = v_stride; a.g_stride = g_stride;
  a.q_scale = q_scale; a.z = z; a.z_stride = z_stride; a.w2 = w2; a.bias = bias;
  a.cap_or_inv_tau = nm ? cap_or_tau : 1.0f / cap_or_tau;
  a.R = R; a.state = state; a.nm = nm; a.weight = weight; a.eps = eps; a.out = out; a.out_stride = out_stride;
  a.out_col = out_col; a.out_scale = out_scale; a.H = H; a.N = N; a.P = P; a.PB = 0; a.seq_slot = seq_slot;
  if (dtype == KRK_DTYPE_F32) return nm ? launch_step<float, true>(a, n_seqs, CS, stream) : launch_step<float, false>(a, n_seqs, CS, stream);
  return nm ? launch_step<bf16, true>(a, n_seqs, CS, stream) : launch_step<bf16, false>(a, n_seqs, CS, stream);
}
