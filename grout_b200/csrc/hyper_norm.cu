// The boundary between two sublayers of a model with several residual streams
// ("hyper-connections"), one kernel:
//
//   X'_t = sum_s mix[s, t] X_s + out[t] * d          the sublayer's result d goes back into all streams
//   u    = sum_t read[t] X'_t                        what the next sublayer looks at
//   y    = u / sqrt(mean(u^2) + eps) * w             (without w: u itself, rounded)
//
// d comes in the activation type or as a stack of 32-bit partial sums (added in order); without
// `mix` there is nothing to put back (the model's first sublayer) and the streams stay as they
// are; without `read` u is the streams' plain sum (the model's last norm).  The streams are
// [S, T, N] in 32-bit; a stream stride of zero says that all of them are still equal (the
// embedding).  New streams are stored, in place if need be, unless a row list picks rows (the
// gather for the head).  All sums are 32-bit, and a row's result depends on that row alone.
//
// One block per row, u staying in shared memory between the two passes; or, for the few rows of a
// decode step, a cluster of blocks per row.
#include "common.cuh"
#include <cooperative_groups.h>
#include <type_traits>
namespace cg = cooperative_groups;

struct HyperNormArgs {
  const float* res_in;      // [S, T, N], stream s at s * in_stride
  long long in_stride;      // floats between streams; 0: one [T, N] that all streams equal
  const void* delta;        // [T, N] activation type, or null
  const float* parts;       // [n_parts][T, N] 32-bit partial sums, or null
  int n_parts;
  long long part_stride;
  const float* mix;         // [S, S] indexed [from, to], or null: nothing is put back
  const float* out;         // [S], with mix
  const float* read;        // [S] or null: ones
  const int* rows;          // [n_rows] or null: all T rows in order
  const float* norm_w;      // [N] or null
  float eps;
  float* res_out;           // [S, T, N] or null
  long long out_stride;
  void* y;                  // [n_rows, N]
  int n_rows, N, S;
};

#define HN_MAX_S 16

template <int V> __device__ __forceinline__ void hn_load(const float* p, float (&o)[V]) {
  if constexpr (V == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    o[0] = v.x, o[1] = v.y, o[2] = v.z, o[3] = v.w;
  } else {
    o[0] = p[0];
  }
}
template <int V> __device__ __forceinline__ void hn_load(const bf16* p, float (&o)[V]) {
  if constexpr (V == 4) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&raw.x);
    const __nv_bfloat162 b = *reinterpret_cast<const __nv_bfloat162*>(&raw.y);
    o[0] = __low2float(a), o[1] = __high2float(a), o[2] = __low2float(b), o[3] = __high2float(b);
  } else {
    o[0] = __bfloat162float(p[0]);
  }
}
template <int V> __device__ __forceinline__ void hn_store(float* p, const float (&v)[V]) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  else p[0] = v[0];
}
template <int V> __device__ __forceinline__ void hn_store(bf16* p, const float (&v)[V]) {
  if constexpr (V == 4) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 raw;
    raw.x = *reinterpret_cast<const uint32_t*>(&a);
    raw.y = *reinterpret_cast<const uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
  } else {
    p[0] = __float2bfloat16_rn(v[0]);
  }
}

// The connection's weights, brought into shared memory before the wait for the producer (no
// kernel writes them): mix [SC, SC] | out [SC] | read [SC] with SC streams at most.
template <int SC>
__device__ __forceinline__ void hn_weights(const HyperNormArgs& a, float* w) {
  const int S = a.S;
  for (int i = threadIdx.x; i < SC * SC + 2 * SC; i += blockDim.x) {
    float v = 0.f;
    if (i < SC * SC) {
      const int from = i / SC, to = i % SC;
      if (a.mix && from < S && to < S) v = a.mix[from * S + to];
    } else if (i < SC * SC + SC) {
      if (a.mix && i - SC * SC < S) v = a.out[i - SC * SC];
    } else if (i - SC * SC - SC < S) {
      v = a.read ? a.read[i - SC * SC - SC] : 1.f;
    }
    w[i] = v;
  }
}

// u's V values at columns n .. of source row t; new streams are stored on the way.  SC: the
// number of streams (EXACT), or the most there can be.
template <typename T, int V, int SC, bool EXACT>
__device__ __forceinline__ void hn_values(const HyperNormArgs& a, const float* w, size_t t, int n, float (&u)[V]) {
  const int N = a.N, S = EXACT ? SC : a.S;
  const size_t at = t * N + n;
  float x[SC][V], d[V];
#pragma unroll
  for (int s = 0; s < SC; ++s) {
    if (s == 0 || (a.in_stride && s < S)) {
      hn_load<V>(a.res_in + (size_t)s * a.in_stride + at, x[s]);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) x[s][e] = 0.f;
    }
  }
#pragma unroll
  for (int e = 0; e < V; ++e) d[e] = 0.f;
  if (a.delta) {
    hn_load<V>((const T*)a.delta + at, d);
  } else if (a.parts) {
    constexpr int PARTS = 4;           // partial sums requested at a time, added in order
    for (int k0 = 0; k0 < a.n_parts; k0 += PARTS) {
      float pk[PARTS][V];
#pragma unroll
      for (int q = 0; q < PARTS; ++q) {
        const int k = k0 + q < a.n_parts ? k0 + q : a.n_parts - 1;
        hn_load<V>(a.parts + (size_t)k * a.part_stride + at, pk[q]);
      }
#pragma unroll
      for (int q = 0; q < PARTS; ++q)
        if (k0 + q < a.n_parts) {
#pragma unroll
          for (int e = 0; e < V; ++e) d[e] += pk[q][e];
        }
    }
  }
  if (!a.in_stride) {
#pragma unroll
    for (int s = 1; s < SC; ++s)
#pragma unroll
      for (int e = 0; e < V; ++e) x[s][e] = x[0][e];
  }
#pragma unroll
  for (int e = 0; e < V; ++e) u[e] = 0.f;
  const float* w_out = w + SC * SC;
  const float* w_read = w_out + SC;
#pragma unroll
  for (int to = 0; to < SC; ++to) {
    if (!EXACT && to >= S) break;
    float nx[V];
    if (a.mix) {
#pragma unroll
      for (int e = 0; e < V; ++e) nx[e] = w_out[to] * d[e];
#pragma unroll
      for (int s = 0; s < SC; ++s) {
        const float m = w[s * SC + to];        // (zero beyond the streams there are)
#pragma unroll
        for (int e = 0; e < V; ++e) nx[e] = fmaf(m, x[s][e], nx[e]);
      }
      if (a.res_out) hn_store<V>(a.res_out + (size_t)to * a.out_stride + at, nx);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) nx[e] = x[to][e];
    }
#pragma unroll
    for (int e = 0; e < V; ++e) u[e] = fmaf(w_read[to], nx[e], u[e]);
  }
}

template <typename T, int V, int SC, bool EXACT>
__global__ void __launch_bounds__(512) hyper_norm_kernel(const HyperNormArgs a) {
  extern __shared__ __align__(16) float hn_row[];        // [N]
  __shared__ float scratch[32];
  __shared__ float w[SC * SC + 2 * SC];
  pdl_launch_dependents_if_small();
  hn_weights<SC>(a, w);
  pdl_wait();
  __syncthreads();
  const int r = blockIdx.x, N = a.N;
  const size_t t = a.rows ? (size_t)a.rows[r] : (size_t)r;
  float ss = 0.f;
  for (int n = threadIdx.x * V; n < N; n += blockDim.x * V) {
    float u[V];
    hn_values<T, V, SC, EXACT>(a, w, t, n, u);
    hn_store<V>(hn_row + n, u);
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(u[e], u[e], ss);
  }
  pdl_launch_dependents_if_large();
  float inv = 1.f;
  if (a.norm_w) inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)N + a.eps);
  for (int n = threadIdx.x * V; n < N; n += blockDim.x * V) {   // a thread reads back what it wrote
    float u[V], nw[V], o[V];
    hn_load<V>(hn_row + n, u);
#pragma unroll
    for (int e = 0; e < V; ++e) nw[e] = 1.f;
    if (a.norm_w) hn_load<V>(a.norm_w + n, nw);
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] = a.norm_w ? u[e] * inv * nw[e] : u[e];
    hn_store<V>((T*)a.y + (size_t)r * N + n, o);
  }
}

// A handful of rows (a decode step): a cluster of HN_CLUSTER blocks shares a row, a thread keeps
// its four columns in registers, and the sums of squares meet through distributed shared memory
// (added in rank order).  The cluster barrier is the hardware's; no block spins on memory.
#define HN_CLUSTER 8
template <typename T, int SC, bool EXACT>
__global__ void hyper_norm_cluster_kernel(const HyperNormArgs a) {
  __shared__ float scratch[32];
  __shared__ float ss_all[HN_CLUSTER];
  __shared__ float w[SC * SC + 2 * SC];
  cg::cluster_group cluster = cg::this_cluster();
  const int rank = (int)cluster.block_rank();
  pdl_launch_dependents_if_small();
  const int N = a.N, cols = N / HN_CLUSTER;
  const int r = blockIdx.x / HN_CLUSTER;
  const int n = rank * cols + threadIdx.x * 4;
  const bool active = threadIdx.x * 4 < cols;
  hn_weights<SC>(a, w);
  float nw[4] = {1.f, 1.f, 1.f, 1.f};
  if (active && a.norm_w) hn_load<4>(a.norm_w + n, nw);
  pdl_wait();
  __syncthreads();
  const size_t t = a.rows ? (size_t)a.rows[r] : (size_t)r;
  float u[4] = {0.f, 0.f, 0.f, 0.f};
  float ss = 0.f;
  if (active) {
    hn_values<T, 4, SC, EXACT>(a, w, t, n, u);
#pragma unroll
    for (int e = 0; e < 4; ++e) ss = fmaf(u[e], u[e], ss);
  }
  ss = block_sum(ss, scratch);
  // every block puts its sum into every block's table (thread k writes to block k): after one
  // cluster barrier each block reads its own shared memory only
  if (threadIdx.x < HN_CLUSTER) cluster.map_shared_rank(ss_all, threadIdx.x)[rank] = ss;
  cluster.sync();
  float total = 0.f;
#pragma unroll
  for (int k = 0; k < HN_CLUSTER; ++k) total += ss_all[k];
  if (active) {
    float o[4];
    const float inv = a.norm_w ? 1.0f / sqrtf(total / (float)N + a.eps) : 1.f;
#pragma unroll
    for (int e = 0; e < 4; ++e) o[e] = a.norm_w ? u[e] * inv * nw[e] : u[e];
    hn_store<4>((T*)a.y + (size_t)r * N + n, o);
  }
}

template <typename T, int V, int SC, bool EXACT>
static int launch_rows(const HyperNormArgs& a, cudaStream_t s) {
  const size_t smem = (size_t)a.N * sizeof(float);
  if (smem > 200 * 1024) return GB_ERR_UNSUPPORTED;
  static size_t configured = 40 * 1024;     // per instantiation
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(hyper_norm_kernel<T, V, SC, EXACT>,
                                         cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  // as many threads as make the turns over a row equally full (the width alone decides)
  const int pieces = (a.N + V - 1) / V, turns = (pieces + 511) / 512;
  const int threads = ((pieces + turns - 1) / turns + 31) / 32 * 32;
  return gb_launch(hyper_norm_kernel<T, V, SC, EXACT>, dim3(a.n_rows), dim3(threads), smem, s, a);
}

template <typename T, int SC, bool EXACT>
static int launch_streams(const HyperNormArgs& a, bool wide, cudaStream_t s) {
  // The cluster kernel adds the squares in another order than the kernel of one block a row, so
  // the 32-bit path never takes it: there a token's result is the same in a step of one row and
  // in a step of thousands.
  if constexpr (!std::is_same<T, float>::value) {
    if (wide && a.n_rows <= 64 && a.N >= 512 && a.N % (4 * HN_CLUSTER) == 0 && a.N / HN_CLUSTER / 4 <= 512) {
      const int threads = ((a.N / HN_CLUSTER / 4 + 31) / 32) * 32;
      return gb_launch_cluster(hyper_norm_cluster_kernel<T, SC, EXACT>, dim3(a.n_rows * HN_CLUSTER), dim3(threads),
                               0, s, HN_CLUSTER, a);
    }
  }
  return wide ? launch_rows<T, 4, SC, EXACT>(a, s) : launch_rows<T, 1, SC, EXACT>(a, s);
}

template <typename T>
static int launch(const HyperNormArgs& a, cudaStream_t s) {
  if (a.n_rows < 0 || a.N <= 0 || a.S <= 0 || !a.res_in || !a.y) return GB_ERR_BAD_ARG;
  if (a.S > HN_MAX_S) return GB_ERR_UNSUPPORTED;
  if (a.mix && (!a.out || (!a.delta && !a.parts))) return GB_ERR_BAD_ARG;
  if (!a.mix && (a.delta || a.parts || a.res_out)) return GB_ERR_BAD_ARG;
  if (a.parts && a.n_parts <= 0) return GB_ERR_BAD_ARG;
  if (a.rows && a.res_out) return GB_ERR_BAD_ARG;
  if (a.n_rows == 0) return 0;
  // 16-byte pieces need every row of every tensor to start on a 16-byte boundary
  const uintptr_t bits = (uintptr_t)a.res_in | (uintptr_t)(a.in_stride * 4) | (uintptr_t)a.delta | (uintptr_t)a.parts |
                         (uintptr_t)(a.part_stride * 4) | (uintptr_t)a.norm_w | (uintptr_t)a.res_out |
                         (uintptr_t)(a.out_stride * 4) | (uintptr_t)a.y;
  const bool wide = (bits & 15) == 0 && a.N % 4 == 0;
  switch (a.S) {
    case 1: return launch_streams<T, 1, true>(a, wide, s);
    case 2: return launch_streams<T, 2, true>(a, wide, s);
    case 3: return launch_streams<T, 3, true>(a, wide, s);
    case 4: return launch_streams<T, 4, true>(a, wide, s);
    case 8: return launch_streams<T, 8, true>(a, wide, s);
    default: break;
  }
  if (a.S < 8) return launch_streams<T, 8, false>(a, wide, s);
  return launch_streams<T, HN_MAX_S, false>(a, wide, s);
}

GB_EXPORT int gb_hyper_norm_f32(const HyperNormArgs* a, cudaStream_t s) { return launch<float>(*a, s); }
GB_EXPORT int gb_hyper_norm_bf16(const HyperNormArgs* a, cudaStream_t s) { return launch<bf16>(*a, s); }
