// Dynamic tanh, a norm without statistics, with the residual sum in front of it:
//
//   v = res_in[s, :] + delta[s, :]           (or n_parts 32-bit partial sums of it, in order)
//   res_out[r, :] = v                        (32-bit residual stream, optional)
//   y[r, :] = tanh(alpha * v) * w + b        (alpha one number; w, b vectors; all 32-bit)
//
// s = rows[r] when a row list is given (the gather before the last norm), else r.  Every
// element stands for itself: there is nothing to sum over a row, so a row is cut into as
// many blocks as keep the GPU busy and no block waits for another.  A thread takes four
// neighbouring elements of a row, or of four rows (one element where the width or an address
// does not allow that); the order in which partial sums are added depends on nothing but
// their number.
#include "common.cuh"

struct DytArgs {
  const float* res_in;
  const void* delta;        // [rows_total, N] in the activation type, or null
  const float* parts;       // instead of delta: n_parts partial sums, part_stride floats apart
  int n_parts;
  long long part_stride;
  const int* rows;          // row list or null
  const float* alpha;       // [1]
  const float* w;           // [N]
  const float* b;           // [N]
  float* res_out;
  void* y;
  int n_rows, N;
};

template <typename T> __device__ __forceinline__ void load4(const T* p, float (&v)[4]);
template <> __device__ __forceinline__ void load4<float>(const float* p, float (&v)[4]) {
  const float4 x = *reinterpret_cast<const float4*>(p);
  v[0] = x.x; v[1] = x.y; v[2] = x.z; v[3] = x.w;
}
template <> __device__ __forceinline__ void load4<bf16>(const bf16* p, float (&v)[4]) {
  const uint2 x = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&x.x);
  const __nv_bfloat162 b = *reinterpret_cast<const __nv_bfloat162*>(&x.y);
  v[0] = __low2float(a); v[1] = __high2float(a); v[2] = __low2float(b); v[3] = __high2float(b);
}
template <typename T> __device__ __forceinline__ void store4(T* p, const float (&v)[4]);
template <> __device__ __forceinline__ void store4<float>(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <> __device__ __forceinline__ void store4<bf16>(bf16* p, const float (&v)[4]) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
  uint2 x;
  x.x = *reinterpret_cast<uint32_t*>(&a);
  x.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = x;
}

#define DYT_THREADS 128

// ROWS rows a thread, one after the other in memory, with PU partial sums of each requested at
// once: a step of many rows keeps more loads under way per thread (one row a thread left the
// kernel waiting for memory in waves), a step of few spreads its rows over the blocks.
template <typename T, int ROWS, int PU>
__global__ void __launch_bounds__(DYT_THREADS) add_dyt_vec_kernel(const DytArgs a) {
  pdl_launch_dependents_if_small();
  const int N = a.N, i = (blockIdx.y * DYT_THREADS + threadIdx.x) * 4, r0 = blockIdx.x * ROWS;
  float wv[4], bv[4], alpha = 0.f;
  if (i < N) {                    // no kernel's output: before the wait
    alpha = *a.alpha;
    load4<float>(a.w + i, wv);
    load4<float>(a.b + i, bv);
  }
  pdl_wait();
  if (i < N) {
    float v[ROWS][4], d[ROWS][4];
    size_t at[ROWS];
#pragma unroll
    for (int k = 0; k < ROWS; ++k) {
      const int r = min(r0 + k, a.n_rows - 1);
      at[k] = (a.rows ? (size_t)a.rows[r] : (size_t)r) * N + i;
#pragma unroll
      for (int e = 0; e < 4; ++e) v[k][e] = d[k][e] = 0.f;
      if (a.res_in) load4<float>(a.res_in + at[k], v[k]);
      if (a.delta) load4<T>((const T*)a.delta + at[k], d[k]);
    }
    for (int k0 = 0; k0 < a.n_parts; k0 += PU) {   // PU of them requested at once, added in order
      float pk[PU][ROWS][4];
#pragma unroll
      for (int u = 0; u < PU; ++u)
        if (k0 + u < a.n_parts) {
#pragma unroll
          for (int k = 0; k < ROWS; ++k) load4<float>(a.parts + (size_t)(k0 + u) * a.part_stride + at[k], pk[u][k]);
        }
#pragma unroll
      for (int u = 0; u < PU; ++u)
        if (k0 + u < a.n_parts) {
#pragma unroll
          for (int k = 0; k < ROWS; ++k)
#pragma unroll
            for (int e = 0; e < 4; ++e) d[k][e] += pk[u][k][e];
        }
    }
#pragma unroll
    for (int k = 0; k < ROWS; ++k) {
      if (r0 + k >= a.n_rows) break;
      float o[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        v[k][e] += d[k][e];
        o[e] = tanhf(alpha * v[k][e]) * wv[e] + bv[e];
      }
      const size_t to = (size_t)(r0 + k) * N + i;
      if (a.res_out) store4<float>(a.res_out + to, v[k]);
      store4<T>((T*)a.y + to, o);
    }
  }
  pdl_launch_dependents_if_large();
}

template <typename T>
__global__ void __launch_bounds__(DYT_THREADS) add_dyt_kernel(const DytArgs a) {
  pdl_launch_dependents_if_small();
  pdl_wait();
  const int N = a.N, i = blockIdx.y * DYT_THREADS + threadIdx.x, r = blockIdx.x;
  if (i < N) {
    const size_t s = a.rows ? (size_t)a.rows[r] : (size_t)r;
    float d = a.delta ? to_f32<T>(((const T*)a.delta)[s * N + i]) : 0.f;
    for (int k = 0; k < a.n_parts; ++k) d += a.parts[(size_t)k * a.part_stride + s * N + i];
    const float v = (a.res_in ? a.res_in[s * N + i] : 0.f) + d;
    if (a.res_out) a.res_out[(size_t)r * N + i] = v;
    ((T*)a.y)[(size_t)r * N + i] = from_f32<T>(tanhf(*a.alpha * v) * a.w[i] + a.b[i]);
  }
  pdl_launch_dependents_if_large();
}

template <typename T>
static int launch(const DytArgs& a, cudaStream_t s) {
  if (a.n_rows < 0 || a.N <= 0 || (!a.res_in && !a.delta && !a.parts)) return GB_ERR_BAD_ARG;
  if ((a.parts != nullptr) != (a.n_parts > 0) || a.n_parts < 0 || (a.parts && a.delta)) return GB_ERR_BAD_ARG;
  if (!a.alpha || !a.w || !a.b || !a.y) return GB_ERR_BAD_ARG;
  // in place is allowed only without a row list (every element then belongs to one thread)
  if (a.rows && a.res_out && a.res_out == a.res_in) return GB_ERR_BAD_ARG;
  if (a.n_rows == 0) return 0;
  const uintptr_t all = (uintptr_t)a.res_in | (uintptr_t)a.delta | (uintptr_t)a.parts | (uintptr_t)a.w |
                        (uintptr_t)a.b | (uintptr_t)a.res_out | (uintptr_t)a.y | (uintptr_t)(a.part_stride * 4);
  const bool vec = a.N % 4 == 0 && (all & 15) == 0;
  const int per = vec ? 4 * DYT_THREADS : DYT_THREADS;
  const long long gy = ((long long)a.N + per - 1) / per;
  if (gy > 65535) return GB_ERR_UNSUPPORTED;
  if (vec && a.n_rows >= 512)
    return gb_launch(add_dyt_vec_kernel<T, 4, 3>, dim3((a.n_rows + 3) / 4, (unsigned)gy), dim3(DYT_THREADS), 0, s, a);
  const dim3 grid(a.n_rows, (unsigned)gy);
  return vec ? gb_launch(add_dyt_vec_kernel<T, 1, 8>, grid, dim3(DYT_THREADS), 0, s, a)
             : gb_launch(add_dyt_kernel<T>, grid, dim3(DYT_THREADS), 0, s, a);
}

GB_EXPORT int gb_add_dyt_f32(const DytArgs* a, cudaStream_t s) { return launch<float>(*a, s); }
GB_EXPORT int gb_add_dyt_bf16(const DytArgs* a, cudaStream_t s) { return launch<bf16>(*a, s); }
