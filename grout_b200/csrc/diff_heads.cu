// The difference of two attention maps, per head (differential attention):
//
//   o = x[t, 2h, :Dv] - lambda * x[t, 2h + 1, :Dv]
//   out[t, h * Dv + d] = o[d] / sqrt(mean(o^2) + eps) * mult
//
// x [T, 2 heads, Ds] holds the two maps' outputs of every head side by side (what lies
// beyond Dv is dropped).  The difference, the mean and the scaling are 32-bit.  A head is
// LPH lanes of a warp, eight neighbouring elements a lane and pass; the order of a head's
// sum depends on Dv alone.  Sizes or addresses that are no multiple of eight elements take
// a warp a head, element by element.
#include "common.cuh"

struct DiffHeadsArgs {
  const void* x;     // [n_rows, 2 heads, Ds]
  void* out;         // [n_rows, heads * Dv]
  int n_rows, heads, Ds, Dv;
  float lambda, eps, mult;
};

template <typename T> __device__ __forceinline__ void load8(const T* p, float (&v)[8]);
template <> __device__ __forceinline__ void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <> __device__ __forceinline__ void load8<bf16>(const bf16* p, float (&v)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {raw.x, raw.y, raw.z, raw.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(&w[i]);
    v[2 * i] = __low2float(x), v[2 * i + 1] = __high2float(x);
  }
}
__device__ __forceinline__ void store8(float* p, const float (&v)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
__device__ __forceinline__ void store8(bf16* p, const float (&v)[8]) {
  uint32_t w[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const __nv_bfloat162 x = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    w[i] = *reinterpret_cast<const uint32_t*>(&x);
  }
  *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]);
}

#define DH_THREADS 128

// PIECES: eight-element pieces a lane holds
template <typename T, int LPH, int PIECES>
__global__ void __launch_bounds__(DH_THREADS) diff_heads_vec_kernel(const DiffHeadsArgs a) {
  pdl_launch_dependents_if_small();
  pdl_wait();
  const int sub = threadIdx.x % LPH, Dv = a.Dv;
  const long long head = (long long)blockIdx.x * (DH_THREADS / LPH) + threadIdx.x / LPH;   // row * heads + h
  const bool live = head < (long long)a.n_rows * a.heads;
  const T* x = (const T*)a.x + (live ? head : 0) * 2 * a.Ds;
  float o[PIECES][8], ss = 0.f;
#pragma unroll
  for (int p = 0; p < PIECES; ++p) {
    const int d = (sub + p * LPH) * 8;
    if (d < Dv) {
      float u[8], v[8];
      load8<T>(x + d, u);
      load8<T>(x + a.Ds + d, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        o[p][e] = u[e] - a.lambda * v[e];
        ss = fmaf(o[p][e], o[p][e], ss);
      }
    }
  }
#pragma unroll
  for (int s = LPH >> 1; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  const float f = a.mult / sqrtf(ss / (float)Dv + a.eps);
  if (live) {
    T* out = (T*)a.out + head * Dv;
#pragma unroll
    for (int p = 0; p < PIECES; ++p) {
      const int d = (sub + p * LPH) * 8;
      if (d < Dv) {
#pragma unroll
        for (int e = 0; e < 8; ++e) o[p][e] *= f;
        store8(out + d, o[p]);
      }
    }
  }
  pdl_launch_dependents_if_large();
}

template <typename T>
__global__ void __launch_bounds__(DH_THREADS) diff_heads_kernel(const DiffHeadsArgs a) {
  pdl_launch_dependents_if_small();
  pdl_wait();
  const int lane = threadIdx.x & 31, Dv = a.Dv;
  const long long head = (long long)blockIdx.x * (DH_THREADS / 32) + (threadIdx.x >> 5);
  if (head >= (long long)a.n_rows * a.heads) return;
  const T* x = (const T*)a.x + head * 2 * a.Ds;
  float ss = 0.f;
  for (int d = lane; d < Dv; d += 32) {
    const float o = to_f32<T>(x[d]) - a.lambda * to_f32<T>(x[a.Ds + d]);
    ss = fmaf(o, o, ss);
  }
  const float f = a.mult / sqrtf(warp_sum(ss) / (float)Dv + a.eps);
  T* out = (T*)a.out + head * Dv;
  for (int d = lane; d < Dv; d += 32)
    out[d] = from_f32<T>((to_f32<T>(x[d]) - a.lambda * to_f32<T>(x[a.Ds + d])) * f);
}

template <typename T, int LPH, int PIECES>
static int launch_vec(const DiffHeadsArgs& a, cudaStream_t s) {
  const long long heads = (long long)a.n_rows * a.heads, per = DH_THREADS / LPH;
  return gb_launch(diff_heads_vec_kernel<T, LPH, PIECES>, dim3((unsigned)((heads + per - 1) / per)),
                   dim3(DH_THREADS), 0, s, a);
}

template <typename T>
static int launch(const DiffHeadsArgs& a, cudaStream_t s) {
  if (!a.x || !a.out || a.n_rows < 0 || a.heads <= 0 || a.Dv <= 0 || a.Ds < a.Dv) return GB_ERR_BAD_ARG;
  if (a.n_rows == 0) return 0;
  if ((long long)a.n_rows * a.heads > 0x7fffffffLL) return GB_ERR_UNSUPPORTED;
  if (a.Dv % 8 == 0 && a.Ds % 8 == 0 && ((((uintptr_t)a.x) | ((uintptr_t)a.out)) & 15) == 0) {
    if (a.Dv <= 32) return launch_vec<T, 4, 1>(a, s);
    if (a.Dv <= 64) return launch_vec<T, 8, 1>(a, s);
    if (a.Dv <= 128) return launch_vec<T, 16, 1>(a, s);
    if (a.Dv <= 256) return launch_vec<T, 32, 1>(a, s);
    if (a.Dv <= 512) return launch_vec<T, 32, 2>(a, s);
  }
  const long long heads = (long long)a.n_rows * a.heads, per = DH_THREADS / 32;
  return gb_launch(diff_heads_kernel<T>, dim3((unsigned)((heads + per - 1) / per)), dim3(DH_THREADS), 0, s, a);
}

GB_EXPORT int gb_diff_heads_f32(const DiffHeadsArgs* a, cudaStream_t s) { return launch<float>(*a, s); }
GB_EXPORT int gb_diff_heads_bf16(const DiffHeadsArgs* a, cudaStream_t s) { return launch<bf16>(*a, s); }
