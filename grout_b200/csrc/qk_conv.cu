// Preparation of queries and keys behind a short causal convolution: per channel of the
// projection's q and k columns
//
//   u_t = sum_p proj_p[t] (partial sums in order) + bias;   c_t = sum_j w[taps - 1 - j] u_{t - j}
//
// with zeros in front of the sequence's start (not the bias), then the rotation of the first
// rot_dim elements of every head (half-split pairs, or neighbours with `interleaved`); q goes
// to q_out, k and v into the paged cache at the token's position.  A value is its key as it
// leaves the convolution, before the rotation (v_from_k), or a column of the projection that
// passes as it is.  All arithmetic is 32-bit; one rounding at the store.  Bias, convolution
// and rotation may each be absent.
//
// The last taps - 1 values u of every sequence are kept (32-bit, `tail`): what a later step's
// first rows look back to.  A block takes a run of rows (run_of_block), a warp of it a head.
#include "short_conv.cuh"

struct QkConvArgs {
  const float* proj;        // [n_parts][T, (nq + nkv) D (+ nkv Dv)] 32-bit sums
  int n_parts;
  long long part_stride;
  const float* bias;        // [(nq + nkv) D] or null
  const float* conv_w;      // [(nq + nkv) D, taps] (the last column is the current token's), or null: taps = 1
  const float* inv_freq;    // [rot_dim / 2] or null
  const int* cu_q;          // [n_seqs + 1]
  const int* token_pos;     // [T]
  const int* slots;         // [n_seqs], < 0 for padding
  const int* block_table;   // [slots, max_pages]
  float* tail;              // [slots, tail_stride]: [taps - 1, (nq + nkv) D]; null when taps = 1
  long long tail_stride;
  void* q_out;              // [T, nq, Ds]
  void* k_pages;            // [n_pages, nkv, page, Ds]
  void* v_pages;
  int T, n_seqs, nq, nkv, D, Dv, Ds, taps, rot_dim, interleaved, v_from_k, max_pages, page;
  float rot_scale;
  int run;                  // rows of a run
  int one_row;              // every sequence brings one row (a decode step): block i is sequence i
};

#define QC_RUN 8
#define QC_WARPS 8
#define QC_AHEAD 4          // rows requested at a time
#define QC_TAPS 4           // taps whose inputs a thread keeps in registers; with more it reads them again

// V neighbouring values of the projection from `at` on, the partial sums added in order.
template <int V>
__device__ __forceinline__ void qc_sum(const QkConvArgs& a, size_t at, float (&v)[V]) {
  auto load = [&](const float* p, float (&o)[V]) {
    if constexpr (V == 2) {
      const float2 x = *reinterpret_cast<const float2*>(p);
      o[0] = x.x, o[1] = x.y;
    } else {
      o[0] = p[0];
    }
  };
  load(a.proj + at, v);
  for (int k0 = 1; k0 < a.n_parts; k0 += 4) {      // four partial sums requested at a time
    float p[4][V];
#pragma unroll
    for (int u = 0; u < 4; ++u)
      load(a.proj + (size_t)(k0 + u < a.n_parts ? k0 + u : a.n_parts - 1) * a.part_stride + at, p[u]);
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (k0 + u < a.n_parts) {
#pragma unroll
        for (int e = 0; e < V; ++e) v[e] += p[u][e];
      }
  }
}

template <typename T, int V>
__device__ __forceinline__ void qc_store(T* p, const float (&v)[V]) {
  if constexpr (V == 2 && sizeof(T) == 2) *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[1]);
  else if constexpr (V == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
  else p[0] = from_f32<T>(v[0]);
}

// TAPS 0: any number of them.  V: neighbouring pairs (or pieces of what is not turned) a lane takes together
template <typename T, int TAPS, int V>
__global__ void __launch_bounds__(32 * QC_WARPS) qk_conv_kernel(const QkConvArgs a) {
  extern __shared__ float qc_sm[];   // the run's sines and cosines [run, rot_dim / 2] each
  pdl_launch_dependents_if_small();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int R = a.run, taps = TAPS > 0 ? TAPS : a.taps;
  int seq, run;
  run_of_block(a.cu_q, a.n_seqs, R, a.one_row, blockIdx.x, seq, run);
  const int row0 = a.cu_q[seq], n_seq = a.cu_q[seq + 1] - row0;
  const int r0 = run * R, n = min(R, n_seq - r0);        // the run: rows r0 .. r0 + n of the sequence
  if (n <= 0) return;
  const int slot = a.slots[seq];
  const int half = a.inv_freq ? a.rot_dim / 2 : 0;
  float* sn = qc_sm;
  float* cs = qc_sm + (size_t)R * half;
  for (int i = threadIdx.x; i < n * half; i += blockDim.x) {
    float s, c;
    sincosf((float)a.token_pos[row0 + r0 + i / half] * a.inv_freq[i % half], &s, &c);
    sn[i] = s * a.rot_scale, cs[i] = c * a.rot_scale;
  }
  __syncthreads();
  const int D = a.D, Ds = a.Ds, nqk = a.nq + a.nkv;
  const int Cc = nqk * D;                                // channels with a bias, a convolution, a kept tail
  const size_t width = (size_t)Cc + (a.v_from_k ? 0 : (size_t)a.nkv * a.Dv);
  const int n_heads = nqk + (a.v_from_k ? 0 : a.nkv);
  const int* table = slot >= 0 ? a.block_table + (size_t)slot * a.max_pages : nullptr;
  float* tail = slot >= 0 && a.tail ? a.tail + (size_t)slot * a.tail_stride : nullptr;

  // u of channels c .. at row rr of the sequence's rows (negative: behind the step)
  auto input = [&](int rr, int c, const float (&b)[V], float (&u)[V]) {
    if (rr >= 0) {
      qc_sum<V>(a, (size_t)(row0 + rr) * width + c, u);
#pragma unroll
      for (int e = 0; e < V; ++e) u[e] += b[e];
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) u[e] = tail && rr + taps - 1 >= 0 ? tail[(size_t)(taps - 1 + rr) * Cc + c + e] : 0.f;
    }
  };
  for (int head = blockIdx.y * QC_WARPS + warp; head < n_heads; head += gridDim.y * QC_WARPS) {
    // (a warp waits for the product where it first reads it: what is no kernel's output, the weights,
    // is fetched before; further waits return at once)
    if (head >= nqk) {                                   // a value head of its own: stored as it is
      const int g = head - nqk;
      pdl_wait();
      for (int i = 0; i < n && table; ++i) {
        const int pos = a.token_pos[row0 + r0 + i];
        T* dst = (T*)a.v_pages + paged_row(table, pos, g, a.nkv, a.page, Ds);
        for (int d = lane; d < Ds; d += 32) {
          float v[1] = {0.f};
          if (d < a.Dv) qc_sum<1>(a, (size_t)(row0 + r0 + i) * width + Cc + (size_t)g * a.Dv + d, v);
          dst[d] = from_f32<T>(v[0]);
        }
      }
      continue;
    }
    // an item is V rotated pairs, or as many pairs of elements that pass unturned
    const int turned_items = half / V;
    const int items = turned_items + (D - 2 * half + 2 * V - 1) / (2 * V);
    for (int it = lane; it < items; it += 32) {
      int e0, e1;
      const bool turned = it < turned_items;
      if (turned) {
        e0 = a.interleaved ? 2 * it : it * V, e1 = a.interleaved ? 2 * it + 1 : it * V + half;
      } else {
        e0 = 2 * half + 2 * V * (it - turned_items), e1 = e0 + V;
      }
      const bool two = e1 < D;
      const int ch[2] = {head * D + e0, head * D + (two ? e1 : e0)};
      constexpr int W = TAPS > 0 ? TAPS : 1;
      float b[2][V], w[W][2][V], x[W][2][V];      // x[j]: the input j rows back
#pragma unroll
      for (int s = 0; s < 2; ++s)
#pragma unroll
        for (int e = 0; e < V; ++e) b[s][e] = a.bias ? a.bias[ch[s] + e] : 0.f;
#pragma unroll
      for (int j = 0; j < W; ++j)
#pragma unroll
        for (int s = 0; s < 2; ++s) {
#pragma unroll
          for (int e = 0; e < V; ++e)
            w[j][s][e] = TAPS > 0 && a.conv_w ? a.conv_w[(size_t)(ch[s] + e) * taps + taps - 1 - j] : 1.f;
        }
      pdl_wait();
      if (TAPS > 0) {
#pragma unroll
        for (int j = 1; j < W; ++j)
#pragma unroll
          for (int s = 0; s < 2; ++s) input(r0 - j, ch[s], b[s], x[j - 1][s]);
      }
      for (int i0 = 0; i0 < n; i0 += QC_AHEAD) {   // several rows are requested before the first is worked on
       float fresh[QC_AHEAD][2][V];
       if (TAPS > 0) {
#pragma unroll
         for (int u = 0; u < QC_AHEAD; ++u)
#pragma unroll
           for (int s = 0; s < 2; ++s)
             if (u == 0 || i0 + u < n) qc_sum<V>(a, (size_t)(row0 + r0 + i0 + u) * width + ch[s], fresh[u][s]);
       }
#pragma unroll
       for (int u = 0; u < QC_AHEAD; ++u) {
        const int i = i0 + u;
        if (i >= n) break;
        float c[2][V];
        if (TAPS > 0) {
#pragma unroll
          for (int j = W - 1; j > 0; --j)
#pragma unroll
            for (int s = 0; s < 2; ++s)
#pragma unroll
              for (int e = 0; e < V; ++e) x[j][s][e] = x[j - 1][s][e];
#pragma unroll
          for (int s = 0; s < 2; ++s) {
#pragma unroll
            for (int e = 0; e < V; ++e) {
              x[0][s][e] = fresh[u][s][e] + b[s][e];
              c[s][e] = w[0][s][e] * x[0][s][e];
#pragma unroll
              for (int j = 1; j < W; ++j) c[s][e] = fmaf(w[j][s][e], x[j][s][e], c[s][e]);
            }
          }
        } else {
#pragma unroll
          for (int s = 0; s < 2; ++s)
#pragma unroll
            for (int e = 0; e < V; ++e) c[s][e] = 0.f;
          for (int j = 0; j < taps; ++j)
#pragma unroll
            for (int s = 0; s < 2; ++s) {
              input(r0 + i - j, ch[s], b[s], x[0][s]);
#pragma unroll
              for (int e = 0; e < V; ++e)
                c[s][e] = fmaf(a.conv_w[(size_t)(ch[s] + e) * taps + taps - 1 - j], x[0][s][e], c[s][e]);
            }
        }
        T* dst = nullptr;
        if (head < a.nq) {
          dst = (T*)a.q_out + ((size_t)(row0 + r0 + i) * a.nq + head) * Ds;
        } else if (table) {
          const size_t at = paged_row(table, a.token_pos[row0 + r0 + i], head - a.nq, a.nkv, a.page, Ds);
          dst = (T*)a.k_pages + at;
          if (a.v_from_k) {                      // the value: the key as it stands now
            qc_store<T, V>((T*)a.v_pages + at + e0, c[0]);
            if (two) qc_store<T, V>((T*)a.v_pages + at + e1, c[1]);
          }
        }
        if (turned) {
#pragma unroll
          for (int e = 0; e < V; ++e) {
            const int pair = a.interleaved ? it : it * V + e;
            const float sv = sn[i * half + pair], cv = cs[i * half + pair], lo = c[0][e], hi = c[1][e];
            c[0][e] = lo * cv - hi * sv;
            c[1][e] = hi * cv + lo * sv;
          }
        }
        if (dst) {
          qc_store<T, V>(dst + e0, c[0]);
          if (two) qc_store<T, V>(dst + e1, c[1]);
        }
       }
      }
      if (TAPS > 1 && tail && n == n_seq) {      // all of the sequence's rows: the last inputs are at hand
#pragma unroll
        for (int j = 0; j < W - 1; ++j)
#pragma unroll
          for (int k = 0; k < 2; ++k)
            if (k == 0 || two) {
#pragma unroll
              for (int e = 0; e < V; ++e) tail[(size_t)(taps - 2 - j) * Cc + ch[k] + e] = x[j][k][e];
            }
      } else if (tail && run == 0) { // entry s: the input at n_seq - (taps - 1) + s; an entry that moves down
                                     // is read before it is overwritten
        for (int s = 0; s < taps - 1; ++s) {
          float t[2][V];
#pragma unroll
          for (int k = 0; k < 2; ++k) input(n_seq - (taps - 1) + s, ch[k], b[k], t[k]);
#pragma unroll
          for (int k = 0; k < 2; ++k)
            if (k == 0 || two) {
#pragma unroll
              for (int e = 0; e < V; ++e) tail[(size_t)s * Cc + ch[k] + e] = t[k][e];
            }
        }
      }
    }
    pdl_wait();
    for (int i = 0; i < n && Ds > D; ++i) {              // a narrower head is filled up with zeros
      T* dst = nullptr;
      T* dst2 = nullptr;
      if (head < a.nq) {
        dst = (T*)a.q_out + ((size_t)(row0 + r0 + i) * a.nq + head) * Ds;
      } else if (table) {
        const size_t at = paged_row(table, a.token_pos[row0 + r0 + i], head - a.nq, a.nkv, a.page, Ds);
        dst = (T*)a.k_pages + at;
        if (a.v_from_k) dst2 = (T*)a.v_pages + at;
      }
      for (int d = D + lane; d < Ds; d += 32) {
        if (dst) dst[d] = from_f32<T>(0.f);
        if (dst2) dst2[d] = from_f32<T>(0.f);
      }
    }
  }
  pdl_launch_dependents_if_large();
}

template <typename T, int TAPS, int V>
static int launch_items(const QkConvArgs& a, cudaStream_t s) {
  const int blocks = a.one_row ? a.n_seqs : a.T / a.run + a.n_seqs;
  const int n_heads = a.nq + a.nkv * (a.v_from_k ? 1 : 2);
  int y = (n_heads + QC_WARPS - 1) / QC_WARPS;           // few runs: a warp per head; many: fewer warps, whose
  while (y > 1 && (long long)blocks * y > 148 * 16) y = (y + 1) / 2;   // sines serve several heads
  const size_t smem = a.inv_freq ? (size_t)a.run * a.rot_dim * sizeof(float) : 0;
  if (smem > 48 * 1024) return GB_ERR_UNSUPPORTED;
  return gb_launch(qk_conv_kernel<T, TAPS, V>, dim3(blocks, y), dim3(32 * QC_WARPS), smem, s, a);
}

template <typename T, int TAPS>
static int launch_taps(const QkConvArgs& a, cudaStream_t s) {
  // two pairs together where every piece of two lies on its boundary
  const long long width = (long long)(a.nq + a.nkv) * a.D + (a.v_from_k ? 0 : (long long)a.nkv * a.Dv);
  const bool even = !a.interleaved && a.rot_dim % 4 == 0 && (a.D - a.rot_dim) % 4 == 0 && a.Ds % 2 == 0 && width % 2 == 0 &&
                    a.part_stride % 2 == 0 &&
                    (((uintptr_t)a.proj | (uintptr_t)a.q_out | (uintptr_t)a.k_pages | (uintptr_t)a.v_pages) & 7) == 0;
  return even ? launch_items<T, TAPS, 2>(a, s) : launch_items<T, TAPS, 1>(a, s);
}

template <typename T>
static int launch(const QkConvArgs& in, cudaStream_t s) {
  QkConvArgs a = in;
  if (a.T < 0 || a.n_seqs <= 0 || a.nq <= 0 || a.nkv <= 0 || a.D <= 0 || a.Dv <= 0 || a.Ds < a.D || a.Ds < a.Dv ||
      a.taps < 1 || a.n_parts < 1 || a.page <= 0 || a.max_pages <= 0 || a.rot_dim < 0 || a.rot_dim % 2 || a.rot_dim > a.D)
    return GB_ERR_BAD_ARG;
  if (!a.proj || !a.cu_q || !a.token_pos || !a.slots || !a.block_table || !a.q_out || !a.k_pages || !a.v_pages)
    return GB_ERR_BAD_ARG;
  if ((a.taps > 1 && (!a.tail || !a.conv_w)) || (a.v_from_k && a.Dv != a.D) || (a.rot_dim && !a.inv_freq))
    return GB_ERR_BAD_ARG;
  if (a.T == 0) return 0;
  if (!a.rot_dim) a.inv_freq = nullptr;
  a.run = a.T >= 1024 ? 2 * QC_RUN : QC_RUN;             // (long runs read fewer rows twice)
  if (a.taps - 1 > a.run) a.run = a.taps - 1;
  switch (a.taps) {
    case 1: return launch_taps<T, 1>(a, s);
    case 2: return launch_taps<T, 2>(a, s);
    case 3: return launch_taps<T, 3>(a, s);
    case QC_TAPS: return launch_taps<T, QC_TAPS>(a, s);
    default: return launch_taps<T, 0>(a, s);
  }
}

GB_EXPORT int gb_qk_conv_f32(const QkConvArgs* a, cudaStream_t s) { return launch<float>(*a, s); }
GB_EXPORT int gb_qk_conv_bf16(const QkConvArgs* a, cudaStream_t s) { return launch<bf16>(*a, s); }
