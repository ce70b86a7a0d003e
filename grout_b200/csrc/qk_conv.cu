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
// first rows look back to.  A step's rows are cut into runs of QC_RUN (never fewer than taps - 1)
// rows that start at each sequence's first; only a sequence's first run looks back behind the
// step, so the thread that owns a channel there reads the kept values and then replaces them.
// Sequence s's runs are given the blocks cu_q[s] / RUN + s up to those of s + 1, which are never
// fewer than it needs and are found by bisection: the host need not know how rows divide into
// sequences.
#include "common.cuh"

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
#define QC_TAPS 4           // taps whose inputs a thread keeps in registers; with more it reads them again

__device__ __forceinline__ float qc_sum(const QkConvArgs& a, size_t at) {
  float v = 0.f;
  for (int k0 = 0; k0 < a.n_parts; k0 += 4) {      // four partial sums requested at a time, added in order
    float p[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int k = k0 + u < a.n_parts ? k0 + u : a.n_parts - 1;
      p[u] = a.proj[(size_t)k * a.part_stride + at];
    }
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (k0 + u < a.n_parts) v += p[u];
  }
  return v;
}

template <typename T, int TAPS>      // TAPS 0: any number of them
__global__ void __launch_bounds__(32 * QC_WARPS) qk_conv_kernel(const QkConvArgs a) {
  extern __shared__ float qc_sm[];   // the run's sines and cosines [run, rot_dim / 2] each
  pdl_launch_dependents_if_small();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int R = a.run, taps = TAPS > 0 ? TAPS : a.taps;
  int seq, run;
  if (a.one_row) {
    seq = blockIdx.x, run = 0;
  } else {                           // the last sequence whose first block is not behind this one
    int lo = 0, hi = a.n_seqs - 1;
    const int b = blockIdx.x;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (a.cu_q[mid] / R + mid <= b) lo = mid; else hi = mid - 1;
    }
    seq = lo, run = b - (a.cu_q[lo] / R + lo);
  }
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
  pdl_wait();
  const int D = a.D, Ds = a.Ds, nqk = a.nq + a.nkv;
  const int Cc = nqk * D;                                // channels with a bias, a convolution, a kept tail
  const size_t width = (size_t)Cc + (a.v_from_k ? 0 : (size_t)a.nkv * a.Dv);
  const int n_heads = nqk + (a.v_from_k ? 0 : a.nkv);
  const int* table = slot >= 0 ? a.block_table + (size_t)slot * a.max_pages : nullptr;
  float* tail = slot >= 0 && a.tail ? a.tail + (size_t)slot * a.tail_stride : nullptr;

  // u of channel c at row rr of the sequence's rows (negative: behind the step)
  auto input = [&](int rr, int c, float b) -> float {
    if (rr >= 0) return qc_sum(a, (size_t)(row0 + rr) * width + c) + b;
    return tail && rr + taps - 1 >= 0 ? tail[(size_t)(taps - 1 + rr) * Cc + c] : 0.f;
  };
  for (int head = blockIdx.y * QC_WARPS + warp; head < n_heads; head += gridDim.y * QC_WARPS) {
    if (head >= nqk) {                                   // a value head of its own: stored as it is
      const int g = head - nqk;
      for (int i = 0; i < n && table; ++i) {
        const int pos = a.token_pos[row0 + r0 + i];
        T* dst = (T*)a.v_pages + paged_row(table, pos, g, a.nkv, a.page, Ds);
        for (int d = lane; d < Ds; d += 32)
          dst[d] = from_f32<T>(d < a.Dv ? qc_sum(a, (size_t)(row0 + r0 + i) * width + Cc + (size_t)g * a.Dv + d) : 0.f);
      }
      continue;
    }
    // an item is a rotated pair, or an element (and its neighbour) that passes unturned
    const int pairs = half + (D - 2 * half + 1) / 2;
    for (int it = lane; it < pairs; it += 32) {
      int e0, e1;
      const bool turned = it < half;
      if (turned) {
        e0 = a.interleaved ? 2 * it : it, e1 = a.interleaved ? 2 * it + 1 : it + half;
      } else {
        e0 = 2 * half + 2 * (it - half), e1 = e0 + 1;
      }
      const bool two = e1 < D;
      const int c0 = head * D + e0, c1 = head * D + (two ? e1 : e0);
      const float b0 = a.bias ? a.bias[c0] : 0.f, b1 = a.bias ? a.bias[c1] : 0.f;
      constexpr int W = TAPS > 0 ? TAPS : 1;
      float w0[W], w1[W], x0[W], x1[W];      // x[j]: the input j rows back
#pragma unroll
      for (int j = 0; j < W; ++j) {
        w0[j] = w1[j] = 1.f, x0[j] = x1[j] = 0.f;
        if (TAPS > 0) {
          if (a.conv_w) {
            w0[j] = a.conv_w[(size_t)c0 * taps + taps - 1 - j];
            w1[j] = a.conv_w[(size_t)c1 * taps + taps - 1 - j];
          }
          if (j > 0) x0[j - 1] = input(r0 - j, c0, b0), x1[j - 1] = input(r0 - j, c1, b1);
        }
      }
#pragma unroll 2
      for (int i = 0; i < n; ++i) {
        float y0, y1;
        if (TAPS > 0) {
#pragma unroll
          for (int j = W - 1; j > 0; --j) x0[j] = x0[j - 1], x1[j] = x1[j - 1];
          x0[0] = input(r0 + i, c0, b0), x1[0] = input(r0 + i, c1, b1);
          y0 = w0[0] * x0[0], y1 = w1[0] * x1[0];
#pragma unroll
          for (int j = 1; j < W; ++j) y0 = fmaf(w0[j], x0[j], y0), y1 = fmaf(w1[j], x1[j], y1);
        } else {
          y0 = 0.f, y1 = 0.f;
          for (int j = 0; j < taps; ++j) {
            y0 = fmaf(a.conv_w[(size_t)c0 * taps + taps - 1 - j], input(r0 + i - j, c0, b0), y0);
            y1 = fmaf(a.conv_w[(size_t)c1 * taps + taps - 1 - j], input(r0 + i - j, c1, b1), y1);
          }
        }
        const float v0 = y0, v1 = y1;
        if (turned) {
          const float s = sn[i * half + it], c = cs[i * half + it];
          y0 = v0 * c - v1 * s;
          y1 = v1 * c + v0 * s;
        }
        if (head < a.nq) {
          T* dst = (T*)a.q_out + ((size_t)(row0 + r0 + i) * a.nq + head) * Ds;
          dst[e0] = from_f32<T>(y0);
          if (two) dst[e1] = from_f32<T>(y1);
        } else if (table) {
          const size_t at = paged_row(table, a.token_pos[row0 + r0 + i], head - a.nq, a.nkv, a.page, Ds);
          T* dst = (T*)a.k_pages + at;
          dst[e0] = from_f32<T>(y0);
          if (two) dst[e1] = from_f32<T>(y1);
          if (a.v_from_k) {
            T* dv = (T*)a.v_pages + at;
            dv[e0] = from_f32<T>(v0);
            if (two) dv[e1] = from_f32<T>(v1);
          }
        }
      }
      if (tail && run == 0) {        // entry s: the input at n_seq - (taps - 1) + s; an entry that moves down
                                     // is read before it is overwritten
        for (int s = 0; s < taps - 1; ++s) {
          const int rr = n_seq - (taps - 1) + s;
          const float t0 = input(rr, c0, b0), t1 = input(rr, c1, b1);
          tail[(size_t)s * Cc + c0] = t0;
          if (two) tail[(size_t)s * Cc + c1] = t1;
        }
      }
    }
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

template <typename T, int TAPS>
static int launch_taps(const QkConvArgs& a, cudaStream_t s) {
  const int blocks = a.one_row ? a.n_seqs : a.T / a.run + a.n_seqs;
  const int n_heads = a.nq + a.nkv * (a.v_from_k ? 1 : 2);
  int y = (n_heads + QC_WARPS - 1) / QC_WARPS;           // few runs: a warp per head; many: fewer warps, whose
  while (y > 1 && (long long)blocks * y > 148 * 16) y = (y + 1) / 2;   // sines serve several heads
  const size_t smem = a.inv_freq ? (size_t)a.run * a.rot_dim * sizeof(float) : 0;
  if (smem > 48 * 1024) return GB_ERR_UNSUPPORTED;
  return gb_launch(qk_conv_kernel<T, TAPS>, dim3(blocks, y), dim3(32 * QC_WARPS), smem, s, a);
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
  a.run = a.taps - 1 > QC_RUN ? a.taps - 1 : QC_RUN;
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
