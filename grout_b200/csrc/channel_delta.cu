// The delta rule with one decay per key channel (Kimi delta attention): a mixer whose memory is
// one matrix S [dk, dv] per head and sequence, updated token by token,
//
//   S <- diag(g) S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q
//
// with g in (0, 1)^dk, beta in (0, 1), k a unit vector and q a unit vector times dk^(-1/2).  q, k and
// v come out of short causal convolutions over time (one filter per channel, no bias) followed by
// silu; g = exp(-exp(A_log) softplus(z + dt_bias)) with logits z from a product of two thin
// matrices; the read-out is RMS-normalised over dv, multiplied by a weight shared by the heads
// and by the sigmoid of a gate that comes from two thin matrices, too.
//
// Everything here is 32-bit whatever the activation type: the projection and the second thin
// product arrive as 32-bit sums, and only y, the o projection's input, is rounded (and the thin
// products' inner values, where activations are 16-bit).
//
//   prepare  a block per run of rows, a warp of it a head of q or k or a
//            run of value channels, the convolutions' inputs passing through registers: convolution,
//            silu, unit vectors, beta, the new tail; the thin products' inner values go to a tensor
//            of their own, the second thin product's input
//   step     a step in which every sequence brings one row: a block per (sequence, head) streams the
//            head's state through registers once (a column's dk elements in eight lanes), and then
//            normalises and gates the head's read-out
//   scan     any other step of short sequences: the columns of S are independent recurrences; a
//            column is held in the registers of eight lanes, 16 columns a block, and the rows are
//            walked in order, their q, k and g staged in shared memory 16 at a time
//   local, chain, out   a step in which a sequence brings many rows goes chunk by chunk instead
//            (channel_delta_chunk.cuh)
//   finish   after scan: one warp per (token, head) normalises and gates
//
// With s' = g s the two sums over dk that a row needs, s' . k and s' . q, are taken together:
// u = beta (v - s' . k) and o = s' . q + u (k . q), so a row costs one round of shuffles.
//
// Columns of the projection: q [G dk] | k [G dk] | v [H dv] | beta logits [H] | inner values [n_low].
// Columns of the second thin product: z [H dk] | gate logits [H dv].  A sequence's state is one row of
// floats: the convolutions' tail [taps - 1, Cc] (Cc = the convolved channels q | k | v), then S as
// [H, dv, dk], a column's dk elements side by side.  Rows of slot < 0 (padding) start from zeros
// and store nothing.
#include "attn_mma.cuh"   // the asynchronous-copy helpers
#include "short_conv.cuh"

struct ChannelDeltaArgs {
  const float* proj;       // [n_tokens, C_all]
  const float* conv_w;     // [Cc, taps], the last column is the current token's
  const float* a_log;      // [H]
  const float* dt_bias;    // [H dk]
  const float* norm_w;     // [dv]
  const int* token_seq;    // [n_tokens]
  const int* cu_q;         // [n_seqs + 1]
  const int* slots;        // [n_seqs]
  float* state;            // [slots, state_stride]
  long long state_stride;
  float* prep;             // [n_tokens, prep_stride]: unit q | unit k | v | beta [H]
  void* low;               // [n_tokens, n_low] in the activation type
  const float* wide;       // [n_tokens, H dk + H dv]: z | gate logits
  float* o;                // [n_tokens, H, dv]
  void* y;                 // [n_tokens, H dv] in the activation type
  int n_tokens, n_seqs, H, G, dk, dv, taps, n_low;
  float unit_eps, norm_eps;
  int prep_stride;         // floats between rows of prep: round4(Cc + H)
  int max_rows;            // the most rows any sequence brings (0: unknown)
  float* chunks;           // [n_tokens / 32 + n_seqs, H, record] scratch of a step that goes chunk by chunk, or null
};

__device__ __forceinline__ int cd_channels(const ChannelDeltaArgs& a) { return 2 * a.G * a.dk + a.H * a.dv; }
__device__ __forceinline__ int cd_columns(const ChannelDeltaArgs& a) { return cd_channels(a) + a.H + a.n_low; }
__device__ __forceinline__ float cd_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
// the logarithm of a channel's decay; `rate` = exp(A_log) of its head
__device__ __forceinline__ float cd_log_decay(float z, float bias, float rate) { return -rate * softplus_f(z + bias); }

#define CD_RUN 8         // rows of a run (never fewer than taps - 1)
#define CD_WARPS 8
#define CD_AHEAD 4       // rows requested at a time

// A lane's E channels among the `cols` from c0 on: E neighbours (VEC, which needs every piece on its
// boundary and whole), or every 32nd.
template <int E, bool VEC>
__device__ __forceinline__ int cd_at(int lane, int e) { return VEC ? lane * E + e : lane + 32 * e; }

template <int E, bool VEC>
__device__ __forceinline__ void cd_load(const float* p, int lane, int cols, float (&o)[E]) {
  if constexpr (VEC && E == 4) {
    const float4 x = lane * E < cols ? *reinterpret_cast<const float4*>(p + lane * E) : make_float4(0.f, 0.f, 0.f, 0.f);
    o[0] = x.x, o[1] = x.y, o[2] = x.z, o[3] = x.w;
  } else if constexpr (VEC && E == 2) {
    const float2 x = lane * E < cols ? *reinterpret_cast<const float2*>(p + lane * E) : make_float2(0.f, 0.f);
    o[0] = x.x, o[1] = x.y;
  } else {
#pragma unroll
    for (int e = 0; e < E; ++e) o[e] = cd_at<E, VEC>(lane, e) < cols ? p[cd_at<E, VEC>(lane, e)] : 0.f;
  }
}
template <int E, bool VEC>
__device__ __forceinline__ void cd_store(float* p, int lane, int cols, const float (&v)[E]) {
  if constexpr (VEC && E == 4) {
    if (lane * E < cols) *reinterpret_cast<float4*>(p + lane * E) = make_float4(v[0], v[1], v[2], v[3]);
  } else if constexpr (VEC && E == 2) {
    if (lane * E < cols) *reinterpret_cast<float2*>(p + lane * E) = make_float2(v[0], v[1]);
  } else {
#pragma unroll
    for (int e = 0; e < E; ++e)
      if (cd_at<E, VEC>(lane, e) < cols) p[cd_at<E, VEC>(lane, e)] = v[e];
  }
}

// What the rows of a run are read from.
struct CdRows {
  const float* proj;
  long long ld;
  const float* tail;       // null: zeros
  int Cc, taps, row0;
  // the input of channels c0 .. at row rr of the sequence's rows (negative: behind the step)
  template <int E, bool VEC>
  __device__ __forceinline__ void get(int rr, int c0, int cols, int lane, float (&o)[E]) const {
    const float* p = rr >= 0 ? proj + (size_t)(row0 + rr) * ld + c0
                             : (tail && rr + taps - 1 >= 0 ? tail + (size_t)(taps - 1 + rr) * Cc + c0 : nullptr);
    cd_load<E, VEC>(p, lane, p ? cols : 0, o);
  }
};

// The convolutions of E channels a lane over the rows of a run: holds the inputs of the last TAPS rows
// (TAPS 0: any number of taps, whose inputs are read again for every row).
template <int E, int TAPS, bool VEC>
struct CdWalk {
  static constexpr int W = TAPS > 0 ? TAPS : 1;
  float w[W][E], x[W][E];
  int c0, cols;
  __device__ __forceinline__ void weights(const float* conv_w, int taps, int first, int count, int lane) {
    c0 = first, cols = count;
    if (TAPS == 0) return;
#pragma unroll
    for (int e = 0; e < E; ++e) {
      const int d = cd_at<E, VEC>(lane, e);
#pragma unroll
      for (int j = 0; j < W; ++j) w[j][e] = d < cols ? conv_w[(size_t)(c0 + d) * W + W - 1 - j] : 0.f;
    }
  }
  __device__ __forceinline__ void before(const CdRows& in, int r0, int lane) {
#pragma unroll
    for (int j = 1; j < W; ++j) in.get<E, VEC>(r0 - j, c0, cols, lane, x[j - 1]);
  }
  // row rr, whose own input `fresh` is
  __device__ __forceinline__ void row(const CdRows& in, const float* conv_w, int rr, int lane, const float (&fresh)[E],
                                      float (&y)[E]) {
#pragma unroll
    for (int e = 0; e < E; ++e) y[e] = 0.f;
    if (TAPS == 0) {
      for (int j = 0; j < in.taps; ++j) {
        in.get<E, VEC>(rr - j, c0, cols, lane, x[0]);
#pragma unroll
        for (int e = 0; e < E; ++e) {
          const int d = cd_at<E, VEC>(lane, e);
          if (d < cols) y[e] = fmaf(conv_w[(size_t)(c0 + d) * in.taps + in.taps - 1 - j], x[0][e], y[e]);
        }
      }
    } else {
#pragma unroll
      for (int j = W - 1; j > 0; --j)
#pragma unroll
        for (int e = 0; e < E; ++e) x[j][e] = x[j - 1][e];
#pragma unroll
      for (int e = 0; e < E; ++e) x[0][e] = fresh[e];
#pragma unroll
      for (int e = 0; e < E; ++e)
#pragma unroll
        for (int j = 0; j < W; ++j) y[e] = fmaf(w[j][e], x[j][e], y[e]);
    }
#pragma unroll
    for (int e = 0; e < E; ++e) y[e] = silu_f(y[e]);
  }
  // The sequence's new tail, after the rows: by the owner of the channels in the first run.  When the run
  // is all of the sequence's n_seq rows the last inputs are at hand; else entry s becomes the input at
  // n_seq - (taps - 1) + s rows, read before it or anything above it is written.
  __device__ __forceinline__ void keep(const CdRows& in, float* tail, bool whole, int n_seq, int lane) {
    if (TAPS > 1 && whole) {
#pragma unroll
      for (int j = 0; j < W - 1; ++j) cd_store<E, VEC>(tail + (size_t)(W - 2 - j) * in.Cc + c0, lane, cols, x[j]);
      return;
    }
    for (int s = 0; s < in.taps - 1; ++s) {
      float v[E];
      in.get<E, VEC>(n_seq - (in.taps - 1) + s, c0, cols, lane, v);
      cd_store<E, VEC>(tail + (size_t)s * in.Cc + c0, lane, cols, v);
    }
  }
};

// A block takes a run of rows, a warp of it a head of q or k, 32 E value channels, or what is
// left of the projection (beta and the inner values).
template <int E, int TAPS, bool VEC>
__global__ void __launch_bounds__(32 * CD_WARPS) channel_delta_prepare_kernel(const ChannelDeltaArgs a, const int R, const int low16) {
  pdl_launch_dependents_if_small();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int H = a.H, G = a.G, dk = a.dk, V = H * a.dv;
  const int Cc = cd_channels(a), C_all = cd_columns(a), P = a.prep_stride;
  int seq, run;
  run_of_block(a.cu_q, a.n_seqs, R, a.max_rows == 1, blockIdx.x, seq, run);
  const int row0 = a.cu_q[seq], n_seq = a.cu_q[seq + 1] - row0;
  const int r0 = run * R, n = min(R, n_seq - r0);
  if (n <= 0) return;
  const int slot = a.slots[seq];
  float* tail = slot >= 0 && a.taps > 1 ? a.state + (size_t)slot * a.state_stride : nullptr;
  const CdRows in = {a.proj, C_all, tail, Cc, a.taps, row0};
  const int v_units = (V + 32 * E - 1) / (32 * E);
  const float q_scale = 1.0f / sqrtf((float)dk);
  // (a warp waits for the product where it first reads it: the convolutions' weights, no kernel's
  // output, are fetched before; further waits return at once)
  for (int unit = blockIdx.y * CD_WARPS + warp; unit < 2 * G + v_units + 1; unit += gridDim.y * CD_WARPS) {
    if (unit < 2 * G + v_units) {
      const bool head = unit < 2 * G;            // a q or k head, which becomes a unit vector
      const int c0 = head ? unit * dk : 2 * G * dk + (unit - 2 * G) * 32 * E;
      const int cols = head ? dk : min(32 * E, Cc - c0);
      const float scale = unit < G ? q_scale : 1.0f;
      CdWalk<E, TAPS, VEC> walk;
      walk.weights(a.conv_w, a.taps, c0, cols, lane);
      pdl_wait();
      walk.before(in, r0, lane);
      for (int i0 = 0; i0 < n; i0 += CD_AHEAD) {   // several rows are requested before the first is worked on
        float fresh[CD_AHEAD][E];
#pragma unroll
        for (int u = 0; u < CD_AHEAD; ++u)
          cd_load<E, VEC>(a.proj + (size_t)(row0 + r0 + min(i0 + u, n - 1)) * C_all + c0, lane, cols, fresh[u]);
#pragma unroll
        for (int u = 0; u < CD_AHEAD; ++u) {
          if (i0 + u >= n) break;
          float v[E], ss = 0.f;
          walk.row(in, a.conv_w, r0 + i0 + u, lane, fresh[u], v);
          if (head) {
#pragma unroll
            for (int e = 0; e < E; ++e) {
              if (cd_at<E, VEC>(lane, e) >= dk) v[e] = 0.f;
              ss = fmaf(v[e], v[e], ss);
            }
            ss = 1.0f / sqrtf(warp_sum(ss) + a.unit_eps) * scale;
#pragma unroll
            for (int e = 0; e < E; ++e) v[e] *= ss;
          }
          cd_store<E, VEC>(a.prep + (size_t)(row0 + r0 + i0 + u) * P + c0, lane, cols, v);
        }
      }
      if (tail && run == 0) walk.keep(in, tail, n == n_seq, n_seq, lane);
    } else {
      pdl_wait();
      for (int i = 0; i < n; ++i) {
        const size_t t = row0 + r0 + i;
        const float* rest = a.proj + t * C_all + Cc;
        for (int h = lane; h < H; h += 32) a.prep[t * P + Cc + h] = cd_sigmoid(rest[h]);
        for (int j = lane; j < a.n_low; j += 32) {
          if (low16) ((bf16*)a.low)[t * a.n_low + j] = from_f32<bf16>(rest[H + j]);
          else ((float*)a.low)[t * a.n_low + j] = rest[H + j];
        }
      }
    }
  }
  pdl_wait();              // (a warp without a unit waits, too: a finished kernel has waited for the one before)
  pdl_launch_dependents_if_large();
}

#define CD_LANES 8       // lanes that share a column of S
#define CD_COLS 16       // columns of S per block of the scan
#define CD_TT 16         // rows staged together

// R floats of a column per lane, in pieces of four: piece i of lane l holds the elements
// (i * 8 + l) * 4 .. + 3, so that the lanes of a column read contiguous bytes at a time.
template <int R>
__device__ __forceinline__ void cd_load_column(float (&S)[R], const float* sp, int dk, int l, bool wide) {
#pragma unroll
  for (int i = 0; i < R / 4; ++i) {
    const int e = (i * CD_LANES + l) * 4;
    if (wide) {
      const float4 x = sp && e < dk ? *reinterpret_cast<const float4*>(sp + e) : make_float4(0.f, 0.f, 0.f, 0.f);
      S[4 * i] = x.x, S[4 * i + 1] = x.y, S[4 * i + 2] = x.z, S[4 * i + 3] = x.w;
    } else {
#pragma unroll
      for (int x = 0; x < 4; ++x) S[4 * i + x] = sp && e + x < dk ? sp[e + x] : 0.f;
    }
  }
}
template <int R>
__device__ __forceinline__ void cd_store_column(const float (&S)[R], float* sp, int dk, int l, bool wide) {
#pragma unroll
  for (int i = 0; i < R / 4; ++i) {
    const int e = (i * CD_LANES + l) * 4;
    if (wide) {
      if (e < dk) *reinterpret_cast<float4*>(sp + e) = make_float4(S[4 * i], S[4 * i + 1], S[4 * i + 2], S[4 * i + 3]);
    } else {
#pragma unroll
      for (int x = 0; x < 4; ++x)
        if (e + x < dk) sp[e + x] = S[4 * i + x];
    }
  }
}

// One row of a column: S <- g S + k u with u = beta (v - (g S) . k); returns (g S) . q + u (k . q).
// (The lanes of every column take k . q anew: one more value in the same round of shuffles.)
template <int R>
__device__ __forceinline__ float cd_row(float (&S)[R], const float* q, const float* k, const float* g, int l,
                                        float v, float beta) {
  float kk[R], d1 = 0.f, d2 = 0.f, kq = 0.f;
#pragma unroll
  for (int i = 0; i < R / 4; ++i) {
    const float4 k4 = reinterpret_cast<const float4*>(k)[i * CD_LANES + l];
    const float4 q4 = reinterpret_cast<const float4*>(q)[i * CD_LANES + l];
    const float4 g4 = reinterpret_cast<const float4*>(g)[i * CD_LANES + l];
    S[4 * i] *= g4.x, S[4 * i + 1] *= g4.y, S[4 * i + 2] *= g4.z, S[4 * i + 3] *= g4.w;
    kk[4 * i] = k4.x, kk[4 * i + 1] = k4.y, kk[4 * i + 2] = k4.z, kk[4 * i + 3] = k4.w;
    d1 = fmaf(S[4 * i], k4.x, d1), d1 = fmaf(S[4 * i + 1], k4.y, d1);
    d1 = fmaf(S[4 * i + 2], k4.z, d1), d1 = fmaf(S[4 * i + 3], k4.w, d1);
    d2 = fmaf(S[4 * i], q4.x, d2), d2 = fmaf(S[4 * i + 1], q4.y, d2);
    d2 = fmaf(S[4 * i + 2], q4.z, d2), d2 = fmaf(S[4 * i + 3], q4.w, d2);
    kq = fmaf(k4.x, q4.x, kq), kq = fmaf(k4.y, q4.y, kq), kq = fmaf(k4.z, q4.z, kq), kq = fmaf(k4.w, q4.w, kq);
  }
#pragma unroll
  for (int m = 1; m < CD_LANES; m <<= 1) {
    d1 += __shfl_xor_sync(0xffffffffu, d1, m);
    d2 += __shfl_xor_sync(0xffffffffu, d2, m);
    kq += __shfl_xor_sync(0xffffffffu, kq, m);
  }
  const float u = beta * (v - d1);
#pragma unroll
  for (int x = 0; x < R; ++x) S[x] = fmaf(kk[x], u, S[x]);
  return fmaf(u, kq, d2);
}

template <typename T, int R>
__global__ void __launch_bounds__(256) channel_delta_step_kernel(const ChannelDeltaArgs a) {
  extern __shared__ __align__(16) float sm[];     // q | k | g [DKP each] | o [dv]
  __shared__ float scratch[32];
  constexpr int DKP = CD_LANES * R;               // dk filled up with zeros
  constexpr int COLS = 256 / CD_LANES;            // columns of a pass
  pdl_launch_dependents_if_small();
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x;
  const int H = a.H, G = a.G, dk = a.dk, dv = a.dv, kvh = h / (H / G);
  const int Cc = cd_channels(a), C_all = cd_columns(a);
  const int t = a.cu_q[seq], slot = a.slots[seq];
  float *qs = sm, *ks = sm + DKP, *gs = sm + 2 * DKP, *os = sm + 3 * DKP;
  const float rate = expf(a.a_log[h]);
  float* head = slot >= 0 ? a.state + (size_t)slot * a.state_stride + (size_t)(a.taps - 1) * Cc + (size_t)h * dv * dk
                          : nullptr;
  const bool wide = (dk & 3) == 0 && (((uintptr_t)head) & 15) == 0;
  if (head)                                       // on its way to L2 while the kernel before drains
    for (int i = tid * 32; i < dk * dv; i += 256 * 32)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(head + i));
  pdl_wait();
  if (a.cu_q[seq + 1] - t <= 0) return;
  const float* p = a.prep + (size_t)t * a.prep_stride;
  const float* z = a.wide + (size_t)t * ((size_t)H * (dk + dv));
  for (int d = tid; d < DKP; d += 256) {
    const bool in = d < dk;
    qs[d] = in ? p[kvh * dk + d] : 0.f;
    ks[d] = in ? p[(G + kvh) * dk + d] : 0.f;
    gs[d] = in ? expf(cd_log_decay(z[h * dk + d], a.dt_bias[h * dk + d], rate)) : 0.f;
  }
  const float beta = p[Cc + h];
  __syncthreads();
  const int l = tid % CD_LANES;
  float ss = 0.f;
  for (int c0 = 0; c0 < dv; c0 += 2 * COLS) {     // two columns a thread group: their loads go together
    const int ca = c0 + tid / CD_LANES, cb = ca + COLS;
    float Sa[R], Sb[R];
    cd_load_column<R>(Sa, head && ca < dv ? head + (size_t)ca * dk : nullptr, dk, l, wide);
    cd_load_column<R>(Sb, head && cb < dv ? head + (size_t)cb * dk : nullptr, dk, l, wide);
    const float va = ca < dv ? p[2 * G * dk + h * dv + ca] : 0.f, vb = cb < dv ? p[2 * G * dk + h * dv + cb] : 0.f;
    const float oa = cd_row<R>(Sa, qs, ks, gs, l, va, beta);
    const float ob = cd_row<R>(Sb, qs, ks, gs, l, vb, beta);
    if (head && ca < dv) cd_store_column<R>(Sa, head + (size_t)ca * dk, dk, l, wide);
    if (head && cb < dv) cd_store_column<R>(Sb, head + (size_t)cb * dk, dk, l, wide);
    if (l == 0 && ca < dv) os[ca] = oa, ss = fmaf(oa, oa, ss);
    if (l == 0 && cb < dv) os[cb] = ob, ss = fmaf(ob, ob, ss);
  }
  pdl_launch_dependents_if_large();
  const float inv = 1.0f / sqrtf(block_sum(ss, scratch) / (float)dv + a.norm_eps);   // (its barriers publish os)
  const float* gate = z + (size_t)H * dk + (size_t)h * dv;
  T* y = (T*)a.y + ((size_t)t * H + h) * dv;
  for (int j = tid; j < dv; j += 256) y[j] = from_f32<T>(os[j] * inv * a.norm_w[j] * cd_sigmoid(gate[j]));
}

template <int R>
__global__ void __launch_bounds__(CD_LANES * CD_COLS) channel_delta_scan_kernel(const ChannelDeltaArgs a) {
  extern __shared__ __align__(16) float sm[];     // q | k | g [CD_TT, DKP each] | v [CD_TT, CD_COLS] | beta [CD_TT]
  constexpr int DKP = CD_LANES * R;
  pdl_launch_dependents_if_small();
  const int seq = blockIdx.z, h = blockIdx.y, tid = threadIdx.x;
  const int col0 = blockIdx.x * CD_COLS, col = col0 + tid / CD_LANES, l = tid % CD_LANES;
  const int H = a.H, G = a.G, dk = a.dk, dv = a.dv, kvh = h / (H / G);
  const int Cc = cd_channels(a);
  float *qs = sm, *ks = qs + CD_TT * DKP, *gs = ks + CD_TT * DKP, *vs = gs + CD_TT * DKP, *bs = vs + CD_TT * CD_COLS;
  const float rate = expf(a.a_log[h]);
  pdl_wait();
  const int row0 = a.cu_q[seq], n = a.cu_q[seq + 1] - row0;
  if (n <= 0) return;
  const int slot = a.slots[seq];
  const bool active = col < dv;
  float* sp = slot >= 0 && active ? a.state + (size_t)slot * a.state_stride + (size_t)(a.taps - 1) * Cc +
                                        ((size_t)h * dv + col) * dk
                                  : nullptr;
  const bool wide = (dk & 3) == 0 && (((uintptr_t)sp) & 15) == 0;
  float S[R];
  cd_load_column<R>(S, sp, dk, l, wide);
  for (int t0 = 0; t0 < n; t0 += CD_TT) {
    const int nt = min(CD_TT, n - t0);
    __syncthreads();
    for (int i = tid; i < nt * DKP; i += CD_LANES * CD_COLS) {
      const int tt = i / DKP, d = i % DKP, t = row0 + t0 + tt;
      const float* p = a.prep + (size_t)t * a.prep_stride;
      const bool in = d < dk;
      qs[i] = in ? p[kvh * dk + d] : 0.f;
      ks[i] = in ? p[(G + kvh) * dk + d] : 0.f;
      gs[i] = in ? expf(cd_log_decay(a.wide[(size_t)t * H * (dk + dv) + h * dk + d], a.dt_bias[h * dk + d], rate)) : 0.f;
    }
    for (int i = tid; i < nt * CD_COLS; i += CD_LANES * CD_COLS) {
      const int c = col0 + i % CD_COLS;
      vs[i] = c < dv ? a.prep[(size_t)(row0 + t0 + i / CD_COLS) * a.prep_stride + 2 * G * dk + h * dv + c] : 0.f;
    }
    if (tid < nt) bs[tid] = a.prep[(size_t)(row0 + t0 + tid) * a.prep_stride + Cc + h];
    __syncthreads();
    for (int tt = 0; tt < nt; ++tt) {
      const float o = cd_row<R>(S, qs + tt * DKP, ks + tt * DKP, gs + tt * DKP, l, vs[tt * CD_COLS + tid / CD_LANES],
                                bs[tt]);
      if (l == 0 && active) a.o[((size_t)(row0 + t0 + tt) * H + h) * dv + col] = o;
    }
  }
  pdl_launch_dependents_if_large();
  if (sp) cd_store_column<R>(S, sp, dk, l, wide);
}

template <typename T>
__global__ void channel_delta_finish_kernel(const ChannelDeltaArgs a) {
  pdl_launch_dependents_if_small();
  pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int nwarps = blockDim.x >> 5;
  const int H = a.H, dk = a.dk, dv = a.dv;
  for (int h = blockIdx.y * nwarps + warp; h < H; h += gridDim.y * nwarps) {
    const float* o = a.o + ((size_t)t * H + h) * dv;
    const float* gate = a.wide + (size_t)t * H * (dk + dv) + (size_t)H * dk + (size_t)h * dv;
    float ss = 0.f;
    for (int j = lane; j < dv; j += 32) ss += o[j] * o[j];
    ss = warp_sum(ss);
    const float inv = 1.0f / sqrtf(ss / (float)dv + a.norm_eps);
    T* y = (T*)a.y + ((size_t)t * H + h) * dv;
    for (int j = lane; j < dv; j += 32) y[j] = from_f32<T>(o[j] * inv * a.norm_w[j] * cd_sigmoid(gate[j]));
  }
  pdl_launch_dependents_if_large();
}

#include "channel_delta_chunk.cuh"

static int cd_check(const ChannelDeltaArgs& a) {
  if (a.n_tokens < 0 || a.n_seqs <= 0 || a.H <= 0 || a.G <= 0 || a.H % a.G || a.dk <= 0 || a.dv <= 0 || a.taps <= 0 ||
      a.n_low <= 0 || !a.proj || !a.state || !a.prep || !a.low || !a.conv_w || !a.token_seq || !a.cu_q || !a.slots)
    return GB_ERR_BAD_ARG;
  if (a.dk > 32 * CD_LANES || a.n_seqs > 65535 || a.H > 65535) return GB_ERR_UNSUPPORTED;
  if (a.prep_stride != (2 * a.G * a.dk + a.H * a.dv + a.H + 3) / 4 * 4) return GB_ERR_BAD_ARG;
  return 0;
}

template <int E, int TAPS>
static int prepare_taps(const ChannelDeltaArgs& a, int low16, cudaStream_t s) {
  int R = a.n_tokens >= 1024 ? 2 * CD_RUN : CD_RUN;      // (long runs read fewer rows twice)
  if (a.taps - 1 > R) R = a.taps - 1;
  const int blocks = a.max_rows == 1 ? a.n_seqs : a.n_tokens / R + a.n_seqs;
  const int units = 2 * a.G + (a.H * a.dv + 32 * E - 1) / (32 * E) + 1;
  const dim3 grid(blocks, (units + CD_WARPS - 1) / CD_WARPS), block(32 * CD_WARPS);
  const int Cc = 2 * a.G * a.dk + a.H * a.dv;
  const bool vec = E <= 4 && a.dk % E == 0 && (a.H * a.dv) % E == 0 && (Cc + a.H + a.n_low) % E == 0 &&
                   a.state_stride % E == 0 && (((uintptr_t)a.proj | (uintptr_t)a.state | (uintptr_t)a.prep) & 15) == 0;
  if constexpr (E <= 4)
    if (vec) return gb_launch(channel_delta_prepare_kernel<E, TAPS, true>, grid, block, 0, s, a, R, low16);
  return gb_launch(channel_delta_prepare_kernel<E, TAPS, false>, grid, block, 0, s, a, R, low16);
}

template <int E>
static int prepare_size(const ChannelDeltaArgs& a, int low16, cudaStream_t s) {
  switch (a.taps) {
    case 2: return prepare_taps<E, 2>(a, low16, s);
    case 3: return prepare_taps<E, 3>(a, low16, s);
    case 4: return prepare_taps<E, 4>(a, low16, s);
    default: return prepare_taps<E, 0>(a, low16, s);
  }
}

static int prepare(const ChannelDeltaArgs& a, int low16, cudaStream_t s) {
  const int e = cd_check(a);
  if (e || a.n_tokens == 0) return e;
  return a.dk <= 128 ? prepare_size<4>(a, low16, s) : prepare_size<8>(a, low16, s);
}

template <typename T, int R>
static int run_rows(const ChannelDeltaArgs& a, cudaStream_t s) {
  constexpr int DKP = CD_LANES * R;
  if (a.max_rows == 1) {
    const size_t smem = (3 * DKP + a.dv) * sizeof(float);
    if (smem > 48 * 1024) return GB_ERR_UNSUPPORTED;
    return gb_launch(channel_delta_step_kernel<T, R>, dim3(a.H, a.n_seqs), dim3(256), smem, s, a);
  }
  if (cc_takes(a)) return cc_run<T>(a, s);
  const size_t smem = (CD_TT * (3 * DKP + CD_COLS + 1)) * sizeof(float);
  static bool configured = false;
  if (smem > 48 * 1024 && !configured) {
    cudaError_t ce = cudaFuncSetAttribute(channel_delta_scan_kernel<R>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                          (int)smem);
    if (ce != cudaSuccess) return (int)ce;
    configured = true;
  }
  const int e = gb_launch(channel_delta_scan_kernel<R>, dim3((a.dv + CD_COLS - 1) / CD_COLS, a.H, a.n_seqs),
                          dim3(CD_LANES * CD_COLS), smem, s, a);
  if (e) return e;
  const int warps = a.H < 8 ? a.H : 8;
  return gb_launch(channel_delta_finish_kernel<T>, dim3(a.n_tokens, (a.H + warps - 1) / warps), dim3(warps * 32), 0, s, a);
}

template <typename T>
static int run(const ChannelDeltaArgs& a, cudaStream_t s) {
  const int e = cd_check(a);
  if (e) return e;
  if (!a.wide || !a.a_log || !a.dt_bias || !a.norm_w || !a.o || !a.y) return GB_ERR_BAD_ARG;
  if (a.n_tokens == 0) return 0;
  const int per_lane = (a.dk + CD_LANES - 1) / CD_LANES;
  if (per_lane <= 4) return run_rows<T, 4>(a, s);
  if (per_lane <= 8) return run_rows<T, 8>(a, s);
  if (per_lane <= 12) return run_rows<T, 12>(a, s);
  if (per_lane <= 16) return run_rows<T, 16>(a, s);
  if (per_lane <= 24) return run_rows<T, 24>(a, s);
  return run_rows<T, 32>(a, s);
}

GB_EXPORT int gb_channel_delta_prepare_f32(const ChannelDeltaArgs* a, cudaStream_t s) { return prepare(*a, 0, s); }
GB_EXPORT int gb_channel_delta_prepare_bf16(const ChannelDeltaArgs* a, cudaStream_t s) { return prepare(*a, 1, s); }
GB_EXPORT int gb_channel_delta_run_f32(const ChannelDeltaArgs* a, cudaStream_t s) { return run<float>(*a, s); }
GB_EXPORT int gb_channel_delta_run_bf16(const ChannelDeltaArgs* a, cudaStream_t s) { return run<bf16>(*a, s); }
