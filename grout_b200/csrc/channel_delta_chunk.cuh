// The delta rule with a decay per channel, chunk by chunk (included by channel_delta.cu; the
// notation is that file's).  With L_t the sums of log g from a chunk's first row to row t
// (per channel) and S_0 the state in front of the chunk, the rows of a chunk obey
//
//   u_t = beta_t (v_t - S_0^T (e^{L_t} k_t) - sum_{i<t} A_ti u_i),   A_ti = sum_d k_td k_id e^{L_td - L_id}
//   o_t = S_0^T (e^{L_t} q_t) + sum_{i<=t} B_ti u_i,                 B_ti = sum_d q_td k_id e^{L_td - L_id}
//   S_n = diag(e^{L_n}) S_0 + sum_i (e^{L_n - L_i} k_i) u_i^T
//
// The first line is a triangular system: u = X v - (W) S_0 with both X v and W from one forward
// substitution that knows nothing of S_0.  So
//
//   local   takes every chunk of every head at the same time: A, B, the substitution for the dv + dk
//           right-hand sides beta v and beta e^{L} k, and leaves the chunk's record
//   chain   walks a sequence's chunks in order, a block per head and CC_COLS columns of S with the
//           state in shared memory: U = U0 - W S and the next state, tiled 32-bit products; it leaves
//           U and the state in front of every chunk in the record
//   out     takes every chunk of every head at the same time again: the read-outs, one product of
//           the record's [e^{L} q | B] with [S_0 ; U], and their norm and gate
//
// Every exponent that is taken is not positive and is summed up from logarithms of one sign, never a
// difference of two running sums (rows of the same half chunk directly, others by way of the end of
// the first half): no quotient of decays overflows, and none loses its digits behind a strong one.
#pragma once

#define CC_ROWS 32       // rows of a chunk
#define CC_HALF 16
#define CC_COLS 32       // columns of S a chain block owns
#define CC_MIN 64        // a step goes chunk by chunk when a sequence brings this many rows
#define CC_MAX_DK 128
#define CC_MAX_DV 1024
#define CC_LOG2E 1.4426950408889634f   // the kernels keep logarithms to base 2: one operation less per power

// A chunk's record for one head: W [dk][32] (per channel the 32 rows) | Kd [32][dk] (e^{L_n - L} k) |
// gC [dk] (e^{L_n}) | QB [dk + 32][32] (per channel the rows of e^L q, then per row i the column of
// B) | SU [dk + 32][dv] (S_0, then U0, which becomes U)
__host__ __device__ __forceinline__ size_t cc_record(int dk, int dv) {
  return (size_t)2 * dk * CC_ROWS + dk + (size_t)(dk + CC_ROWS) * (CC_ROWS + dv);
}
__host__ __device__ __forceinline__ int cc_at_qb(int dk) { return 2 * dk * CC_ROWS + dk; }
__host__ __device__ __forceinline__ int cc_at_su(int dk) { return cc_at_qb(dk) + (dk + CC_ROWS) * CC_ROWS; }
// Chunk z of a sequence whose rows start at `first` has an entry that no other chunk has.
__host__ __device__ __forceinline__ size_t cc_entry(int first, int z, int seq) {
  return (size_t)(first / CC_ROWS + z + seq);
}

// Sums over the warp's lanes of 32 values a lane holds: lane i gets the sum of value i.
__device__ __forceinline__ float cc_transpose_sum(float (&v)[32], int lane) {
#pragma unroll
  for (int m = 16; m > 0; m >>= 1) {
    const bool up = lane & m;
#pragma unroll
    for (int i = 0; i < m; ++i) {
      const float give = up ? v[i] : v[i + m], keep = up ? v[i + m] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, m);
    }
  }
  return v[0];
}

template <int E>
__device__ __forceinline__ void cc_read(const float* p, float (&o)[E]) {
  if constexpr (E == 4) {
    const float4 x = *reinterpret_cast<const float4*>(p);
    o[0] = x.x, o[1] = x.y, o[2] = x.z, o[3] = x.w;
  } else if constexpr (E == 2) {
    const float2 x = *reinterpret_cast<const float2*>(p);
    o[0] = x.x, o[1] = x.y;
  } else {
    o[0] = p[0];
  }
}

// E channels a lane: heads of up to 32 E.  The block's rows, zero beyond dk and beyond the chunk's end.
template <int E>
__global__ void __launch_bounds__(256, 2) channel_delta_local_kernel(const ChannelDeltaArgs a) {
  constexpr int DKP = 32 * E, LD = DKP + 4;      // (16-byte rows; a column's rows on different banks)
  extern __shared__ __align__(16) float sm[];
  float *Ks = sm, *Qs = Ks + CC_ROWS * LD, *Ls = Qs + CC_ROWS * LD, *Fs = Ls + CC_ROWS * LD;
  float *Kr = Fs + CC_ROWS * LD;                 // [16][LD]: the first half's keys, faded to its end
  float *As = Kr + CC_HALF * LD, *Bs = As + CC_ROWS * CC_ROWS, *beta = Bs + CC_ROWS * CC_ROWS;
  pdl_launch_dependents_if_small();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, seq = blockIdx.z, z = blockIdx.x;
  const int H = a.H, G = a.G, dk = a.dk, dv = a.dv, kvh = h / (H / G), Cc = cd_channels(a);
  const float rate = expf(a.a_log[h]);
  pdl_wait();
  const int first = a.cu_q[seq], n_seq = a.cu_q[seq + 1] - first;
  const int n = min(CC_ROWS, n_seq - z * CC_ROWS), row0 = first + z * CC_ROWS;
  if (n <= 0) return;
#pragma unroll 4
  for (int i = tid; i < CC_ROWS * DKP; i += 256) {
    const int t = i / DKP, d = i % DKP;
    float q = 0.f, k = 0.f, lg = 0.f;
    if (t < n && d < dk) {
      const float* p = a.prep + (size_t)(row0 + t) * a.prep_stride;
      q = p[kvh * dk + d], k = p[(G + kvh) * dk + d];
      lg = CC_LOG2E * cd_log_decay(a.wide[(size_t)(row0 + t) * H * (dk + dv) + h * dk + d], a.dt_bias[h * dk + d], rate);
    }
    Qs[t * LD + d] = q, Ks[t * LD + d] = k, Ls[t * LD + d] = lg;
  }
  if (tid < CC_ROWS) beta[tid] = tid < n ? a.prep[(size_t)(row0 + tid) * a.prep_stride + Cc + h] : 0.f;
  __syncthreads();
  const size_t entry = (cc_entry(first, z, seq) * H + h) * cc_record(dk, dv);
  float* wq = a.chunks + entry;
  float* kd = wq + (size_t)dk * CC_ROWS;
  float* gc = kd + (size_t)CC_ROWS * dk;
  float* qb = wq + cc_at_qb(dk);
  float* u0 = wq + cc_at_su(dk) + (size_t)dk * dv;
  // per channel: Fs, the logarithms summed up from the start of a row's half chunk on; and, from the
  // chunk's end back, what is left of a row's key at the end of its half and of the chunk (rows
  // beyond the chunk's end have no decay)
  if (tid < DKP) {
    float s = 0.f;
#pragma unroll 8
    for (int t = 0; t < CC_ROWS; ++t) {
      if (t == CC_HALF) s = 0.f;
      s += Ls[t * LD + tid];
      Fs[t * LD + tid] = s;
    }
  } else if (tid >= 128 && tid - 128 < DKP) {
    const int d = tid - 128;
    float s = 0.f, in_half = 0.f;
#pragma unroll 4
    for (int t = CC_ROWS - 1; t >= 0; --t) {
      const float k = Ks[t * LD + d], lg = Ls[t * LD + d];
      if (d < dk) kd[t * dk + d] = k * exp2f(s);
      if (t < CC_HALF) {
        Kr[t * LD + d] = k * exp2f(in_half);
        in_half += lg;
      }
      s += lg;
    }
    if (d < dk) gc[d] = exp2f(s);
  }
  __syncthreads();
  // A and B: a warp takes rows warp, warp + 8, ...; its lanes share the channels
  for (int t = warp; t < CC_ROWS; t += 8) {
    float kt[E], qt[E], ki[E], li[E], since[E], part[32];
    cc_read<E>(Ks + t * LD + lane * E, kt);
    cc_read<E>(Qs + t * LD + lane * E, qt);
    const int base = t & CC_HALF;                // the first row of t's half chunk
#pragma unroll
    for (int x = 0; x < E; ++x) since[x] = 0.f;  // the logarithms behind row base + j, up to t's
#pragma unroll
    for (int j = CC_HALF - 1; j >= 0; --j) {
      part[j] = part[CC_HALF + j] = 0.f;
      if (base + j <= t) {
        cc_read<E>(Ks + (base + j) * LD + lane * E, ki);
        cc_read<E>(Ls + (base + j) * LD + lane * E, li);
#pragma unroll
        for (int x = 0; x < E; ++x) {
          const float w = ki[x] * exp2f(since[x]);
          since[x] += li[x];
          part[j] = fmaf(kt[x], w, part[j]);
          part[CC_HALF + j] = fmaf(qt[x], w, part[CC_HALF + j]);
        }
      }
    }
    float sum = cc_transpose_sum(part, lane);    // lanes 0 .. 15: A, 16 .. 31: B
    const int j = lane & (CC_HALF - 1);
    if (lane < CC_HALF) As[t * CC_ROWS + base + j] = base + j < t ? sum : 0.f;
    else Bs[t * CC_ROWS + base + j] = base + j <= t ? sum : 0.f;
    if (base) {                                  // the other half, by way of its last row
      cc_read<E>(Fs + t * LD + lane * E, li);
#pragma unroll
      for (int x = 0; x < E; ++x) {
        const float w = exp2f(li[x]);
        kt[x] *= w, qt[x] *= w;
      }
#pragma unroll
      for (int i = 0; i < CC_HALF; ++i) {
        part[i] = part[CC_HALF + i] = 0.f;
        cc_read<E>(Kr + i * LD + lane * E, ki);
#pragma unroll
        for (int x = 0; x < E; ++x) {
          part[i] = fmaf(kt[x], ki[x], part[i]);
          part[CC_HALF + i] = fmaf(qt[x], ki[x], part[CC_HALF + i]);
        }
      }
      sum = cc_transpose_sum(part, lane);
      (lane < CC_HALF ? As : Bs)[t * CC_ROWS + j] = sum;
    } else {
      (lane < CC_HALF ? As : Bs)[t * CC_ROWS + CC_HALF + j] = 0.f;
    }
  }
  __syncthreads();
  // the substitution: a thread takes one right-hand side (dv of values, then dk of e^{L} k)
  for (int c = tid; c < dv + dk; c += 256) {
    float x[CC_ROWS];
    const int d = c - dv;
#pragma unroll
    for (int t = 0; t < CC_ROWS; ++t) {
      if (d < 0) x[t] = t < n ? a.prep[(size_t)(row0 + t) * a.prep_stride + 2 * G * dk + h * dv + c] : 0.f;
      else x[t] = Ks[t * LD + d] * exp2f(Fs[t * LD + d] + (t < CC_HALF ? 0.f : Fs[(CC_HALF - 1) * LD + d]));
    }
#pragma unroll
    for (int t = 0; t < CC_ROWS; ++t) {
      float s = x[t];
#pragma unroll
      for (int i0 = 0; i0 < t; i0 += 4) {        // (entries of A from the diagonal on are zero, x there still finite)
        const float4 w = *reinterpret_cast<const float4*>(As + t * CC_ROWS + i0);
        s = fmaf(-w.x, x[i0], s);
        if (i0 + 1 < t) s = fmaf(-w.y, x[i0 + 1], s);
        if (i0 + 2 < t) s = fmaf(-w.z, x[i0 + 2], s);
        if (i0 + 3 < t) s = fmaf(-w.w, x[i0 + 3], s);
      }
      x[t] = beta[t] * s;
    }
    if (d < 0) {
#pragma unroll
      for (int t = 0; t < CC_ROWS; ++t) u0[(size_t)t * dv + c] = x[t];
    } else {
      float4* out = reinterpret_cast<float4*>(wq + (size_t)d * CC_ROWS);
#pragma unroll
      for (int t = 0; t < CC_ROWS; t += 4) out[t / 4] = make_float4(x[t], x[t + 1], x[t + 2], x[t + 3]);
    }
  }
  pdl_launch_dependents_if_large();
  for (int i = tid; i < 8 * dk; i += 256) {      // e^{L} q, four rows of a channel a thread
    const int d = i / 8, t = (i % 8) * 4;
    const float before = t < CC_HALF ? 0.f : Fs[(CC_HALF - 1) * LD + d];
    float v[4];
#pragma unroll
    for (int x = 0; x < 4; ++x) v[x] = Qs[(t + x) * LD + d] * exp2f(Fs[(t + x) * LD + d] + before);
    *reinterpret_cast<float4*>(qb + (size_t)d * CC_ROWS + t) = make_float4(v[0], v[1], v[2], v[3]);
  }
  for (int i = tid; i < CC_ROWS * CC_ROWS; i += 256)     // B by columns
    qb[(size_t)dk * CC_ROWS + i] = Bs[(i % CC_ROWS) * CC_ROWS + i / CC_ROWS];
}

__device__ __forceinline__ void cc_copy16(float* smem, const float* gmem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(s), "l"(gmem));
}

// floats of a chain block's stage: W | Kd | gC | U0's columns
__host__ __device__ __forceinline__ int cc_stage(int dk) { return 2 * dk * CC_ROWS + dk + CC_ROWS * CC_COLS; }

__global__ void __launch_bounds__(256) channel_delta_chain_kernel(const ChannelDeltaArgs a) {
  extern __shared__ __align__(16) float sm[];
  pdl_launch_dependents_if_small();
  const int tid = threadIdx.x;
  const int h = blockIdx.y, seq = blockIdx.z, col0 = blockIdx.x * CC_COLS;
  const int H = a.H, dk = a.dk, dv = a.dv, Cc = cd_channels(a);
  const int stage = cc_stage(dk);
  float* S = sm + 2 * stage;                     // [dk][CC_COLS]
  float* P = S + dk * CC_COLS;                   // [4][CC_ROWS][CC_COLS]: a quarter of the channels' part of W S each
  float* U = P + 4 * CC_ROWS * CC_COLS;          // [CC_ROWS][CC_COLS]
  pdl_wait();
  const int first = a.cu_q[seq], n_seq = a.cu_q[seq + 1] - first;
  if (n_seq <= 0) return;
  const int slot = a.slots[seq];
  float* sp = slot >= 0 ? a.state + (size_t)slot * a.state_stride + (size_t)(a.taps - 1) * Cc + (size_t)h * dv * dk
                        : nullptr;
  const int chunks = (n_seq + CC_ROWS - 1) / CC_ROWS;
  auto record = [&](int z) { return a.chunks + (cc_entry(first, z, seq) * H + h) * cc_record(dk, dv); };
  const int whole = 2 * dk * CC_ROWS + dk;                 // (dk is a multiple of four)
  auto stage_in = [&](int z) {
    float* dst = sm + (z & 1) * stage;
    const float* src = record(z);
    for (int i = tid * 4; i < whole; i += 1024) cc_copy16(dst + i, src + i);
    const int t = tid / 8, c = (tid % 8) * 4;
    if (col0 + c < dv) cc_copy16(dst + whole + t * CC_COLS + c, src + cc_at_su(dk) + (size_t)(dk + t) * dv + col0 + c);
    cp_async_commit();
  };
  for (int s = 0; s < 2 && col0 + CC_COLS > dv; ++s)       // columns no copy brings
    for (int i = tid; i < CC_ROWS * CC_COLS; i += 256)
      if (col0 + i % CC_COLS >= dv) sm[s * stage + whole + i] = 0.f;
  stage_in(0);
  // the state: element (k, c) of the head's matrix lies at c dk + k
  for (int i = tid; i < dk * CC_COLS; i += 256) {
    const int c = i / dk, k = i % dk;
    S[k * CC_COLS + c] = sp && col0 + c < dv ? sp[(size_t)(col0 + c) * dk + k] : 0.f;
  }
  // tiles: 4 rows by 4 columns of W S a thread, a quarter of the channels each; 4 by 4 of the state
  const int quarter = tid >> 6, tr = (tid & 63) / 8 * 4, tc = (tid & 7) * 4;
  const int per = (dk + 3) / 4, k_lo = quarter * per, k_hi = min(dk, k_lo + per);
  const int sk = tid / 8 * 4, urow = tid / 8;
  const bool col_in = col0 + tc < dv;                      // (dv is a multiple of four)
  for (int z = 0; z < chunks; ++z) {
    if (z + 1 < chunks) { stage_in(z + 1); cp_async_wait<1>(); } else { cp_async_wait<0>(); }
    __syncthreads();
    const float* w = sm + (z & 1) * stage;
    const float* kd = w + dk * CC_ROWS;
    const float* gc = kd + CC_ROWS * dk;
    const float* u0 = gc + dk;
    float* su = record(z) + cc_at_su(dk) + col0 + tc;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll 8
    for (int k = k_lo; k < k_hi; ++k) {
      const float4 x = *reinterpret_cast<const float4*>(w + k * CC_ROWS + tr);
      const float4 y = *reinterpret_cast<const float4*>(S + k * CC_COLS + tc);
      const float xv[4] = {x.x, x.y, x.z, x.w}, yv[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], yv[j], acc[i][j]);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
      *reinterpret_cast<float4*>(P + (quarter * CC_ROWS + tr + i) * CC_COLS + tc) =
          make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    __syncthreads();
    {                                            // U = U0 - W S, four columns of a row a thread
      float4 u = *reinterpret_cast<const float4*>(u0 + urow * CC_COLS + tc);
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const float4 x = *reinterpret_cast<const float4*>(P + (q * CC_ROWS + urow) * CC_COLS + tc);
        u.x -= x.x, u.y -= x.y, u.z -= x.z, u.w -= x.w;
      }
      *reinterpret_cast<float4*>(U + urow * CC_COLS + tc) = u;
      if (col_in) *reinterpret_cast<float4*>(su + (size_t)(dk + urow) * dv) = u;
    }
    __syncthreads();
    if (sk < dk) {                               // S <- diag(e^{L_n}) S + Kd^T U
      float s[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float4 x = *reinterpret_cast<const float4*>(S + (sk + i) * CC_COLS + tc);
        if (col_in) *reinterpret_cast<float4*>(su + (size_t)(sk + i) * dv) = x;
        const float g = gc[sk + i];
        s[i][0] = g * x.x, s[i][1] = g * x.y, s[i][2] = g * x.z, s[i][3] = g * x.w;
      }
#pragma unroll 8
      for (int t = 0; t < CC_ROWS; ++t) {
        const float4 x = *reinterpret_cast<const float4*>(kd + t * dk + sk);
        const float4 y = *reinterpret_cast<const float4*>(U + t * CC_COLS + tc);
        const float xv[4] = {x.x, x.y, x.z, x.w}, yv[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) s[i][j] = fmaf(xv[i], yv[j], s[i][j]);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
        *reinterpret_cast<float4*>(S + (sk + i) * CC_COLS + tc) = make_float4(s[i][0], s[i][1], s[i][2], s[i][3]);
    }
    __syncthreads();                             // S is whole, the stage and P may be overwritten
  }
  pdl_launch_dependents_if_large();
  if (sp)
    for (int i = tid; i < dk * CC_COLS; i += 256) {
      const int c = i / dk, k = i % dk;
      if (col0 + c < dv) sp[(size_t)(col0 + c) * dk + k] = S[k * CC_COLS + c];
    }
}

// The read-outs of a chunk: [32 x (dk + 32)] times [(dk + 32) x dv], 128 columns at a time, a thread 4 rows
// (its warp's) by 4 columns, 32 elements of the sum staged together (two stages); then the norm
// over a row's dv numbers, the weight and the gate.
#define CO_COLS 128
#define CO_STAGE (CC_ROWS * (CC_ROWS + CO_COLS))
template <typename T>
__global__ void __launch_bounds__(256) channel_delta_out_kernel(const ChannelDeltaArgs a) {
  extern __shared__ __align__(16) float sm[];    // two stages [A: 32 x 32 | B: 32 x CO_COLS] | the read-outs [32][dv]
  pdl_launch_dependents_if_small();
  const int tid = threadIdx.x, lane = tid & 31, row = tid / 32 * 4;
  const int h = blockIdx.y, seq = blockIdx.z, z = blockIdx.x;
  const int H = a.H, dk = a.dk, dv = a.dv, K = dk + CC_ROWS;
  float* os = sm + 2 * CO_STAGE;
  pdl_wait();
  const int first = a.cu_q[seq], n = min(CC_ROWS, a.cu_q[seq + 1] - first - z * CC_ROWS);
  if (n <= 0) return;
  const float* rec = a.chunks + (cc_entry(first, z, seq) * H + h) * cc_record(dk, dv);
  const float* qb = rec + cc_at_qb(dk);
  const float* su = rec + cc_at_su(dk);
  const int tiles = (K + CC_ROWS - 1) / CC_ROWS, col_tiles = (dv + CO_COLS - 1) / CO_COLS;
  auto stage_in = [&](int s) {                   // stage s: column tile s / tiles, rows (s % tiles) 32 ..
    float* as = sm + (s & 1) * CO_STAGE;
    float* bs = as + CC_ROWS * CC_ROWS;
    const int k0 = s % tiles * CC_ROWS, c0 = s / tiles * CO_COLS;
    {
      const int k = tid / 8, r = (tid % 8) * 4;
      if (k0 + k < K) cc_copy16(as + k * CC_ROWS + r, qb + (size_t)(k0 + k) * CC_ROWS + r);
    }
#pragma unroll
    for (int it = 0; it < 4; ++it) {
      const int k = tid / 32 + 8 * it, c = lane * 4;
      if (k0 + k < K && c0 + c < dv) cc_copy16(bs + k * CO_COLS + c, su + (size_t)(k0 + k) * dv + c0 + c);
    }
    cp_async_commit();
  };
  float acc[4][4];
  stage_in(0);
  const int stages = tiles * col_tiles;
  for (int s = 0; s < stages; ++s) {
    if (s + 1 < stages) { stage_in(s + 1); cp_async_wait<1>(); } else { cp_async_wait<0>(); }
    __syncthreads();
    const float* as = sm + (s & 1) * CO_STAGE;
    const float* bs = as + CC_ROWS * CC_ROWS;
    if (s % tiles == 0) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
    }
    const int nk = min(CC_ROWS, K - s % tiles * CC_ROWS);
#pragma unroll 8
    for (int k = 0; k < nk; ++k) {               // (columns beyond dv hold what no one reads)
      const float4 x = *reinterpret_cast<const float4*>(as + k * CC_ROWS + row);
      const float4 y = *reinterpret_cast<const float4*>(bs + k * CO_COLS + lane * 4);
      const float xv[4] = {x.x, x.y, x.z, x.w}, yv[4] = {y.x, y.y, y.z, y.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xv[i], yv[j], acc[i][j]);
    }
    const int c = s / tiles * CO_COLS + lane * 4;
    if (s % tiles == tiles - 1 && c < dv) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        *reinterpret_cast<float4*>(os + (row + i) * dv + c) = make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    }
    __syncthreads();
  }
  pdl_launch_dependents_if_large();
#pragma unroll
  for (int i = 0; i < 4; ++i) {                  // (a warp finishes the rows it has made)
    const int r = row + i;
    if (r >= n) break;
    const size_t t = (size_t)first + z * CC_ROWS + r;
    float ss = 0.f;
    for (int j = lane; j < dv; j += 32) ss = fmaf(os[r * dv + j], os[r * dv + j], ss);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)dv + a.norm_eps);
    const float* gate = a.wide + t * H * (dk + dv) + (size_t)H * dk + (size_t)h * dv;
    T* y = (T*)a.y + (t * H + h) * dv;
    for (int j = lane; j < dv; j += 32) y[j] = from_f32<T>(os[r * dv + j] * inv * a.norm_w[j] * cd_sigmoid(gate[j]));
  }
}

static bool cc_takes(const ChannelDeltaArgs& a) {
  return a.chunks && a.max_rows >= CC_MIN && a.dk <= CC_MAX_DK && a.dk % 4 == 0 && a.dv % 4 == 0 &&
         a.dv <= CC_MAX_DV && (((uintptr_t)a.chunks) & 15) == 0;
}

template <int E>
static int cc_local(const ChannelDeltaArgs& a, int chunks, cudaStream_t s) {
  constexpr int LD = 32 * E + 4;
  const size_t smem = ((4 * CC_ROWS + CC_HALF) * LD + 2 * CC_ROWS * CC_ROWS + CC_ROWS) * sizeof(float);
  static bool configured = false;
  if (smem > 48 * 1024 && !configured) {
    cudaError_t e = cudaFuncSetAttribute(channel_delta_local_kernel<E>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                         (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  return gb_launch(channel_delta_local_kernel<E>, dim3(chunks, a.H, a.n_seqs), dim3(256), smem, s, a);
}

template <typename T>
static int cc_run(const ChannelDeltaArgs& a, cudaStream_t s) {
  const int chunks = (a.max_rows + CC_ROWS - 1) / CC_ROWS;
  int e = a.dk <= 32 ? cc_local<1>(a, chunks, s) : a.dk <= 64 ? cc_local<2>(a, chunks, s) : cc_local<4>(a, chunks, s);
  if (e) return e;
  size_t smem = (2 * cc_stage(a.dk) + a.dk * CC_COLS + 5 * CC_ROWS * CC_COLS) * sizeof(float);
  // a grid that has an SM for every block: one block an SM, wherever it finds room first (two would
  // halve each other's pace while other SMs stand idle)
  if ((long long)((a.dv + CC_COLS - 1) / CC_COLS) * a.H * a.n_seqs <= 148 && smem < 120 * 1024) smem = 120 * 1024;
  static size_t chain_smem = 48 * 1024, out_smem = 48 * 1024;    // (out_smem: per activation type)
  if (smem > chain_smem) {
    cudaError_t ce = cudaFuncSetAttribute(channel_delta_chain_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                          (int)smem);
    if (ce != cudaSuccess) return (int)ce;
    chain_smem = smem;
  }
  e = gb_launch(channel_delta_chain_kernel, dim3((a.dv + CC_COLS - 1) / CC_COLS, a.H, a.n_seqs), dim3(256), smem, s, a);
  if (e) return e;
  smem = (2 * CO_STAGE + CC_ROWS * a.dv) * sizeof(float);
  if (smem > out_smem) {
    cudaError_t ce = cudaFuncSetAttribute(channel_delta_out_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                          (int)smem);
    if (ce != cudaSuccess) return (int)ce;
    out_smem = smem;
  }
  return gb_launch(channel_delta_out_kernel<T>, dim3(chunks, a.H, a.n_seqs), dim3(256), smem, s, a);
}
