// A feed-forward made of many small experts, of which every token uses a few.
//
//   z = x Wr^T (32-bit);  s = softmax(z) over all router outputs
//   choice score c = s + correction;  the outputs form n_groups equal groups of
//   neighbours, a group's score is its largest c, and only outputs of the
//   keep_groups best groups can be chosen (the others count as -inf);  the `top`
//   outputs with the largest c are chosen and weigh in with their s, as it is
//   expert e < E:   g = min(x Wg_e^T, limit), u = clamp(x Wu_e^T, -limit, limit),
//                   y = (g sigmoid(slope g) (u + 1)) Wd_e^T
//   output >= E:    an expert that hands its input on, y = x
//   out = sum over the chosen of s * y
//
// Each of these terms is an argument.  `score_fn` 1 takes s = sigmoid(z), every output
// by itself, instead of the softmax; `score_fn` 2 lets the logits z choose and takes the
// softmax over the chosen logits alone as the weights; `router_bias` is added to z; `correction` may be null (no correction); a limit
// of +inf clamps nothing; `up_offset` is the 1 in (u + 1) and may be 0; with
// `weigh_input` the weight multiplies the expert's input instead of its result,
// y = expert(s x): gate and up have no bias, so their 32-bit sums are multiplied by s
// before the activation, and the second product is stored as it is.
//
// Further forms: `group_top2` scores a group by the sum of its two largest c (of its only
// one where a group has a single output); `normalize` makes a token's weights s / (sum of
// the chosen s + 1e-20) * weight_scale (without it they are s * weight_scale); with no
// gate weights an expert is ungated, y = max(x Wu_e^T, 0)^2 Wd_e^T (no limit, slope or
// offset).
//
// A shared expert (ungated, weights ws_up [Fs, W] and ws_down [W, Fs]) runs for every token with
// weight 1 in the same two launches: its tiles come first in the tensor-core kernels' grid,
// its rows are the tokens as they lie in x, its result is out[top, token, :].
//
// Nothing here needs the host to know how many tokens an expert got, so a step
// can be captured: `route` chooses and counts, and its last block turns the counts into a
// list of (token, choice) pairs ordered by expert; the two products walk
// tiles of that list; a block finds its expert from the counts, and blocks
// beyond the last tile return.  A pair's row is computed the same way wherever it
// lands in the list, so a token's result does not depend on the batch.  A step of few rows
// (`small`, a decode step) needs no list: a block of the products belongs to an expert and
// finds the expert's pairs among the step's few choices itself, pair p's inner activations
// lie in row p, and since its weights are known from the start it asks for the first of them
// before it waits for the choices.  The
// weighted results are left as `top` 32-bit partial sums [top, T, W]
// (choice j of token t in out[j, t, :]), which the norm that follows adds in
// order.
#include "attn_mma.cuh"

struct MoeArgs {
  const void* x;            // [T, W] activations
  const float* router_w;    // [E + n_identity, W]
  const float* correction;  // [E + n_identity]
  const void* w_gate;       // [E, F, W], or null: the experts have no gate
  const void* w_up;         // [E, F, W]
  const void* w_down;       // [E, W, F]
  int* ids;                 // [T, top] chosen outputs
  float* wts;               // [T, top] their scores
  int* rank;                // [T, top] place of the pair among its expert's pairs
  int* counts;              // [E + 1] pairs per expert, and the tickets of `route`'s blocks; zero on entry
  int* offsets;             // [E + 1]
  int* perm;                // [T top] pairs (t * top + j) ordered by expert
  void* act;                // [T top, F] activations of the experts' inner layer, in list order
  float* out;               // [top, T, W] (rows beyond it, if any, are the caller's)
  int T, W, F, E, n_identity, top, n_groups, keep_groups;
  float limit, slope;
  int score_fn;              // 0: softmax over the outputs, 1: sigmoid of each, 2: softmax over the chosen
  int weigh_input;           // the weight multiplies the expert's input, not its result
  float up_offset;           // y = act(g) (u + up_offset)
  const float* router_bias;  // [E + n_identity] added to z, or null
  int group_top2;            // a group's score is the sum of its two largest c, not its largest
  int normalize;             // the chosen outputs' weights are divided by their sum
  float weight_scale;        // and multiplied by this
  const void* ws_up;         // [Fs, W] the shared expert, or null
  const void* ws_down;       // [W, Fs]
  void* act_s;               // [T, Fs] its inner activations
  int Fs;
  int small;                 // a step of few rows: no ordered list, blocks of the products by expert
  int early;                 // with `small`: a block's first weights are requested before the choices are known
  int stage_router;          // the router's rows fit in a block's shared memory and are fetched before the wait
  int route_only;            // stop behind `route` (the products are another source's kernels)
};

#define MOE_MAX_OUTPUTS 1024

#define MOE_ROUTE_THREADS 256
#define MOE_ROUTE_CHUNK 8     // router outputs whose sums a thread carries side by side

// What one warp does with a token's logits z [n_all]: turns them into scores, chooses, and writes
// the choices and their weights.  c [n_all] and gval [n_groups] are shared-memory scratch.
__device__ __forceinline__ void moe_choose(const MoeArgs& a, float* z, float* c, float* gval, int t, int lane) {
  const int n_all = a.E + a.n_identity;
  if (a.score_fn == 1) {
    for (int e = lane; e < n_all; e += 32) z[e] = 1.0f / (1.0f + expf(-z[e]));
  } else if (a.score_fn == 0) {
    float mx = -INFINITY, sum = 0.f;
    for (int e = lane; e < n_all; e += 32) mx = fmaxf(mx, z[e]);
    mx = warp_max(mx);
    for (int e = lane; e < n_all; e += 32) { z[e] = expf(z[e] - mx); sum += z[e]; }
    sum = warp_sum(sum);
    for (int e = lane; e < n_all; e += 32) z[e] = z[e] / sum;
  }   // score_fn 2: the logits themselves choose; the chosen ones' weights are worked out below
  for (int e = lane; e < n_all; e += 32) c[e] = z[e] + (a.correction ? a.correction[e] : 0.f);
  __syncwarp();
  if (a.n_groups > 1 && a.keep_groups < a.n_groups) {
    const int per = n_all / a.n_groups;
    for (int g = lane; g < a.n_groups; g += 32) {
      float b1 = -INFINITY, b2 = -INFINITY;           // the group's two largest
      for (int e = g * per; e < (g + 1) * per; ++e) {
        const float v = c[e];
        b2 = fmaxf(b2, fminf(b1, v));
        b1 = fmaxf(b1, v);
      }
      gval[g] = a.group_top2 && per > 1 ? b1 + b2 : b1;
    }
    __syncwarp();
    // a group that `keep_groups` others come before (larger, or equal and earlier) is dropped
    for (int g = lane; g < a.n_groups; g += 32) {
      const float v = gval[g];
      int before = 0;
      for (int o = 0; o < a.n_groups; ++o) before += gval[o] > v || (gval[o] == v && o < g);
      if (before >= a.keep_groups)
        for (int e = g * per; e < (g + 1) * per; ++e) c[e] = -INFINITY;
    }
    __syncwarp();
  }
  float chosen_sum = 0.f, first_z = 0.f;
  for (int j = 0; j < a.top; ++j) {   // the largest first; of equal ones the earlier
    float bv = -INFINITY;
    int bi = 0x7fffffff;
    for (int e = lane; e < n_all; e += 32) {         // (one that is taken is NaN: no comparison holds)
      const float v = c[e];
      if (v > bv || (v == bv && e < bi)) { bv = v; bi = e; }
    }
  #pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
    }
    const int best = bi < n_all ? bi : 0;
    const float w = z[best];
    if (j == 0) first_z = w;
    chosen_sum += a.score_fn == 2 ? expf(w - first_z) : w;   // (the first logit is the largest)
    __syncwarp();
    if (lane == 0) {
      c[best] = NAN;                  // taken
      a.ids[(size_t)t * a.top + j] = best;
      a.wts[(size_t)t * a.top + j] = w;
    }
    __syncwarp();
  }
  if (lane == 0) {
    float* w = a.wts + (size_t)t * a.top;
    for (int j = 0; j < a.top; ++j) {
      // softmax over the chosen logits alone, or the scores, as they are or as shares of their sum
      const float v = a.score_fn == 2 ? expf(w[j] - first_z) / chosen_sum
                      : a.normalize   ? w[j] / (chosen_sum + 1e-20f) : w[j];
      w[j] = v * a.weight_scale;
    }
  }
}

// What the block that finishes last does: the counts become the list of pairs ordered by
// expert.  cnt and off [E] are shared-memory scratch; the counts and the blocks' tickets are
// left at zero for the next call.
__device__ __forceinline__ void moe_order_pairs(const MoeArgs& a, int* cnt, int* off) {
  const int tid = threadIdx.x, lane = tid & 31, nt = blockDim.x;
  for (int e = tid; e < a.E; e += nt) cnt[e] = __ldcg(&a.counts[e]);   // (all requested at once)
  __syncthreads();
  if (tid < 32) {                                      // exclusive sums, 32 experts a turn
    int run = 0;
    for (int e0 = 0; e0 < a.E; e0 += 32) {
      const int c0 = e0 + lane < a.E ? cnt[e0 + lane] : 0;
      int v = c0;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int u = __shfl_up_sync(0xffffffffu, v, o);
        if (lane >= o) v += u;
      }
      if (e0 + lane < a.E) {
        off[e0 + lane] = run + v - c0;
        a.offsets[e0 + lane] = run + v - c0;
      }
      run += __shfl_sync(0xffffffffu, v, 31);
    }
    if (lane == 0) a.offsets[a.E] = run;
  }
  __syncthreads();
  const int n_pairs = a.T * a.top;
  for (int p0 = tid; p0 < n_pairs; p0 += 8 * nt) {     // eight pairs' loads are requested together
    int e[8], r[8];
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      const int p = p0 + u * nt < n_pairs ? p0 + u * nt : p0;
      e[u] = __ldcg(&a.ids[p]), r[u] = __ldcg(&a.rank[p]);
    }
#pragma unroll
    for (int u = 0; u < 8; ++u)
      if (p0 + u * nt < n_pairs && e[u] < a.E) a.perm[off[e[u]] + r[u]] = p0 + u * nt;
  }
  for (int e = tid; e <= a.E; e += nt) a.counts[e] = 0;
}

// True in every thread of the block that draws the last ticket of the grid (counts[E]): every
// block publishes its choices before it draws, so the last one sees all of them.
__device__ __forceinline__ bool moe_last_block(const MoeArgs& a) {
  __shared__ int is_last;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) is_last = atomicAdd(&a.counts[a.E], 1) == (int)gridDim.x - 1;
  __syncthreads();
  if (is_last) __threadfence();
  return is_last != 0;
}

template <typename T>
__global__ void __launch_bounds__(MOE_ROUTE_THREADS) moe_route_kernel(const MoeArgs a) {
  extern __shared__ float sm[];   // z [n_all], c [n_all], a score per group
  __shared__ float part[MOE_ROUTE_THREADS / 32][MOE_ROUTE_CHUNK];
  pdl_launch_dependents_if_small();
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int nwarps = blockDim.x >> 5;
  const int n_all = a.E + a.n_identity, W = a.W;
  float* z = sm;
  float* c = sm + n_all;
  float* gval = c + n_all;         // [n_groups] scores of the groups
  const float* router = a.router_w;
  if (a.stage_router) {            // (no kernel's output: before the wait)
    float* rs = sm + ((2 * n_all + a.n_groups + 3) & ~3);
    for (int i = tid * 4; i < n_all * W; i += MOE_ROUTE_THREADS * 4) cp_async16(rs + i, a.router_w + i, true);
    cp_async_commit();
    router = rs;
  }
  pdl_wait();
  const T* x = (const T*)a.x + (size_t)t * W;
  if (a.stage_router) {
    cp_async_wait<0>();
    __syncthreads();
  }
  // every thread takes a slice of the row against a few router rows at a time, so that
  // all of a slice's loads are under way together; the sums are put together in a fixed
  // order (lanes by the shuffle tree, then warp after warp)
  for (int e0 = 0; e0 < n_all; e0 += MOE_ROUTE_CHUNK) {
    float acc[MOE_ROUTE_CHUNK];
#pragma unroll
    for (int u = 0; u < MOE_ROUTE_CHUNK; ++u) acc[u] = 0.f;
    const int nu = min(MOE_ROUTE_CHUNK, n_all - e0);
#pragma unroll 4
    for (int i = tid; i < W; i += MOE_ROUTE_THREADS) {
      const float xv = to_f32<T>(x[i]);
#pragma unroll
      for (int u = 0; u < MOE_ROUTE_CHUNK; ++u)
        if (u < nu) acc[u] = fmaf(xv, router[(size_t)(e0 + u) * W + i], acc[u]);
    }
#pragma unroll
    for (int u = 0; u < MOE_ROUTE_CHUNK; ++u) {
      const float v = warp_sum(acc[u]);
      if (lane == 0) part[warp][u] = v;
    }
    __syncthreads();
    if (tid < MOE_ROUTE_CHUNK && e0 + tid < n_all) {
      float v = 0.f;
      for (int w = 0; w < nwarps; ++w) v += part[w][tid];
      z[e0 + tid] = v + (a.router_bias ? a.router_bias[e0 + tid] : 0.f);
    }
    __syncthreads();
  }
  if (warp == 0) {        // one warp turns logits into scores and chooses
    moe_choose(a, z, c, gval, t, lane);
  }
  if (a.small && a.n_identity == 0) return;          // the products' blocks read the choices themselves
  __syncthreads();
  if (!a.small)
    for (int j = tid; j < a.top; j += blockDim.x) {   // the choices' places among their experts' pairs
      const int e = a.ids[(size_t)t * a.top + j];
      a.rank[(size_t)t * a.top + j] = e < a.E ? atomicAdd(&a.counts[e], 1) : -1;
    }
  pdl_launch_dependents_if_large();
  for (int j = 0; j < a.top; ++j) {     // experts that hand their input on
    if (a.ids[(size_t)t * a.top + j] < a.E) continue;
    const float w = a.wts[(size_t)t * a.top + j];
    float* o = a.out + ((size_t)j * a.T + t) * W;
    for (int i = tid; i < W; i += blockDim.x) o[i] = w * to_f32<T>(x[i]);
  }
  if (a.small) return;
  if (!moe_last_block(a)) return;
  int* cnt = reinterpret_cast<int*>(sm);               // (the choices' shared memory is free)
  moe_order_pairs(a, cnt, cnt + a.E);
}

// The same for many rows: the block brings eight router rows at a time into shared memory, a
// warp makes the logits of TPW tokens side by side (four neighbouring elements a lane) and
// chooses for one after the other; the block counts its choices per expert in shared memory and adds them to the
// experts' counts in one go.
#define MOE_ROWS_WARPS 8
template <typename T> __device__ __forceinline__ void moe_load4(const T* p, float (&v)[4]);
template <> __device__ __forceinline__ void moe_load4<float>(const float* p, float (&v)[4]) {
  const float4 x = *reinterpret_cast<const float4*>(p);
  v[0] = x.x, v[1] = x.y, v[2] = x.z, v[3] = x.w;
}
template <> __device__ __forceinline__ void moe_load4<bf16>(const bf16* p, float (&v)[4]) {
  const uint2 x = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162 a = *reinterpret_cast<const __nv_bfloat162*>(&x.x), b = *reinterpret_cast<const __nv_bfloat162*>(&x.y);
  v[0] = __low2float(a), v[1] = __high2float(a), v[2] = __low2float(b), v[3] = __high2float(b);
}

template <typename T, int TPW>
__global__ void __launch_bounds__(MOE_ROWS_WARPS * 32) moe_route_rows_kernel(const MoeArgs a) {
  extern __shared__ float sm[];
  pdl_launch_dependents_if_small();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n_all = a.E + a.n_identity, W = a.W, top = a.top;
  const int per_tok = 2 * n_all + a.n_groups;
  float* mine = sm + (size_t)warp * TPW * per_tok;
  int* cnt = reinterpret_cast<int*>(sm + (size_t)MOE_ROWS_WARPS * TPW * per_tok);   // [E]
  int* base = cnt + a.E;                                                            // [E]
  float* rs = sm + (((size_t)MOE_ROWS_WARPS * TPW * per_tok + 2 * a.E + 3) & ~(size_t)3);   // [MOE_ROUTE_CHUNK, W]
  auto stage = [&](int e0) {       // (no kernel's output)
    const int n = min(MOE_ROUTE_CHUNK, n_all - e0) * W;
    for (int i = tid * 4; i < n; i += MOE_ROWS_WARPS * 32 * 4) cp_async16(rs + i, a.router_w + (size_t)e0 * W + i, true);
    cp_async_commit();
  };
  stage(0);
  for (int e = tid; e < a.E; e += blockDim.x) cnt[e] = 0;
  pdl_wait();
  const int t0 = (blockIdx.x * MOE_ROWS_WARPS + warp) * TPW;
  const T* x = (const T*)a.x;
  for (int e0 = 0; e0 < n_all; e0 += MOE_ROUTE_CHUNK) {
    float acc[TPW][MOE_ROUTE_CHUNK];
#pragma unroll
    for (int k = 0; k < TPW; ++k)
#pragma unroll
      for (int u = 0; u < MOE_ROUTE_CHUNK; ++u) acc[k][u] = 0.f;
    if (e0) {
      __syncthreads();             // everyone is done with the rows before these
      stage(e0);
    }
    cp_async_wait<0>();
    __syncthreads();
    const int last = min(MOE_ROUTE_CHUNK, n_all - e0) - 1;
#pragma unroll 4
    for (int i = lane * 4; i < W; i += 128) {
      float xv[TPW][4];
#pragma unroll
      for (int k = 0; k < TPW; ++k) moe_load4<T>(x + (size_t)min(t0 + k, a.T - 1) * W + i, xv[k]);
#pragma unroll
      for (int u = 0; u < MOE_ROUTE_CHUNK; ++u) {
        const float4 w = *reinterpret_cast<const float4*>(rs + (size_t)min(u, last) * W + i);
#pragma unroll
        for (int k = 0; k < TPW; ++k)
          acc[k][u] = fmaf(xv[k][3], w.w, fmaf(xv[k][2], w.z, fmaf(xv[k][1], w.y, fmaf(xv[k][0], w.x, acc[k][u]))));
      }
    }
#pragma unroll
    for (int k = 0; k < TPW; ++k)
#pragma unroll
      for (int u = 0; u < MOE_ROUTE_CHUNK; ++u) {
        const float v = warp_sum(acc[k][u]);
        if (lane == 0 && e0 + u < n_all)
          mine[k * per_tok + e0 + u] = v + (a.router_bias ? a.router_bias[e0 + u] : 0.f);
      }
  }
  __syncthreads();
  for (int k = 0; k < TPW; ++k) {
    const int t = t0 + k;
    if (t >= a.T) break;
    float* z = mine + k * per_tok;
    moe_choose(a, z, z + n_all, z + 2 * n_all, t, lane);
    __syncwarp();
    for (int j = lane; j < top; j += 32) {             // the pair's place among the block's for its expert
      const int e = a.ids[(size_t)t * top + j];
      a.rank[(size_t)t * top + j] = e < a.E ? atomicAdd(&cnt[e], 1) : -1;
    }
  }
  __syncthreads();
  for (int e = tid; e < a.E; e += blockDim.x) base[e] = cnt[e] ? atomicAdd(&a.counts[e], cnt[e]) : 0;
  __syncthreads();
  for (int k = 0; k < TPW; ++k) {
    const int t = t0 + k;
    if (t >= a.T) break;
    for (int j = lane; j < top; j += 32) {
      const int e = a.ids[(size_t)t * top + j];
      if (e < a.E) a.rank[(size_t)t * top + j] += base[e];
    }
    for (int j = 0; j < top; ++j) {                    // experts that hand their input on
      if (a.ids[(size_t)t * top + j] < a.E) continue;
      const float w = a.wts[(size_t)t * top + j];
      float* o = a.out + ((size_t)j * a.T + t) * W;
      for (int i = lane; i < W; i += 32) o[i] = w * to_f32<T>(x[(size_t)t * W + i]);
    }
  }
  pdl_launch_dependents_if_large();
  if (!moe_last_block(a)) return;
  moe_order_pairs(a, cnt, base);
}

#define MOE_BM 16
#define MOE_BN 64
#define MOE_BK 32

// Which expert and which of its tiles of BM pairs block `b` has; false beyond the last.
template <int BM = MOE_BM>
__device__ __forceinline__ bool moe_find_tile(const int* offsets, int E, int b, int& e_out,
                                              int& first, int& n_rows) {
  int tiles = 0;
  for (int e = 0; e < E; ++e) {
    const int cnt = offsets[e + 1] - offsets[e];
    const int nt = (cnt + BM - 1) / BM;
    if (b < tiles + nt) {
      e_out = e;
      first = offsets[e] + (b - tiles) * BM;
      n_rows = min(BM, offsets[e + 1] - first);
      return true;
    }
    tiles += nt;
  }
  return false;
}

// act[p, f] = fn(x[token(p)] . Wg_e[f], x[token(p)] . Wu_e[f]) for the pairs p of a tile
template <typename T>
__global__ void __launch_bounds__(256) moe_up_kernel(const MoeArgs a) {
  __shared__ float As[MOE_BM][MOE_BK];
  __shared__ float Gs[MOE_BN][MOE_BK + 1];
  __shared__ float Us[MOE_BN][MOE_BK + 1];
  __shared__ int tok[MOE_BM];
  pdl_launch_dependents_if_small();
  pdl_wait();
  int e, first, n_rows;
  if (!moe_find_tile(a.offsets, a.E, blockIdx.x, e, first, n_rows)) return;
  const int tid = threadIdx.x, W = a.W, F = a.F;
  const int f0 = blockIdx.y * MOE_BN;
  if (tid < MOE_BM) tok[tid] = tid < n_rows ? a.perm[first + tid] / a.top : -1;
  __syncthreads();
  const bool gated = a.w_gate != nullptr;
  const T* wg = gated ? (const T*)a.w_gate + (size_t)e * F * W : nullptr;
  const T* wu = (const T*)a.w_up + (size_t)e * F * W;
  const int tx = tid & 63, ty = tid >> 6;      // column, group of four rows
  float accg[4] = {0.f, 0.f, 0.f, 0.f}, accu[4] = {0.f, 0.f, 0.f, 0.f};
  for (int k0 = 0; k0 < W; k0 += MOE_BK) {
    for (int i = tid; i < MOE_BM * MOE_BK; i += 256) {
      const int r = i / MOE_BK, k = i % MOE_BK;
      As[r][k] = (tok[r] >= 0 && k0 + k < W) ? to_f32<T>(((const T*)a.x)[(size_t)tok[r] * W + k0 + k]) : 0.f;
    }
    for (int i = tid; i < MOE_BN * MOE_BK; i += 256) {
      const int n = i / MOE_BK, k = i % MOE_BK;
      const bool ok = f0 + n < F && k0 + k < W;
      if (gated) Gs[n][k] = ok ? to_f32<T>(wg[(size_t)(f0 + n) * W + k0 + k]) : 0.f;
      Us[n][k] = ok ? to_f32<T>(wu[(size_t)(f0 + n) * W + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < MOE_BK; ++k) {
      const float g = gated ? Gs[tx][k] : 0.f, u = Us[tx][k];
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const float x = As[ty * 4 + r][k];
        accg[r] = fmaf(x, g, accg[r]);
        accu[r] = fmaf(x, u, accu[r]);
      }
    }
    __syncthreads();
  }
  pdl_launch_dependents_if_large();
  if (f0 + tx >= F) return;
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const int row = ty * 4 + r;
    if (row >= n_rows) continue;
    float g = accg[r], u = accu[r];
    if (a.weigh_input) { const float w = a.wts[a.perm[first + row]]; g *= w; u *= w; }
    float y;
    if (gated) {
      g = fminf(g, a.limit);
      u = fminf(fmaxf(u, -a.limit), a.limit);
      y = g / (1.0f + expf(-a.slope * g)) * (u + a.up_offset);
    } else {
      u = fmaxf(u, 0.f);
      y = u * u;
    }
    ((T*)a.act)[(size_t)(first + row) * F + f0 + tx] = from_f32<T>(y);
  }
}

// out[j, t, :] = s * (act[p] . Wd_e^T) for the pairs p = t * top + j of a tile
template <typename T>
__global__ void __launch_bounds__(256) moe_down_kernel(const MoeArgs a) {
  __shared__ float As[MOE_BM][MOE_BK];
  __shared__ float Bs[MOE_BN][MOE_BK + 1];
  __shared__ int pair[MOE_BM];
  pdl_launch_dependents_if_small();
  pdl_wait();
  int e, first, n_rows;
  if (!moe_find_tile(a.offsets, a.E, blockIdx.x, e, first, n_rows)) return;
  const int tid = threadIdx.x, W = a.W, F = a.F;
  const int n0 = blockIdx.y * MOE_BN;
  if (tid < MOE_BM) pair[tid] = tid < n_rows ? a.perm[first + tid] : -1;
  __syncthreads();
  const T* wd = (const T*)a.w_down + (size_t)e * W * F;
  const int tx = tid & 63, ty = tid >> 6;
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  for (int k0 = 0; k0 < F; k0 += MOE_BK) {
    for (int i = tid; i < MOE_BM * MOE_BK; i += 256) {
      const int r = i / MOE_BK, k = i % MOE_BK;
      As[r][k] = (r < n_rows && k0 + k < F) ? to_f32<T>(((const T*)a.act)[(size_t)(first + r) * F + k0 + k]) : 0.f;
    }
    for (int i = tid; i < MOE_BN * MOE_BK; i += 256) {
      const int n = i / MOE_BK, k = i % MOE_BK;
      Bs[n][k] = (n0 + n < W && k0 + k < F) ? to_f32<T>(wd[(size_t)(n0 + n) * F + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < MOE_BK; ++k) {
      const float b = Bs[tx][k];
#pragma unroll
      for (int r = 0; r < 4; ++r) acc[r] = fmaf(As[ty * 4 + r][k], b, acc[r]);
    }
    __syncthreads();
  }
  pdl_launch_dependents_if_large();
  if (n0 + tx >= W) return;
#pragma unroll
  for (int r = 0; r < 4; ++r) {
    const int row = ty * 4 + r;
    if (row >= n_rows) continue;
    const int p = pair[row], t = p / a.top, j = p % a.top;
    a.out[((size_t)j * a.T + t) * W + n0 + tx] = (a.weigh_input ? 1.0f : a.wts[p]) * acc[r];
  }
}


// ---- the two products on the tensor cores (bfloat16, widths that are multiples of 8) ----
// A block of four warps takes a tile of BM pairs and 64 output columns (mma.sync m16n8k16,
// 32-bit sums).  With BM = 128 or 64 (many tokens) the warps are two by two, each with half
// the rows and 32 columns;
// with BM = 16 (a decode step: a handful of pairs per expert, the weights' bytes are the
// cost) the tile is 32 columns wide, so that more blocks stream weights at once, and the
// warps share the 16 rows and take 8 columns each.  Rows of the activations
// (gathered by token for the first product, in list order for the second) and rows of the
// expert's weight reach shared memory by 16-byte asynchronous copies, STAGES chunks of 64
// columns of the inner size in flight; rows and columns beyond the tile's end are filled
// with zeros.  The first product runs gate and up side by side and applies the expert's
// activation to its 32-bit sums; the second multiplies by the pair's weight and stores 32-bit.
#define MT_BN 64
#define MT_BK 64
#define MT_LD (MT_BK + 8)

__device__ __forceinline__ void ldmatrix_x2(uint32_t (&r)[2], const void* smem) {
  const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(s));
}

// The three products: an expert's second, its first with gate and up side by side, its first
// without a gate.
enum MoeMode { MOE_DOWN = 0, MOE_GATED = 1, MOE_UNGATED = 2 };

template <int MODE, int BM>
struct MoeTile {
  static constexpr bool UP = MODE != MOE_DOWN;
  static constexpr int NB = MODE == MOE_GATED ? 2 : 1;
  static constexpr int BN = BM >= 64 ? MT_BN : 32;
  static constexpr int THREADS = 128;
  // a warp's share of the tile: MI pieces of 16 rows by NJ pieces of 8 columns.  Many rows:
  // the four warps are two by two, each with half the rows and 32 columns, so that a
  // fragment read from shared memory feeds several MMAs.  16 rows: the warps share them
  // and take 8 columns each.
  static constexpr int MI = BM >= 64 ? BM / 32 : 1;
  static constexpr int NJ = BM >= 64 ? 4 : 1;
  static constexpr int STAGES = BM >= 64 ? 3 : 4;
  static constexpr int STAGE_ELEMS = (BM + NB * BN) * MT_LD;
  static constexpr size_t SMEM = (size_t)STAGES * STAGE_ELEMS * sizeof(bf16);
};

template <int MODE, int BM, bool SMALL>
__global__ void __launch_bounds__(128) moe_tc_kernel(const MoeArgs a) {
  using Tile = MoeTile<MODE, BM>;
  constexpr bool UP = Tile::UP, GATED = MODE == MOE_GATED;
  constexpr int NB = Tile::NB, STAGES = Tile::STAGES, BN = Tile::BN, NT = Tile::THREADS;
  constexpr int MI = Tile::MI, NJ = Tile::NJ;
  extern __shared__ __align__(16) bf16 tiles[];
  __shared__ int src_row[BM];
  __shared__ int pair_of[BM];                  // the tile's pairs
  pdl_launch_dependents_if_small();
  if (!SMALL) pdl_wait();
  int e = 0, first = 0, n_rows = 0;
  const int shared_tiles = a.Fs > 0 ? (a.T + BM - 1) / BM : 0;
  const bool shared = (int)blockIdx.x < shared_tiles;      // a tile of the shared expert: tokens as they come
  const int F = shared ? a.Fs : a.F;
  const int K = UP ? a.W : F, N = UP ? F : a.W;
  const int n0 = blockIdx.y * BN;
  if (n0 >= N) return;
  if (shared) {
    first = blockIdx.x * BM;
    n_rows = min(BM, a.T - first);
  } else if (SMALL) {
    const int per_expert = (a.T + BM - 1) / BM;            // an expert has at most one pair a token
    e = (blockIdx.x - shared_tiles) / per_expert;
    first = ((blockIdx.x - shared_tiles) % per_expert) * BM;   // its pairs from this one on
  } else if (!moe_find_tile<BM>(a.offsets, a.E, blockIdx.x - shared_tiles, e, first, n_rows)) {
    return;
  }
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  auto list_rows = [&] {       // which rows of A the tile has: from the list, from the choices, or as tokens come
    if (SMALL && !shared) {
      __shared__ int found_s[NT / 32];
      int seen = 0;
      for (int p0 = 0; p0 < a.T * a.top; p0 += NT) {
        const int p = p0 + tid;
        const bool mine = p < a.T * a.top && __ldcg(&a.ids[p]) == e;
        const unsigned votes = __ballot_sync(0xffffffffu, mine);
        if (lane == 0) found_s[warp] = __popc(votes);
        __syncthreads();
        int at = seen;
        for (int w = 0; w < NT / 32; ++w) {
          if (w < warp) at += found_s[w];
          seen += found_s[w];
        }
        at += __popc(votes & ((1u << lane) - 1)) - first;
        if (mine && at >= 0 && at < BM) pair_of[at] = p;
        __syncthreads();
      }
      n_rows = min(BM, seen - first);
    } else {
      for (int i = tid; i < n_rows; i += NT) pair_of[i] = shared ? 0 : a.perm[first + i];
      __syncthreads();
    }
    for (int i = tid; i < BM; i += NT) {
      int r = -1;
      if (i < n_rows) r = shared ? first + i : UP ? pair_of[i] / a.top : SMALL ? pair_of[i] : first + i;
      src_row[i] = r;
    }
    __syncthreads();
  };
  const bf16* A = (const bf16*)(UP ? a.x : shared ? a.act_s : a.act);
  const bf16* B0 = shared ? (const bf16*)(UP ? a.ws_up : a.ws_down)
                          : (const bf16*)(GATED ? a.w_gate : UP ? a.w_up : a.w_down) + (size_t)e * N * K;
  const bf16* B1 = GATED ? (const bf16*)a.w_up + (size_t)e * N * K : nullptr;
  auto load_a = [&](int stage, int k0) {
    bf16* As = tiles + stage * Tile::STAGE_ELEMS;
    for (int c = tid; c < BM * 8; c += NT) {             // rows x 8 pieces of 8 elements
      const int r = c >> 3, pc = (c & 7) * 8, kc = k0 + pc;
      const bool ok = src_row[r] >= 0 && kc < K;
      cp_async16(As + r * MT_LD + pc, ok ? A + (size_t)src_row[r] * K + kc : A, ok);
    }
  };
  auto load_b = [&](int stage, int k0) {
    bf16* Bs = tiles + stage * Tile::STAGE_ELEMS + BM * MT_LD;
#pragma unroll
    for (int i = 0; i < BN * 8 / NT; ++i) {
      const int c = tid + i * NT, r = c >> 3, pc = (c & 7) * 8, kc = k0 + pc;
      const bool ok = n0 + r < N && kc < K;
      cp_async16(Bs + r * MT_LD + pc, ok ? B0 + (size_t)(n0 + r) * K + kc : B0, ok);
      if (GATED) cp_async16(Bs + (BN + r) * MT_LD + pc, ok ? B1 + (size_t)(n0 + r) * K + kc : B1, ok);
    }
  };
  float acc[NB][MI][NJ][4];
#pragma unroll
  for (int b = 0; b < NB; ++b)
#pragma unroll
    for (int m = 0; m < MI; ++m)
#pragma unroll
      for (int j = 0; j < NJ; ++j)
#pragma unroll
        for (int x = 0; x < 4; ++x) acc[b][m][j][x] = 0.f;
  const int row_w = BM >= 64 ? (warp >> 1) * (BM / 2) : 0;
  const int col_w = BM >= 64 ? (warp & 1) * 32 : warp * 8;
  const int arow = row_w + (lane & 7) + ((lane >> 3) & 1) * 8, acol = (lane >> 4) * 8;
  // two 8-column pieces at a time (four 8 x 8 blocks), or one (two blocks: lanes 0-15 give the rows)
  const int brow = col_w + (lane & 7) + (NJ > 1 ? (lane >> 4) * 8 : 0), bcol = ((lane >> 3) & 1) * 8;
  const int nk = (K + MT_BK - 1) / MT_BK;
  const bool early = SMALL && (a.early || shared);
  if (early) {                                   // weights, which no kernel writes: before the wait
#pragma unroll
    for (int st = 0; st < STAGES - 1; ++st)
      if (st < nk) load_b(st, st * MT_BK);
    cp_async_commit();
  }
  if (SMALL) pdl_wait();
  list_rows();
  if (SMALL && n_rows <= 0) {                    // an expert nobody chose (the copies under way land first)
    cp_async_wait<0>();
    return;
  }
#pragma unroll
  for (int st = 0; st < STAGES - 1; ++st) {      // a group per stage, empty beyond the end
    if (st < nk) {
      load_a(st, st * MT_BK);
      if (!early) load_b(st, st * MT_BK);
    }
    cp_async_commit();
  }
  for (int kt = 0; kt < nk; ++kt) {
    cp_async_wait<STAGES - 2>();                  // chunk kt has landed
    __syncthreads();                              // ... for every thread; chunk kt - 1 is done with
    if (kt + STAGES - 1 < nk) {
      load_a((kt + STAGES - 1) % STAGES, (kt + STAGES - 1) * MT_BK);
      load_b((kt + STAGES - 1) % STAGES, (kt + STAGES - 1) * MT_BK);
    }
    cp_async_commit();
    const bf16* As = tiles + (kt % STAGES) * Tile::STAGE_ELEMS;
    const bf16* Bs = As + BM * MT_LD;
#pragma unroll
    for (int k = 0; k < MT_BK / 16; ++k) {
      uint32_t af[MI][4];
#pragma unroll
      for (int m = 0; m < MI; ++m) ldmatrix_x4(af[m], As + (arow + m * 16) * MT_LD + k * 16 + acol);
#pragma unroll
      for (int b = 0; b < NB; ++b) {
        if (NJ == 1) {
          uint32_t bf[2];
          ldmatrix_x2(bf, Bs + (b * BN + brow) * MT_LD + k * 16 + bcol);
#pragma unroll
          for (int m = 0; m < MI; ++m) mma_16816(acc[b][m][0], af[m], bf[0], bf[1]);
        } else {
#pragma unroll
          for (int j = 0; j + 1 < NJ; j += 2) {
            uint32_t bf[4];
            ldmatrix_x4(bf, Bs + (b * BN + j * 8 + brow) * MT_LD + k * 16 + bcol);
#pragma unroll
            for (int m = 0; m < MI; ++m) {
              mma_16816(acc[b][m][j], af[m], bf[0], bf[1]);
              mma_16816(acc[b][m][j + 1], af[m], bf[2], bf[3]);
            }
          }
        }
      }
    }
  }
  cp_async_wait<0>();
  pdl_launch_dependents_if_large();
  const int g = lane >> 2, t = lane & 3;
#pragma unroll
  for (int m = 0; m < MI; ++m)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int row = row_w + m * 16 + g + half * 8;
      if (row >= n_rows) continue;
      if (UP) {
        bf16* dst = (bf16*)(shared ? a.act_s : a.act) + (size_t)(SMALL && !shared ? pair_of[row] : first + row) * N;
        const float wi = a.weigh_input && !shared ? a.wts[pair_of[row]] : 1.0f;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const int col = n0 + col_w + j * 8 + t * 2;
          float y[2];
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            if (GATED) {
              const float gt = fminf(wi * acc[0][m][j][half * 2 + x], a.limit);
              const float up = fminf(fmaxf(wi * acc[NB - 1][m][j][half * 2 + x], -a.limit), a.limit);
              y[x] = gt / (1.0f + expf(-a.slope * gt)) * (up + a.up_offset);
            } else {
              const float up = fmaxf(wi * acc[0][m][j][half * 2 + x], 0.f);
              y[x] = up * up;
            }
          }
          if (col + 1 < N) *reinterpret_cast<uint32_t*>(dst + col) = pack_bf16(y[0], y[1]);
          else if (col < N) dst[col] = from_f32<bf16>(y[0]);
        }
      } else {
        const int p = pair_of[row];
        const int tok = shared ? first + row : p / a.top, jc = shared ? a.top : p % a.top;
        const float w = a.weigh_input || shared ? 1.0f : a.wts[p];
        float* dst = a.out + ((size_t)jc * a.T + tok) * N;
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const int col = n0 + col_w + j * 8 + t * 2;
          if (col + 1 < N)
            *reinterpret_cast<float2*>(dst + col) = make_float2(w * acc[0][m][j][half * 2], w * acc[0][m][j][half * 2 + 1]);
          else if (col < N) dst[col] = w * acc[0][m][j][half * 2];
        }
      }
    }
}

template <int MODE, int BM, bool SMALL = false>
static int moe_tc_launch(const MoeArgs& a, long long pairs, cudaStream_t s) {
  const long long tiles = (SMALL ? (long long)a.E * ((a.T + BM - 1) / BM) : pairs / BM + (pairs < a.E ? pairs : a.E)) +
                          (a.Fs > 0 ? (a.T + BM - 1) / BM : 0);
  if (tiles > 0x7fffffffLL) return GB_ERR_UNSUPPORTED;
  const size_t smem = MoeTile<MODE, BM>::SMEM;
  cudaError_t ce = cudaFuncSetAttribute(moe_tc_kernel<MODE, BM, SMALL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (ce != cudaSuccess) return (int)ce;
  const int N = MODE == MOE_DOWN ? a.W : (a.Fs > a.F ? a.Fs : a.F), BN = MoeTile<MODE, BM>::BN;
  return gb_launch(moe_tc_kernel<MODE, BM, SMALL>, dim3((unsigned)tiles, (N + BN - 1) / BN),
                   dim3(MoeTile<MODE, BM>::THREADS), smem, s, a);
}

template <int BM, bool SMALL = false>
static int moe_tc_products(const MoeArgs& a, long long pairs, cudaStream_t s) {
  int e = a.w_gate ? moe_tc_launch<MOE_GATED, BM, SMALL>(a, pairs, s) : moe_tc_launch<MOE_UNGATED, BM, SMALL>(a, pairs, s);
  return e ? e : moe_tc_launch<MOE_DOWN, BM, SMALL>(a, pairs, s);
}

// A step whose products need no ordered list: few rows, few choices to look through, and
// hardly more blocks (one tile of 16 pairs an expert and 16 rows) than the list would give.
#define MOE_SMALL_ROWS 64
#define MOE_SMALL_PAIRS 512
static bool moe_small(const MoeArgs& a, long long pairs) {
  return a.T <= MOE_SMALL_ROWS && pairs <= MOE_SMALL_PAIRS && pairs <= 4LL * a.E &&
         (long long)a.E * ((a.T + 15) / 16) <= 256;
}

static int moe_check(const MoeArgs& a) {
  if (a.T < 0 || a.W <= 0 || a.F <= 0 || a.E <= 0 || a.n_identity < 0 || a.top <= 0 ||
      a.n_groups <= 0 || a.keep_groups <= 0 || a.keep_groups > a.n_groups)
    return GB_ERR_BAD_ARG;
  const int n_all = a.E + a.n_identity;
  if (n_all % a.n_groups || a.top > n_all) return GB_ERR_BAD_ARG;
  if (n_all > MOE_MAX_OUTPUTS) return GB_ERR_UNSUPPORTED;
  if (a.score_fn < 0 || a.score_fn > 2) return GB_ERR_BAD_ARG;
  if (a.Fs < 0 || (a.Fs > 0 && (!a.ws_up || !a.ws_down || !a.act_s || a.w_gate))) return GB_ERR_BAD_ARG;
  if (!a.x || !a.router_w || !a.w_up || !a.w_down || !a.ids || !a.wts ||
      !a.rank || !a.counts || !a.offsets || !a.perm || !a.act || !a.out)
    return GB_ERR_BAD_ARG;
  return 0;
}

template <typename T>
static int moe_forward(MoeArgs a, cudaStream_t s) {
  int e = moe_check(a);
  if (e) return e;
  if (a.T == 0) return 0;
  const int n_all = a.E + a.n_identity;
  const long long pairs = (long long)a.T * a.top;
  const bool tensor_cores =
      sizeof(T) == 2 && a.W % 8 == 0 && a.F % 8 == 0 && a.Fs % 8 == 0 &&
      ((((uintptr_t)a.ws_up) | ((uintptr_t)a.ws_down) | ((uintptr_t)a.act_s) | ((uintptr_t)a.x) |
        ((uintptr_t)a.act) | ((uintptr_t)a.w_gate) | ((uintptr_t)a.w_up) | ((uintptr_t)a.w_down) |
        ((uintptr_t)a.out)) & 15) == 0;
  a.small = tensor_cores && !a.route_only && moe_small(a, pairs);
  // (where most experts would be asked for weights in vain they wait for the choices)
  a.early = a.small && pairs >= a.E;
  const size_t choice = (size_t)(2 * n_all + a.n_groups) * sizeof(float);
  const size_t staged = ((choice + 15) & ~(size_t)15) + (size_t)n_all * a.W * sizeof(float);
  a.stage_router = a.T <= 64 && a.W % 4 == 0 && ((uintptr_t)a.router_w & 15) == 0 && staged <= 160 * 1024;
  static bool raised = false;      // more than the 48 KB a kernel gets without asking
  if (a.stage_router && !raised) {
    cudaError_t ce = cudaFuncSetAttribute(moe_route_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
    if (ce != cudaSuccess) return (int)ce;
    raised = true;
  }
  const int TPW = 2;
  const size_t by_rows = ((MOE_ROWS_WARPS * TPW * choice + (size_t)2 * a.E * sizeof(int) + 15) & ~(size_t)15) +
                         (size_t)(n_all < MOE_ROUTE_CHUNK ? n_all : MOE_ROUTE_CHUNK) * a.W * sizeof(float);
  static bool raised_rows = false;
  // (its logits are summed in another order; in the 32-bit path a token's are the same to the bit
  // whatever the step brings, so that path keeps to the kernel of a block a token)
  if (sizeof(T) == 2 && a.T > 64 && a.W % 4 == 0 && (((uintptr_t)a.router_w | (uintptr_t)a.x) & 15) == 0 &&
      by_rows <= 200 * 1024) {
    if (!raised_rows) {
      cudaError_t ce = cudaFuncSetAttribute(moe_route_rows_kernel<T, TPW>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
      if (ce != cudaSuccess) return (int)ce;
      raised_rows = true;
    }
    e = gb_launch(moe_route_rows_kernel<T, TPW>, dim3((a.T + MOE_ROWS_WARPS * TPW - 1) / (MOE_ROWS_WARPS * TPW)),
                  dim3(MOE_ROWS_WARPS * 32), by_rows, s, a);
  } else {
    e = gb_launch(moe_route_kernel<T>, dim3(a.T), dim3(MOE_ROUTE_THREADS), a.stage_router ? staged : choice, s, a);
  }
  if (e || a.route_only) return e;
  // the most tiles the pairs can make: every expert may end in a tile that is not full
  if (tensor_cores) {
    if (a.small) return moe_tc_products<16, true>(a, pairs, s);
    // few pairs per expert (a decode step): narrow tiles, deeper pipeline; 64 pairs an expert
    // and more: tiles of 128 rows
    if (pairs <= 4LL * a.E) return moe_tc_products<16>(a, pairs, s);
    if (pairs >= 64LL * a.E) return moe_tc_products<128>(a, pairs, s);
    return moe_tc_products<64>(a, pairs, s);
  }
  if (a.Fs > 0) return GB_ERR_UNSUPPORTED;       // the plain kernels know no shared expert
  const long long tiles = pairs / MOE_BM + (pairs < a.E ? pairs : a.E);
  if (tiles > 0x7fffffffLL) return GB_ERR_UNSUPPORTED;
  e = gb_launch(moe_up_kernel<T>, dim3((unsigned)tiles, (a.F + MOE_BN - 1) / MOE_BN), dim3(256), 0, s, a);
  if (e) return e;
  return gb_launch(moe_down_kernel<T>, dim3((unsigned)tiles, (a.W + MOE_BN - 1) / MOE_BN), dim3(256), 0, s, a);
}

// Three launches: route (with the ordering of the pairs), the experts' first products with
// their activation, their second products with the weights.
GB_EXPORT int gb_moe_forward_f32(const MoeArgs* a, cudaStream_t s) { return moe_forward<float>(*a, s); }
GB_EXPORT int gb_moe_forward_bf16(const MoeArgs* a, cudaStream_t s) { return moe_forward<bf16>(*a, s); }
