// The products of routed experts for many rows (a prompt) on pairs of SMs: a grouped
// product, every expert its own weight and its own run of rows, with
// tcgen05.mma.cta_group::2.
//
// `route` (moe.cu) has left the (token, choice) pairs ordered by expert: list row i is pair
// perm[i], expert e has the list rows offsets[e] .. offsets[e + 1] - 1.  `gather` copies the
// tokens' activations into the list's order, so that an expert's rows are neighbours and one
// TMA box brings 128 of them.  Two launches of the pair kernel follow: the experts' first
// products with their activation (act[i, f]) and their second products with the pair's
// weight (out[choice, token, :], 32-bit).
//
// The pair kernel is that of gemm_tc2.cu with another list of tiles: tile after tile of 256
// list rows x BN columns, expert after expert, dealt to the clusters round robin, an expert's
// row tiles fastest (the clusters running together read the same rows of its weight).  The
// counts are on the device, so every role of every block works the list out from the
// offsets, which all of them keep in shared memory.  A tile's rows beyond its expert's are
// the next expert's (or nothing): they are multiplied and not stored.  Columns beyond the
// expert's likewise.
//
// The experts' first product comes in two forms (MODE): ungated, max(x Wu^T, 0)^2, 256
// columns a tile; gated, where a tile is 128 features, block r of the pair holding the gate
// rows and the up rows of 64 of them one after the other, so that the accumulator's columns
// are 64 gates, their 64 ups, 64 gates, 64 ups.
//
// A shared expert (ungated; weights ws_up, ws_down of Fs inner columns) is the first entry of
// the list: its rows are all tokens, as they lie in x, its weight is 1 and its result
// out[top, token, :].
//
// No copy in this file is a multicast copy.  All waits are bounded (tc_common.cuh); on expiry
// a block records a code in args.error and leaves; its partner's waits run out the same way.
#include "tc_pair.cuh"

#define MP_BM 128        // list rows per block (256 per pair)
#define MP_BNH 128       // weight rows per block (256 per pair)
#define MP_BN 256
#define MP_BK 64
#define MP_STAGES 6
#define MP_THREADS 192   // warp 0: loads; warp 1: MMA issue (first block of the pair); warps 2-5: epilogue
#define MP_MAX_EXPERTS 1024

#define GB_ERR_MP_FULL 141
#define GB_ERR_MP_EMPTY 142
#define GB_ERR_MP_ACC_FULL 143
#define GB_ERR_MP_ACC_EMPTY 144

struct MoePairArgs {
  const void* x;         // [T, W]
  void* xg;              // [T top, W] scratch: the activations in the list's order
  const void* w_gate;    // [E, F, W], or null: the experts have no gate
  const void* w_up;      // [E, F, W]
  const void* w_down;    // [E, W, F]
  const void* ws_up;     // [Fs, W], or null: no shared expert
  const void* ws_down;   // [W, Fs]
  const int* offsets;    // [E + 1]
  const int* perm;       // [T top]
  const float* wts;      // [T top]
  void* act;             // [T top, F]
  void* act_s;           // [T, Fs]
  float* out;            // [top (+ 1 with a shared expert), T, W]
  int* error;
  int T, W, F, Fs, E, top;
  float limit, slope, up_offset;
  int weigh_input;
};

enum MpMode { MP_DOWN = 0, MP_GATED = 1, MP_UNGATED = 2 };

static constexpr int MP_A_BYTES = MP_BM * MP_BK * 2;
static constexpr int MP_B_BYTES = MP_BNH * MP_BK * 2;
static constexpr int MP_STAGE_BYTES = MP_A_BYTES + MP_B_BYTES;
static constexpr size_t MP_SMEM = (size_t)MP_STAGES * MP_STAGE_BYTES + 1024 + 256;
// f32 accumulate, bf16 x bf16, both K-major, M = 256 (over the pair), N = 256
static constexpr uint32_t MP_IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(MP_BN >> 3) << 17) |
                                     ((uint32_t)(256 >> 4) << 24);

#define MP_GATHER_ROWS 4   // rows a block copies side by side: that many loads of a thread under way
__global__ void __launch_bounds__(128) moe_gather_kernel(const MoePairArgs a) {
  pdl_launch_dependents_if_small();
  pdl_wait();
  const int i0 = blockIdx.x * MP_GATHER_ROWS, n = a.W / 8, listed = a.offsets[a.E];
  const uint4* src[MP_GATHER_ROWS];
#pragma unroll
  for (int r = 0; r < MP_GATHER_ROWS; ++r)
    src[r] = reinterpret_cast<const uint4*>((const bf16*)a.x + (size_t)(i0 + r < listed ? a.perm[i0 + r] / a.top : 0) * a.W);
  uint4* dst = reinterpret_cast<uint4*>((bf16*)a.xg + (size_t)i0 * a.W);
  for (int c = threadIdx.x; c < n; c += blockDim.x) {
    uint4 v[MP_GATHER_ROWS];
#pragma unroll
    for (int r = 0; r < MP_GATHER_ROWS; ++r) v[r] = src[r][c];
#pragma unroll
    for (int r = 0; r < MP_GATHER_ROWS; ++r)
      if (i0 + r < listed) dst[(size_t)r * n + c] = v[r];
  }
  pdl_launch_dependents_if_large();
}

// The walk over the list of tiles that every role makes for itself.  Entry 0 is the shared
// expert (no tiles without one), entry e + 1 expert e.
struct MpWalk {
  const int* offs;       // the offsets in shared memory
  int E, T, Fs, tiles_n, tiles_n_shared;
  int entry, base;       // the entry the walk stands at, and the number of its first tile
  int rows, first;       // its list rows (the shared expert's: all tokens, from 0)
  __device__ __forceinline__ void enter(int e) {
    entry = e;
    if (e == 0) {
      first = 0;
      rows = Fs > 0 ? T : 0;
    } else {
      first = offs[e - 1];
      rows = offs[e] - first;
    }
  }
  __device__ __forceinline__ int count() const {
    return ((rows + 255) / 256) * (entry == 0 ? tiles_n_shared : tiles_n);
  }
  // moves to the entry that holds `tile` (no smaller than the last one asked for); false beyond the end
  __device__ __forceinline__ bool seek(int tile) {
    while (tile >= base + count()) {
      base += count();
      if (entry == E) return false;
      enter(entry + 1);
    }
    return true;
  }
  __device__ __forceinline__ void place(int tile, int& tm, int& tn) const {
    const int tiles_m = (rows + 255) / 256, t = tile - base;
    tm = t % tiles_m;
    tn = t / tiles_m;
  }
};

template <int MODE>
__global__ void __launch_bounds__(MP_THREADS, 1)
moe_pair_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_b,
                const __grid_constant__ CUtensorMap map_b2, const __grid_constant__ CUtensorMap map_as,
                const __grid_constant__ CUtensorMap map_bs, const MoePairArgs a) {
  constexpr bool UP = MODE != MP_DOWN;
  constexpr int TILE_COLS = MODE == MP_GATED ? MP_BN / 2 : MP_BN;   // columns of the result per tile
  extern __shared__ uint8_t smem_raw[];
  uint8_t* tiles = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint64_t* bars = (uint64_t*)(tiles + (size_t)MP_STAGES * MP_STAGE_BYTES);
  uint64_t* full = bars;                      // [stages]  used in the pair's first block
  uint64_t* empty = full + MP_STAGES;         // [stages]  in both blocks
  uint64_t* acc_full = empty + MP_STAGES;     // [2]       in both blocks
  uint64_t* acc_empty = acc_full + 2;         // [2]       used in the pair's first block
  __shared__ uint32_t tmem_base_s;
  __shared__ int abort_s;
  __shared__ int offs_s[MP_MAX_EXPERTS + 1];
  volatile int* abort_flag = &abort_s;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t rank = cluster_rank();
  const int cluster = blockIdx.x >> 1, n_clusters = gridDim.x >> 1;
  const int N = UP ? a.F : a.W, Ns = UP ? a.Fs : a.W;
  const int K = UP ? a.W : a.F, Ks = UP ? a.W : a.Fs;

  if (threadIdx.x == 0) {
    tma_prefetch_map(&map_a);
    tma_prefetch_map(&map_b);
    for (int s = 0; s < MP_STAGES; ++s) {
      mbar_init(&full[s], 1);
      mbar_init(&empty[s], 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&acc_full[i], 1);
      mbar_init(&acc_empty[i], 8);   // four epilogue warps in each block of the pair
    }
    abort_s = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {   // the same warp in both blocks, as the pair's allocation asks
    asm volatile("tcgen05.alloc.cta_group::2.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(
                     smem_u32(&tmem_base_s)),
                 "r"(512u)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::2.sync.aligned;" ::: "memory");
  }
  pdl_wait();            // the offsets are an earlier kernel's
  for (int e = threadIdx.x; e <= a.E; e += MP_THREADS) offs_s[e] = a.offsets[e];
  tc_fence_before();
  cluster_sync_all();    // barriers, tensor memory and offsets of both blocks are there from here on
  tc_fence_after();
  const uint32_t tmem_base = tmem_base_s;
  MpWalk walk;
  walk.offs = offs_s;
  walk.E = a.E, walk.T = a.T, walk.Fs = a.Fs;
  walk.tiles_n = (N + TILE_COLS - 1) / TILE_COLS;
  walk.tiles_n_shared = (Ns + TILE_COLS - 1) / TILE_COLS;
  walk.base = 0;
  walk.enter(0);

  if (warp == 0) {
    // ------------------------------------------------------------------ loads (both blocks)
    if (lane == 0) {
      bool ok = true;
      int s = 0;
      uint32_t round = 0;
      for (int tile = cluster; ok && walk.seek(tile); tile += n_clusters) {
        int tm, tn;
        walk.place(tile, tm, tn);
        const bool shared = walk.entry == 0;
        const CUtensorMap* ma = shared ? &map_as : &map_a;
        const CUtensorMap* mb = shared ? &map_bs : &map_b;
        const int kblocks = ((shared ? Ks : K) + MP_BK - 1) / MP_BK;
        const int row_a = walk.first + tm * 256 + (int)rank * MP_BM;
        const int row_b = (shared ? 0 : (walk.entry - 1) * N) + tn * TILE_COLS + (int)rank * (TILE_COLS / 2);
        for (int kb = 0; kb < kblocks; ++kb) {
          if (!mbar_wait(&empty[s], (round & 1) ^ 1, abort_flag)) {
            if (!*abort_flag) atomicCAS(a.error, 0, GB_ERR_MP_EMPTY);
            *abort_flag = 1;
            ok = false;
            break;
          }
          const uint32_t bar = map_to_rank(&full[s], 0);
          if (rank == 0) mbar_expect_tx(&full[s], 2 * MP_STAGE_BYTES);   // both blocks' bytes
          uint8_t* sa = tiles + (size_t)s * MP_STAGE_BYTES;
          tma_load_2d_pair(sa, ma, kb * MP_BK, row_a, bar);
          tma_load_2d_pair(sa + MP_A_BYTES, mb, kb * MP_BK, row_b, bar);
          if (MODE == MP_GATED)       // (boxes of 64 rows: the gates, then their ups)
            tma_load_2d_pair(sa + MP_A_BYTES + MP_B_BYTES / 2, &map_b2, kb * MP_BK, row_b, bar);
          if (++s == MP_STAGES) {
            s = 0;
            ++round;
          }
        }
      }
      pdl_launch_dependents();
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issue (first block)
    if (rank == 0 && lane == 0) {
      int s = 0;
      uint32_t round = 0;
      int t = 0;
      bool ok = true;
      for (int tile = cluster; ok && walk.seek(tile); tile += n_clusters, ++t) {
        const int kblocks = ((walk.entry == 0 ? Ks : K) + MP_BK - 1) / MP_BK;
        const int ab = t & 1;
        if (!mbar_wait(&acc_empty[ab], (((uint32_t)t >> 1) & 1) ^ 1, abort_flag)) {
          if (!*abort_flag) atomicCAS(a.error, 0, GB_ERR_MP_ACC_EMPTY);
          *abort_flag = 1;
          break;
        }
        tc_fence_after();
        const uint32_t acc = tmem_base + ab * MP_BN;
        for (int kb = 0; kb < kblocks; ++kb) {
          if (!mbar_wait(&full[s], round & 1, abort_flag)) {
            if (!*abort_flag) atomicCAS(a.error, 0, GB_ERR_MP_FULL);
            *abort_flag = 1;
            ok = false;
            break;
          }
          tc_fence_after();
          const uint32_t sa = smem_u32(tiles + (size_t)s * MP_STAGE_BYTES);
          const uint64_t da = make_smem_desc(sa), db = make_smem_desc(sa + MP_A_BYTES);
#pragma unroll
          for (int k = 0; k < MP_BK / 16; ++k)
            tc_mma_pair(acc, da + 2 * k, db + 2 * k, MP_IDESC, (kb > 0 || k > 0) ? 1u : 0u);
          tc_commit_pair(&empty[s]);      // the stage is free in both blocks
          if (++s == MP_STAGES) {
            s = 0;
            ++round;
          }
        }
        if (ok) tc_commit_pair(&acc_full[ab]);   // both blocks may drain their half of the tile
      }
    }
  } else {
    // ------------------------------------------------------------------ epilogue (both blocks)
    const int q = warp & 3;   // the TMEM lanes this warp may touch
    const uint32_t lane_addr = tmem_base + ((uint32_t)(q * 32) << 16);
    int t = 0;
    for (int tile = cluster; walk.seek(tile); tile += n_clusters, ++t) {
      int tm, tn;
      walk.place(tile, tm, tn);
      const bool shared = walk.entry == 0;
      const int n_cols = shared ? Ns : N;
      const int ab = t & 1;
      const int in_tile = tm * 256 + (int)rank * MP_BM + q * 32 + lane;
      const bool live = in_tile < walk.rows;
      const int row = walk.first + in_tile;              // list row (the shared expert's: token)
      float wt = 1.f;
      float* orow = nullptr;
      bf16* arow = nullptr;
      if (live) {                                        // what the tile's sums do not decide, before the wait for them
        if (UP) {
          if (!shared && a.weigh_input) wt = a.wts[a.perm[row]];
          arow = shared ? (bf16*)a.act_s + (size_t)row * a.Fs : (bf16*)a.act + (size_t)row * a.F;
        } else if (shared) {
          orow = a.out + ((size_t)a.top * a.T + row) * a.W;
        } else {
          const int p = a.perm[row], tok = p / a.top, jc = p - tok * a.top;
          if (!a.weigh_input) wt = a.wts[p];
          orow = a.out + ((size_t)jc * a.T + tok) * a.W;
        }
      }
      if (!mbar_wait_warp(&acc_full[ab], ((uint32_t)t >> 1) & 1, abort_flag)) {
        if (lane == 0) {
          if (!*abort_flag) atomicCAS(a.error, 0, GB_ERR_MP_ACC_FULL);
          *abort_flag = 1;
        }
        break;
      }
      tc_fence_after();
      const int col0 = tn * TILE_COLS;
#pragma unroll 1
      for (int c0 = 0; c0 < TILE_COLS; c0 += 16) {
        // accumulator columns of result columns c0 .. c0 + 15: with a gate the 64 features of a
        // block are 64 gates and 64 ups
        const uint32_t at = lane_addr + ab * MP_BN + (MODE == MP_GATED ? (c0 >> 6) * 128 + (c0 & 63) : c0);
        uint32_t v[16], u[16];
        tc_ld16(at, v);
        if (MODE == MP_GATED) tc_ld16(at + 64, u);
        tc_wait_ld();
        const int col = col0 + c0;
        const bool store = live && col < n_cols;
        if (UP && store) {
          uint32_t w[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) {
            float y[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              float g = wt * __uint_as_float(v[2 * i + e]);
              if (MODE == MP_GATED) {
                g = fminf(g, a.limit);
                const float up = fminf(fmaxf(wt * __uint_as_float(u[2 * i + e]), -a.limit), a.limit);
                y[e] = g / (1.0f + __expf(-a.slope * g)) * (up + a.up_offset);
              } else {
                g = fmaxf(g, 0.f);
                y[e] = g * g;
              }
            }
            w[i] = pack2(y[0], y[1]);
          }
          // (widths are multiples of eight, so a piece of eight columns is inside or outside whole)
          *reinterpret_cast<uint4*>(arow + col) = make_uint4(w[0], w[1], w[2], w[3]);
          if (col + 8 < n_cols) *reinterpret_cast<uint4*>(arow + col + 8) = make_uint4(w[4], w[5], w[6], w[7]);
        } else if (store) {
#pragma unroll
          for (int c = 0; c < 16; c += 4) {
            if (col + c < n_cols)
              *reinterpret_cast<float4*>(orow + col + c) =
                  make_float4(wt * __uint_as_float(v[c]), wt * __uint_as_float(v[c + 1]),
                              wt * __uint_as_float(v[c + 2]), wt * __uint_as_float(v[c + 3]));
          }
        }
        __syncwarp();          // together again for the next warp-wide load
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive_cluster(map_to_rank(&acc_empty[ab], 0));   // the accumulator may be reused
    }
  }

  // ------------------------------------------------------------------ teardown
  tc_fence_before();
  cluster_sync_all();   // neither block leaves while its partner may still touch its memory
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::2.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(512u)
                 : "memory");
  }
}

template <int MODE>
static int launch(const MoePairArgs& a, int sms, cudaStream_t s) {
  constexpr bool UP = MODE != MP_DOWN;
  static bool configured = false;
  if (!configured) {
    cudaError_t ce = cudaFuncSetAttribute(moe_pair_kernel<MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MP_SMEM);
    if (ce != cudaSuccess) return (int)ce;
    configured = true;
  }
  const uint64_t P = (uint64_t)a.T * a.top, K = UP ? a.W : a.F, N = UP ? a.F : a.W;
  const int box_b = MODE == MP_GATED ? MP_BNH / 2 : MP_BNH;
  CUtensorMap ma, mb, mb2, mas, mbs;
  int e = tc_make_map_2d(&ma, UP ? a.xg : a.act, P, K, K * 2, MP_BM, MP_BK);
  if (e) return e;
  e = tc_make_map_2d(&mb, MODE == MP_GATED ? a.w_gate : UP ? a.w_up : a.w_down, (uint64_t)a.E * N, K, K * 2, box_b, MP_BK);
  if (e) return e;
  mb2 = mb, mas = ma, mbs = mb;
  if (MODE == MP_GATED) {
    e = tc_make_map_2d(&mb2, a.w_up, (uint64_t)a.E * N, K, K * 2, box_b, MP_BK);
    if (e) return e;
  }
  if (a.Fs > 0) {
    const uint64_t Ks = UP ? a.W : a.Fs, Ns = UP ? a.Fs : a.W;
    e = tc_make_map_2d(&mas, UP ? a.x : a.act_s, (uint64_t)a.T, Ks, Ks * 2, MP_BM, MP_BK);
    if (e) return e;
    e = tc_make_map_2d(&mbs, UP ? a.ws_up : a.ws_down, Ns, Ks, Ks * 2, MP_BNH, MP_BK);
    if (e) return e;
  }
  return gb_launch_cluster(moe_pair_kernel<MODE>, dim3((unsigned)(2 * (sms / 2))), dim3(MP_THREADS), MP_SMEM, s, 2,
                           ma, mb, mb2, mas, mbs, a);
}

// Three launches (gather, first products, second products) behind `route`.  W, F and Fs must
// be multiples of eight and every tensor 16-byte aligned; a shared expert goes with ungated
// experts.
GB_EXPORT int gb_moe_pair_bf16(const MoePairArgs* args, cudaStream_t s) {
  const MoePairArgs& a = *args;
  if (a.T < 0 || a.W <= 0 || a.F <= 0 || a.E <= 0 || a.top <= 0 || a.Fs < 0) return GB_ERR_BAD_ARG;
  if (!a.x || !a.xg || !a.w_up || !a.w_down || !a.offsets || !a.perm || !a.wts || !a.act || !a.out || !a.error)
    return GB_ERR_BAD_ARG;
  if (a.Fs > 0 && (!a.ws_up || !a.ws_down || !a.act_s || a.w_gate)) return GB_ERR_BAD_ARG;
  if (a.E > MP_MAX_EXPERTS || a.W % 8 || a.F % 8 || a.Fs % 8) return GB_ERR_UNSUPPORTED;
  const uintptr_t all = (uintptr_t)a.x | (uintptr_t)a.xg | (uintptr_t)a.w_gate | (uintptr_t)a.w_up |
                        (uintptr_t)a.w_down | (uintptr_t)a.ws_up | (uintptr_t)a.ws_down | (uintptr_t)a.act |
                        (uintptr_t)a.act_s | (uintptr_t)a.out;
  if (all & 15) return GB_ERR_BAD_ARG;
  const long long most = 0x7fffffffLL - 512;            // TMA coordinates are 32-bit
  if ((long long)a.T * a.top > most || (long long)a.E * a.F > most || (long long)a.E * a.W > most) return GB_ERR_UNSUPPORTED;
  if (a.T == 0) return 0;
  static int sms = 0;
  if (!sms) {
    int dev = 0;
    cudaError_t e = cudaGetDevice(&dev);
    if (e == cudaSuccess) e = cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    if (e != cudaSuccess) return (int)e;
  }
  if (sms < 2) return GB_ERR_UNSUPPORTED;
  int e = gb_launch(moe_gather_kernel, dim3((unsigned)((a.T * a.top + MP_GATHER_ROWS - 1) / MP_GATHER_ROWS)), dim3(128), 0, s, a);
  if (e) return e;
  e = a.w_gate ? launch<MP_GATED>(a, sms, s) : launch<MP_UNGATED>(a, sms, s);
  if (e) return e;
  return launch<MP_DOWN>(a, sms, s);
}
