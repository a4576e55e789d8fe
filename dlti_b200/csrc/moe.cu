// Mixtures of experts and gated activations.
//
//   moe_route        one warp per token: sigmoid scores, groups, the top experts and their weights (or the top logits and their
//                    softmax); every (token, choice) pair
//                    = token * top + choice is appended to its expert's list. Further blocks of the same launch apply an
//                    activation to other columns of the same projection (the shared expert).
//   moe_gemm         grouped GEMM over the lists, bf16, by CTA pairs: weights are the 256-row operand of tcgen05.mma and the
//                    pairs of a list its columns (32 to 256 of them), so one kernel serves one decoded token and whole
//                    prompts. The first GEMM of an expert gathers the pairs' source rows and leaves its results one list after
//                    the other; the second reads them as they lie and scatters to row `pair`. Gate and up rows alternate in the
//                    first one's weights, so that the activation is an exchange between neighbouring lanes of the epilogue.
//   moe_gemm_f32     the same in fp32 FMAs
//
// Pair lists are filled with atomics, so their order differs from run to run; a pair's result does not depend on its place.
#include "pair.cuh"
#include "rows.cuh"

namespace {

__device__ __forceinline__ float gated(float g, float u, float limit) {
  if (limit == 0.f) return silu_f(g) * u;
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * sigmoid_f(1.702f * g) * (u + 1.f);
}
__device__ __forceinline__ float gated_fast(float g, float u, float limit) {          // 16-bit results
  if (limit == 0.f) return g * fast_sigmoid(g) * u;
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g * fast_sigmoid(1.702f * g) * (u + 1.f);
}

struct RouteParams {
  const float* z; long long z_ld; int col;                 // router logits at column col of fp32 rows
  const float* corr;
  int E, top, groups, keep; float scale;
  int softmax;                                             // logits + corr decide, weights = their softmax among the chosen
  int sg; float* share;                                    // share[t] = sigmoid of column sg (sg < 0: none)
  float* wgt; int *lists, *counts;                         // [T, top]; [E, T]; [E]
  const void* p; long long p_ld; int og, ou, ff; float limit;      // projection columns of the activation (ff 0: none; og < 0: square of relu)
  void* h; long long h_ld;
  long long T;
};
constexpr int ROUTE_WARPS = 4;

__device__ __forceinline__ unsigned ordered(float v) {     // unsigned integers in the order of the floats
  const unsigned u = __float_as_uint(v);
  return u & 0x80000000u ? ~u : u | 0x80000000u;
}
// Expert choice of one token by one warp, R scores a lane. sc: choice scores, sg: group scores (shared memory); sel / share: the
// chosen experts and their scores.
template <bool ACC, int R>
__device__ __forceinline__ void route_token(const RouteParams& p, long long t, float* sc, float* sg, int* sel, float* share) {
  const int lane = threadIdx.x & 31, n = p.E / p.groups;
  const float* zr = p.z + t * p.z_ld + p.col;
  float s[R], c[R];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int e = lane + 32 * i;
    s[i] = 0.f;
    c[i] = -INFINITY;
    if (e < p.E) {
      const float v = zr[e];
      if (ACC) const_cast<float*>(zr)[e] = 0.f;
      s[i] = p.softmax ? v + p.corr[e] : sigmoid_f(v);
      c[i] = p.softmax ? s[i] : s[i] + p.corr[e];
    }
  }
  if (p.sg >= 0 && lane == 0) {
    float* zs = const_cast<float*>(p.z) + t * p.z_ld + p.sg;
    p.share[t] = sigmoid_f(*zs);
    if (ACC) *zs = 0.f;
  }
  if (p.keep < p.groups) {
    __syncwarp();
#pragma unroll
    for (int i = 0; i < R; ++i)
      if (lane + 32 * i < p.E) sc[lane + 32 * i] = c[i];
    __syncwarp();
    for (int g = lane; g < p.groups; g += 32) {            // a group's score: its two largest choice scores
      float a = -INFINITY, b = -INFINITY;
      for (int e = g * n; e < (g + 1) * n; ++e) {
        const float v = sc[e];
        if (v > a) { b = a; a = v; }
        else if (v > b) b = v;
      }
      sg[g] = n > 1 ? a + b : a;
    }
    __syncwarp();
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int e = lane + 32 * i;
      if (e < p.E) {
        const int g = e / n;
        int better = 0;
        for (int o = 0; o < p.groups; ++o) better += sg[o] > sg[g] || (sg[o] == sg[g] && o < g);
        if (better >= p.keep) c[i] = -INFINITY;
      }
    }
  }
  float sum = 0.f, largest = 0.f;
  for (int k = 0; k < p.top; ++k) {
    unsigned best = 0;
    int bi = p.E;
    float bs = 0.f;
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const unsigned o = c[i] == -INFINITY ? 0u : ordered(c[i]);
      if (o > best) { best = o; bi = lane + 32 * i; bs = s[i]; }
    }
    const unsigned top = __reduce_max_sync(0xffffffffu, best);
    int e = (int)__reduce_min_sync(0xffffffffu, best == top && bi < p.E ? (unsigned)bi : 0x7fffffffu);
    if (e >= p.E) e = k;                                   // only where the scores are not numbers
    bs = __shfl_sync(0xffffffffu, bi == e ? bs : 0.f, e & 31);
    if (p.softmax) {
      if (k == 0) largest = bs;
      bs = expf(bs - largest);
    }
    if ((e & 31) == lane)
#pragma unroll
      for (int i = 0; i < R; ++i)
        if (e == lane + 32 * i) c[i] = -INFINITY;
    if (lane == 0) {
      sel[k] = e;
      share[k] = bs;
    }
    sum += bs;
  }
  __syncwarp();
  const float f = p.scale / (sum + 1e-20f);
  for (int k = lane; k < p.top; k += 32) p.wgt[t * p.top + k] = share[k] * f;
}

// A block routes `per` tokens a warp, counts its pairs in shared memory and takes its places in the lists with one atomic per expert.
template <bool ACC, int R>
__device__ __forceinline__ void route_block(const RouteParams& p, int per) {
  extern __shared__ float route_s[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tokens = ROUTE_WARPS * per;
  int* cnt = reinterpret_cast<int*>(route_s);              // [E] pairs of this block, then their first place
  int* sel = cnt + p.E;                                    // [tokens][top]
  int* rank = sel + tokens * p.top;                        // [tokens][top] (scores first)
  float* sc = reinterpret_cast<float*>(rank + tokens * p.top) + warp * (p.E + p.groups);
  for (int e = threadIdx.x; e < p.E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  const long long t0 = (long long)blockIdx.x * tokens;
  for (int i = 0; i < per; ++i) {
    const int x = warp * per + i;
    if (t0 + x >= p.T) break;
    route_token<ACC, R>(p, t0 + x, sc, sc + p.E, sel + x * p.top, reinterpret_cast<float*>(rank + x * p.top));
    __syncwarp();
    for (int k = lane; k < p.top; k += 32) rank[x * p.top + k] = atomicAdd(cnt + sel[x * p.top + k], 1);
  }
  __syncthreads();
  for (int e = threadIdx.x; e < p.E; e += blockDim.x)
    if (cnt[e]) cnt[e] = atomicAdd(p.counts + e, cnt[e]);
  __syncthreads();
  const int n = (int)min((long long)tokens, p.T - t0) * p.top;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const int e = sel[i], r = cnt[e] + rank[i];
    if ((unsigned)r < (unsigned)p.T) p.lists[e * p.T + r] = (int)(t0 * p.top + i);
  }
}

template <typename T, bool ACC, int W, int R>
__global__ void __launch_bounds__(32 * ROUTE_WARPS) moe_route_kernel(const RouteParams p, int route_blocks, int route_per) {
  griddep_wait();
  griddep_launch();
  if ((int)blockIdx.x < route_blocks) {
    route_block<ACC, R>(p, route_per);
    return;
  }
  const int per = p.ff / W;
  const long long total = p.T * per, step = (long long)(gridDim.x - route_blocks) * blockDim.x;
  for (long long i = (long long)(blockIdx.x - route_blocks) * blockDim.x + threadIdx.x; i < total; i += step) {
    const long long t = i / per;
    const int c = (int)(i - t * per) * W;
    const void* row = reinterpret_cast<const uint8_t*>(p.p) + t * p.p_ld * (ACC ? 4 : sizeof(T));
    T* o = reinterpret_cast<T*>(p.h) + t * p.h_ld + c;
    if (p.og < 0) {
      float u[W];
      if constexpr (W == 1) u[0] = take<T, ACC>(row, p.ou + c);
      else take_n<T, ACC, W>(row, p.ou + c, u);
#pragma unroll
      for (int j = 0; j < W; ++j) {
        u[j] = fmaxf(u[j], 0.f);
        u[j] *= u[j];
      }
      if constexpr (W == 1) *o = Cvt<T>::from_f(u[0]);
      else put_n(o, u);
    } else if constexpr (W == 1) {
      const float g = take<T, ACC>(row, p.og + c), u = take<T, ACC>(row, p.ou + c);
      *o = Cvt<T>::from_f(gated(g, u, p.limit));
    } else {
      float g[W], u[W];
      take_n<T, ACC, W>(row, p.og + c, g);
      take_n<T, ACC, W>(row, p.ou + c, u);
#pragma unroll
      for (int j = 0; j < W; ++j) g[j] = gated_fast(g[j], u[j], p.limit);
      put_n(o, g);
    }
  }
}

// ---- grouped GEMM ------------------------------------------------------------------------------------------
struct MoeGemmParams {
  const int *lists, *counts;
  int E, cap, div;                                         // experts; capacity of a list; pairs per source row
  int rows, wrows, K;                                      // output columns; weight rows of an expert
  float limit;
  void* out; long long o_ld;
  int x_rows, o_rows;                                      // list entries outside these are not followed (counters of an aborted step)
  int NT, MT, stages;                                      // columns of a tile (multiple of 32, at most 256), weight tiles of an expert
};
// UP: the source of list entry i is row lists[i] / div, its result goes to row (start of the list) + i (MOE_SWIGLU: activation of
// rows 2 r and 2 r + 1, MOE_RELU2: of row r). Otherwise the source is row (start of the list) + i and the result goes to row lists[i].
enum MoeMode : int { MOE_DOWN = 0, MOE_SWIGLU = 1, MOE_RELU2 = 2 };
constexpr int MG_GATHERS = 8, MG_THREADS = 320 + 32 * MG_GATHERS, MG_A_BYTES = 16384, MG_MAX_STAGES = 10, MG_SMEM = 226 * 1024;
constexpr int MG_TAIL = 8 * (3 * MG_MAX_STAGES + 4) + 16;  // barriers, TMEM address
constexpr long long MG_WAIT_LIMIT = 4000000000LL;

// rows r0 .. r3 of a matrix (box of one row) one after the other; completion bytes on a barrier that may live in the peer CTA
__device__ __forceinline__ void tma_gather4_2sm(uint32_t dst, const CUtensorMap* m, uint32_t bar_cluster, int c, int r0, int r1, int r2, int r3) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.tile::gather4.mbarrier::complete_tx::bytes.cta_group::2 "
      "[%0], [%1, {%3, %4, %5, %6, %7}], [%2];" ::"r"(dst),
      "l"(reinterpret_cast<uint64_t>(m)), "r"(bar_cluster), "r"(c), "r"(r0), "r"(r1), "r"(r2), "r"(r3)
      : "memory");
}

struct MoeTile { int e, m, n0, nn; };
// tile t of the launch; first[e] = tiles before expert e
__device__ __forceinline__ MoeTile moe_tile(const MoeGemmParams& p, const int* first, const int* cnt, int t) {
  int lo = 0, hi = p.E - 1;                                // the last expert whose first tile is not after t
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (first[mid] <= t) lo = mid;
    else hi = mid - 1;
  }
  const int r = t - first[lo], c = cnt[lo];
  const int nt = (c + p.NT - 1) / p.NT, per = ((c + nt - 1) / nt + 31) & ~31;
  const int n0 = (r / p.MT) * per;
  return MoeTile{lo, r % p.MT, n0, min(c - n0, per)};
}

// A CTA of the pair stages 128 weight rows and half of the tile's columns; the leader issues the MMAs, and each CTA ends up with its
// 128 rows of the accumulator (two of them, so that the epilogue overlaps the next tile). Warp 0: weights; warp 1: MMAs; warps 2-9:
// epilogue; warps 10-17: the gathered columns, four rows a copy (a copy costs its issuing thread about 100 clk, so they share them),
// or warp 10 where they lie together. Waits are bounded: a CTA that gives up writes NaN.
template <int MODE>
__global__ void __cluster_dims__(2, 1, 1) __launch_bounds__(MG_THREADS, 1)
moe_gemm_kernel(const MoeGemmParams p, const __grid_constant__ CUtensorMap tw, const __grid_constant__ CUtensorMap tx) {
  constexpr bool UP = MODE != MOE_DOWN;
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t stage_bytes = MG_A_BYTES + p.NT * 64;
  const uint32_t full = base + p.stages * stage_bytes, empty = full + 8 * MG_MAX_STAGES, passed = empty + 8 * MG_MAX_STAGES,
                 acc_full = passed + 8 * MG_MAX_STAGES, acc_empty = acc_full + 16, slot = acc_empty + 16;
  uint8_t* tail = smem_raw + (slot - smem_u32(smem_raw)) + 16;
  volatile uint32_t* slot_ptr = reinterpret_cast<volatile uint32_t*>(tail - 16);
  int* s_dst = reinterpret_cast<int*>(tail);               // [2][256]
  int* s_first = s_dst + 512;                              // [E]: tiles before an expert
  int* s_row = s_first + p.E;                              // [E]: pairs before an expert
  int* s_cnt = s_row + p.E;                                // [E]
  __shared__ int2 s_scan[32];
  __shared__ int s_fail;
  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
  const uint32_t rank = __shfl_sync(0xffffffffu, cluster_ctarank(), 0);
  const int cid = blockIdx.x >> 1, ncl = gridDim.x >> 1;
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tw);
    tma_prefetch_desc(&tx);
    s_fail = 0;
    for (int s = 0; s < p.stages; ++s) {
      mbar_init(full + 8 * s, 1);                          // the leader's: bytes of both CTAs
      mbar_init(empty + 8 * s, 1);
      mbar_init(passed + 8 * s, MG_GATHERS);
    }
    for (int a = 0; a < 2; ++a) {
      mbar_init(acc_full + 8 * a, 1);
      mbar_init(acc_empty + 8 * a, 16);                    // the leader's: eight warps of both CTAs
    }
    mbar_fence_init();
  }
  griddep_wait();
  cluster_sync_all();
  if (warp == 1) {
    tmem_alloc2(slot, 512);
    tmem_relinquish2();
  }
  // tiles and pairs before every expert: a block-wide prefix sum, MG_THREADS experts at a time
  int2 carry = make_int2(0, 0);
  for (int e0 = 0; e0 < p.E; e0 += MG_THREADS) {
    const int e = e0 + threadIdx.x;
    const int c = e < p.E ? max(0, min(p.counts[e], p.cap)) : 0;
    const int v = (c + p.NT - 1) / p.NT * p.MT;
    int x = v, y = c;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int xo = __shfl_up_sync(0xffffffffu, x, o), yo = __shfl_up_sync(0xffffffffu, y, o);
      if (lane >= o) { x += xo; y += yo; }
    }
    if (lane == 31) s_scan[warp] = make_int2(x, y);
    __syncthreads();
    int2 before = carry;
    for (int w = 0; w < MG_THREADS / 32; ++w) {
      if (w < warp) { before.x += s_scan[w].x; before.y += s_scan[w].y; }
      carry.x += s_scan[w].x;
      carry.y += s_scan[w].y;
    }
    if (e < p.E) {
      s_cnt[e] = c;
      s_first[e] = before.x + x - v;
      s_row[e] = before.y + y - c;
    }
    __syncthreads();
  }
  const int total = carry.x;
  tc_fence_before();
  cluster_sync_all();
  tc_fence_after();
  griddep_launch();                                        // only now: the next kernel may want tensor memory too
  const uint32_t tmem = __shfl_sync(0xffffffffu, *slot_ptr, 0);
  const int nkb = (p.K + 63) / 64;
  volatile int* fail = &s_fail;
  auto wait = [&](uint32_t bar, uint32_t parity) {
    if (mbar_try_wait(bar, parity)) return true;
    const long long t0 = clock64();
    while (!mbar_try_wait(bar, parity))
      if (*fail || clock64() - t0 > MG_WAIT_LIMIT) {
        *fail = 1;
        return false;
      }
    return true;
  };
  auto wait_warp = [&](uint32_t bar, uint32_t parity) { return __all_sync(0xffffffffu, wait(bar, parity)) != 0; };     // the warp stays together
  auto failed = [&]() { return __any_sync(0xffffffffu, *fail) != 0; };
  const uint32_t lead_full = mapa_rank(full, 0);

  if (warp == 0 || (!UP && warp == 10)) {
    if (lane == 0) {
      int s = 0, round = 0;
      for (int t = cid; t < total && !*fail; t += ncl) {
        const MoeTile x = moe_tile(p, s_first, s_cnt, t);
        if (x.nn <= 0) continue;
        const int w0 = x.e * p.wrows + x.m * 256 + (int)rank * 128;
        const int nh = ((x.nn + 31) & ~31) >> 1, r0 = s_row[x.e] + x.n0 + (int)rank * nh;
        const int groups = ((min(nh, x.nn) + 3) >> 2) + ((max(0, x.nn - nh) + 3) >> 2);
        for (int kb = 0; kb < nkb; ++kb) {
          // Gathering, the weights of a k block follow the gathering warps: one without rows in this tile has nothing else that would
          // keep it within a phase of the others.
          if (UP ? !wait(passed + 8 * s, round & 1) : round > 0 && !wait(empty + 8 * s, (round - 1) & 1)) break;
          const uint32_t dst = base + s * stage_bytes, bar = lead_full + 8 * s;
          if (warp == 0) {
            if (rank == 0) mbar_expect_tx(full + 8 * s, 2 * MG_A_BYTES + (UP ? groups * 512 : p.NT * 128));
            tma_load_2d_2sm(dst, &tw, bar, kb * 64, w0);
          } else {
            tma_load_2d_2sm(dst + MG_A_BYTES, &tx, bar, kb * 64, r0);
          }
          if (++s == p.stages) { s = 0; ++round; }
        }
      }
    }
  } else if (warp == 1) {
    if (rank == 0) {
      const bool leader = elect_one_sync();
      int s = 0, round = 0, tile = 0;
      for (int t = cid; t < total && !failed(); t += ncl) {
        const MoeTile x = moe_tile(p, s_first, s_cnt, t);
        if (x.nn <= 0) continue;
        const int a = tile & 1, use = tile >> 1;
        if (use > 0 && !wait_warp(acc_empty + 8 * a, (use - 1) & 1)) break;
        tc_fence_after();
        const uint32_t idesc = umma_idesc_f16(DLTI_BF16, 256, (x.nn + 31) & ~31, false, false), d = tmem + a * 256;
        for (int kb = 0; kb < nkb; ++kb) {
          if (!wait_warp(full + 8 * s, round & 1)) break;
          tc_fence_after();
          const uint32_t sm = base + s * stage_bytes;
          const DescLoHi da = desc_split(sm, 0, 1024), db = desc_split(sm + MG_A_BYTES, 0, 1024);
          if (leader) {
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) umma_f16_ss_2sm(d, da.at(kk * 32), db.at(kk * 32), idesc, kb > 0 || kk > 0);
            umma_commit_2sm(empty + 8 * s);
            if (kb == nkb - 1) umma_commit_2sm(acc_full + 8 * a);
          }
          __syncwarp();
          if (++s == p.stages) { s = 0; ++round; }
        }
        ++tile;
      }
    }
  } else if (warp < 10) {
    const int quarter = warp & 3, half = (warp - 2) >> 2;
    const uint32_t lead_empty = mapa_rank(acc_empty, 0);
    int tile = 0;
    for (int t = cid; t < total; t += ncl) {
      const MoeTile x = moe_tile(p, s_first, s_cnt, t);
      if (x.nn <= 0) continue;
      const int a = tile & 1, use = tile >> 1;
      int* dst = s_dst + a * 256;
      const int i0 = threadIdx.x - 64;
      if (i0 < x.nn) dst[i0] = UP ? s_row[x.e] + x.n0 + i0 : p.lists[(long long)x.e * p.cap + x.n0 + i0];
      asm volatile("bar.sync 1, 256;" ::: "memory");
      const bool ok = wait_warp(acc_full + 8 * a, use & 1);
      tc_fence_after();
      const uint32_t d = tmem + ((uint32_t)(quarter * 32) << 16) + a * 256;
      const int row = x.m * 256 + (int)rank * 128 + quarter * 32 + lane;
      // Each round of exchanges hands half of a lane's columns to the lane next to it (then two, then four away) for half of that
      // one's rows: at the end lane l has column l % 8 of eight neighbouring rows, and stores them in one piece.
      const int b0 = lane & 1, b1 = lane & 2, b2 = lane & 4, r0 = row & ~7;
      auto swap_f = [&](bool odd, float a, float b, int d) { return __shfl_xor_sync(0xffffffffu, odd ? a : b, d); };
      auto swap_u = [&](bool odd, uint32_t a, uint32_t b, int d) { return __shfl_xor_sync(0xffffffffu, odd ? a : b, d); };
      using B = __nv_bfloat16;
      for (int c = half * 32; c < x.nn; c += 64) {
        uint32_t v[32];
        if (ok) {
          tmem_ld_32x32b_x32(d + c, v);
          tmem_wait_ld();
        } else {
#pragma unroll
          for (int j = 0; j < 32; ++j) v[j] = 0x7fffffffu;
        }
#pragma unroll
        for (int j = 0; j < 32; j += 8) {
          const int i = c + j + (lane & 7), to = dst[i & 255];      // stale past the tile's columns
          B* out = reinterpret_cast<B*>(p.out) + (long long)to * p.o_ld;
          const bool on = i < x.nn && (unsigned)to < (unsigned)p.o_rows;
          if constexpr (MODE == MOE_SWIGLU) {              // even lanes hold gates, odd lanes up values
            float f[4];
#pragma unroll
            for (int y = 0; y < 4; ++y) {
              const float v0 = __uint_as_float(v[j + 2 * y]), v1 = __uint_as_float(v[j + 2 * y + 1]), other = swap_f(b0, v0, v1, 1);
              f[y] = gated_fast(b0 ? other : v0, b0 ? v1 : other, p.limit);
            }
            uint32_t u[2];
#pragma unroll
            for (int y = 0; y < 2; ++y) {
              const float other = swap_f(b1, f[2 * y], f[2 * y + 1], 2);
              u[y] = b1 ? Cvt<B>::pack2(other, f[2 * y + 1]) : Cvt<B>::pack2(f[2 * y], other);
            }
            const uint32_t other = swap_u(b2, u[0], u[1], 4);
            if (on && r0 / 2 < p.rows) *reinterpret_cast<uint2*>(out + r0 / 2) = b2 ? make_uint2(other, u[1]) : make_uint2(u[0], other);
          } else {
            uint32_t u[4];
#pragma unroll
            for (int y = 0; y < 4; ++y) {
              float v0 = __uint_as_float(v[j + 2 * y]), v1 = __uint_as_float(v[j + 2 * y + 1]);
              if constexpr (MODE == MOE_RELU2) {           // what is not a number stays so
                v0 = v0 < 0.f ? 0.f : v0 * v0;
                v1 = v1 < 0.f ? 0.f : v1 * v1;
              }
              const float other = swap_f(b0, v0, v1, 1);
              u[y] = b0 ? Cvt<B>::pack2(other, v1) : Cvt<B>::pack2(v0, other);
            }
            uint2 w[2];
#pragma unroll
            for (int y = 0; y < 2; ++y) {
              const uint32_t other = swap_u(b1, u[2 * y], u[2 * y + 1], 2);
              w[y] = b1 ? make_uint2(other, u[2 * y + 1]) : make_uint2(u[2 * y], other);
            }
            const uint32_t o0 = swap_u(b2, w[0].x, w[1].x, 4), o1 = swap_u(b2, w[0].y, w[1].y, 4);
            if (on && r0 < p.rows) *reinterpret_cast<uint4*>(out + r0) = b2 ? make_uint4(o0, o1, w[1].x, w[1].y) : make_uint4(w[0].x, w[0].y, o0, o1);
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive_peer(lead_empty + 8 * a);
      ++tile;
    }
  } else if (UP) {
    // rows past the list keep what their shared memory held: their columns are dropped
    const int g = (warp - 10) + lane * MG_GATHERS;          // a short list's copies are spread over the warps too
    int s = 0, round = 0;
    for (int t = cid; t < total && !failed(); t += ncl) {
      const MoeTile x = moe_tile(p, s_first, s_cnt, t);
      if (x.nn <= 0) continue;
      const int nh = ((x.nn + 31) & ~31) >> 1, first = (int)rank * nh, n = min(nh, x.nn - first);
      const bool mine = g < 32 && 4 * g < n;
      int src[4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
        src[i] = mine ? (int)min((unsigned)p.lists[(long long)x.e * p.cap + x.n0 + first + min(4 * g + i, n - 1)] / p.div, (unsigned)p.x_rows - 1) : 0;
      for (int kb = 0; kb < nkb; ++kb) {
        if (round > 0 && !wait_warp(empty + 8 * s, (round - 1) & 1)) break;
        if (mine) tma_gather4_2sm(base + s * stage_bytes + MG_A_BYTES + g * 512, &tx, lead_full + 8 * s, kb * 64, src[0], src[1], src[2], src[3]);
        __syncwarp();
        if (lane == 0) mbar_arrive(passed + 8 * s);
        if (++s == p.stages) { s = 0; ++round; }
      }
    }
  }
  if (*fail) {                                             // copies may still be in flight: leave their shared memory alone for a while
    const long long t0 = clock64();
    while (clock64() - t0 < 20000000LL) {
    }
  }
  tc_fence_before();
  __syncwarp();
  cluster_sync_all();                                      // the pair's tensor cores read both CTAs' shared memory until here
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc2(tmem, 512);
  }
}

// CTA = (64 outputs, expert), 16 pairs at a time; thread = one output of 4 pairs
template <int MODE>
__global__ void __launch_bounds__(256) moe_gemm_f32_kernel(const float* __restrict__ X, long long x_ld, const float* __restrict__ Wt, long long w_ld,
                                                           const MoeGemmParams p) {
  constexpr bool UP = MODE != MOE_DOWN;
  __shared__ float sw[2][16][65], sx[16][17];
  __shared__ int s_src[16], s_to[16], s_start;
  const int e = blockIdx.y, r0 = blockIdx.x * 64, cnt = max(0, min(p.counts[e], p.cap));
  if (threadIdx.x < 32) {                                  // pairs before this expert
    int before = 0;
    for (int i = threadIdx.x; i < e; i += 32) before += max(0, min(p.counts[i], p.cap));
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) before += __shfl_xor_sync(0xffffffffu, before, o);
    if (threadIdx.x == 0) s_start = before;
  }
  const int r = threadIdx.x & 63, tg = threadIdx.x >> 6;
  constexpr int parts = MODE == MOE_SWIGLU ? 2 : 1;
  for (int n0 = 0; n0 < cnt; n0 += 16) {
    __syncthreads();
    if (threadIdx.x < 16) {
      const int i = min(n0 + (int)threadIdx.x, cnt - 1), pair = p.lists[(long long)e * p.cap + i];
      s_src[threadIdx.x] = min(UP ? (unsigned)pair / p.div : (unsigned)(s_start + i), (unsigned)p.x_rows - 1);
      s_to[threadIdx.x] = UP ? s_start + i : pair;
    }
    __syncthreads();
    float acc[2][4] = {};
    for (int k0 = 0; k0 < p.K; k0 += 16) {
      for (int i = threadIdx.x; i < parts * 64 * 16; i += 256) {
        const int q = i / (64 * 16), rr = (i / 16) % 64, k = i % 16;
        sw[q][k][rr] = (r0 + rr < p.rows && k0 + k < p.K) ? Wt[((long long)e * p.wrows + (MODE == MOE_SWIGLU ? 2 * (r0 + rr) + q : r0 + rr)) * w_ld + k0 + k] : 0.f;
      }
      {
        const int i = threadIdx.x, tt = i / 16, k = i % 16;
        sx[tt][k] = k0 + k < p.K ? X[(long long)s_src[tt] * x_ld + k0 + k] : 0.f;
      }
      __syncthreads();
      for (int q = 0; q < parts; ++q) {
        float part[4] = {};
#pragma unroll
        for (int k = 0; k < 16; ++k) {
          const float w = sw[q][k][r];
#pragma unroll
          for (int j = 0; j < 4; ++j) part[j] = fmaf(w, sx[tg * 4 + j][k], part[j]);
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[q][j] += part[j];
      }
      __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = tg * 4 + j;
      float v = acc[0][j];
      if (MODE == MOE_SWIGLU) v = gated(v, acc[1][j], p.limit);
      if (MODE == MOE_RELU2) v = v < 0.f ? 0.f : v * v;
      if (n0 + i < cnt && r0 + r < p.rows && (unsigned)s_to[i] < (unsigned)p.o_rows)
        reinterpret_cast<float*>(p.out)[(long long)s_to[i] * p.o_ld + r0 + r] = v;
    }
  }
}

template <typename T, bool ACC, int W>
int launch_route(const RouteParams& p, cudaStream_t st) {
  const int per = p.T >= 4096 ? 2 : 1, tokens = ROUTE_WARPS * per;
  const int rb = p.E ? (int)((p.T + tokens - 1) / tokens) : 0;
  const int ab = p.ff ? grid_for(p.T * (p.ff / W), 32 * ROUTE_WARPS) : 0;
  const size_t smem = p.E ? (size_t)(p.E + 2 * tokens * p.top + ROUTE_WARPS * (p.E + p.groups)) * 4 : 0;
  if (smem > 48 * 1024) { dlti_set_error("moe_route: too many experts and choices"); return DLTI_ERR_TOO_LARGE; }
  auto kern = p.E <= 32 ? moe_route_kernel<T, ACC, W, 1> : p.E <= 64 ? moe_route_kernel<T, ACC, W, 2> : p.E <= 128 ? moe_route_kernel<T, ACC, W, 4>
              : p.E <= 256 ? moe_route_kernel<T, ACC, W, 8> : moe_route_kernel<T, ACC, W, 32>;
  DLTI_CUDA_CHECK(dlti_launch_pdl(p.T, kern, dim3(rb + ab), dim3(32 * ROUTE_WARPS), smem, st, p, rb, per));
  dlti_count_launch();
  return 0;
}

}  // namespace

// experts 0: no routing; ff 0: no activation. acc: z and p are the decode GEMM's accumulator (zero on return in the columns read).
DLTI_API int dlti_moe_route(const float* z, long long z_ld, int col, const float* corr, int E, int top, int groups, int keep, float scale,
                            int softmax, float* wgt, int* lists, int* counts, int sg, float* share, const void* p, long long p_ld, int og, int ou, int ff, float limit, void* h,
                            long long h_ld, long long T, int acc, int dtype, cudaStream_t st) {
  if (T <= 0) return 0;
  if (E && (!z || !corr || !wgt || !lists || !counts || groups < 1 || E % groups || keep < 1 || keep > groups || top < 1 || top > E / groups * keep))
    return DLTI_ERR_BAD_ARG;
  if (E > 1024 || T * (top > 1 ? top : 1) > 0x7fffffffLL) { dlti_set_error("moe_route: up to 1024 experts"); return DLTI_ERR_TOO_LARGE; }
  if ((ff && (!p || !h)) || (softmax && groups > 1) || (sg >= 0 && (!E || !share))) return DLTI_ERR_BAD_ARG;
  if (!E && !ff) return 0;
  const RouteParams r{z, z_ld, col, corr, E, top, groups, keep, scale, softmax, sg, share, wgt, lists, counts, p, p_ld, og, ou, ff, limit, h, h_ld, T};
  using B = __nv_bfloat16;
  if (dtype == DLTI_BF16) {
    const bool vec = ((ff | (og < 0 ? 0 : og) | ou) & 7) == 0 && ((p_ld | h_ld) & 7) == 0 && ((reinterpret_cast<uintptr_t>(p) | reinterpret_cast<uintptr_t>(h)) & 15) == 0;
    if (vec) return acc ? launch_route<B, true, 8>(r, st) : launch_route<B, false, 8>(r, st);
    return acc ? launch_route<B, true, 1>(r, st) : launch_route<B, false, 1>(r, st);
  }
  if (dtype != DLTI_FP32) return DLTI_ERR_UNSUPPORTED;
  return acc ? launch_route<float, true, 1>(r, st) : launch_route<float, false, 1>(r, st);
}

// The pairs lists[e, 0 .. counts[e]) of every expert; W_e = rows e * wrows ... of W, cap = capacity of a list.
// up: rows X[pair / div] times W_e; out = their activation, one list after the other (1: rows 2 r and 2 r + 1 are gate and up of output r,
// clipped; 2: square of relu). Otherwise: rows of X in that order times W_e, result to out[pair]. X: x_rows rows, out: o_rows rows of `rows` columns.
DLTI_API int dlti_moe_gemm(const void* X, long long x_ld, long long x_rows, int div, const void* Wt, long long w_ld, int wrows, int E,
                           const int* lists, const int* counts, int cap, int rows, int up, int K, float limit, void* out, long long o_ld,
                           int o_rows, int dtype, cudaStream_t st) {
  if (o_rows <= 0 || E <= 0) return 0;
  if (x_rows < 1 || x_rows > 0x7fffffffLL || rows < 1 || K < 1 || div < 1 || up < 0 || up > 2 || rows * (up == MOE_SWIGLU ? 2 : 1) > wrows) return DLTI_ERR_BAD_ARG;
  MoeGemmParams p{lists, counts, E, cap, div, rows, wrows, K, limit, out, o_ld, (int)x_rows, o_rows, 0, 0, 0};
  if (dtype == DLTI_FP32) {
    (up == MOE_SWIGLU ? moe_gemm_f32_kernel<MOE_SWIGLU> : up ? moe_gemm_f32_kernel<MOE_RELU2> : moe_gemm_f32_kernel<MOE_DOWN>)<<<dim3((rows + 63) / 64, E), 256, 0, st>>>((const float*)X, x_ld, (const float*)Wt,
                                                                                                           w_ld, p);
    dlti_count_launch();
    return (int)cudaGetLastError();
  }
  if (dtype != DLTI_BF16) return DLTI_ERR_UNSUPPORTED;
  if (E > 1024) { dlti_set_error("moe_gemm: up to 1024 experts"); return DLTI_ERR_TOO_LARGE; }
  if (o_ld % 8 || o_ld < rows || x_ld % 8 || ((reinterpret_cast<uintptr_t>(X) | reinterpret_cast<uintptr_t>(out)) & 15)) return DLTI_ERR_BAD_ARG;
  const long long avg = (o_rows + E - 1) / E;              // pairs of an expert, were they spread evenly
  p.NT = avg > 96 ? 256 : avg > 40 ? 128 : avg > 12 ? 64 : 32;
  p.MT = (rows * (up == MOE_SWIGLU ? 2 : 1) + 255) / 256;
  const int stage = MG_A_BYTES + p.NT * 64, tail = MG_TAIL + 2048 + 3 * E * 4;
  p.stages = (MG_SMEM - 1024 - tail) / stage;
  if (p.stages > MG_MAX_STAGES) p.stages = MG_MAX_STAGES;
  const int smem = p.stages * stage + tail + 1024;
  CUtensorMap tw, tx;
  int rc;
  if ((rc = dlti_get_tmap(&tw, Wt, K, (uint64_t)E * wrows, w_ld, 64, 128))) return rc;
  if ((rc = dlti_get_tmap(&tx, X, K, x_rows, x_ld, 64, up ? 1 : p.NT / 2))) return rc;
  auto kern = up == MOE_SWIGLU ? moe_gemm_kernel<MOE_SWIGLU> : up ? moe_gemm_kernel<MOE_RELU2> : moe_gemm_kernel<MOE_DOWN>;
  static bool done[64][3] = {};
  int dev = 0;
  DLTI_CUDA_CHECK(cudaGetDevice(&dev));
  if (!done[dev & 63][up]) {
    DLTI_CUDA_CHECK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, MG_SMEM));
    done[dev & 63][up] = true;
  }
  // at most one tile per pair and weight tile
  const long long most = (long long)p.MT * (E < o_rows ? E + (o_rows - E) / p.NT + 1 : o_rows);
  const int clusters = dlti_num_sms() / 2;
  DLTI_CUDA_CHECK(dlti_launch_pdl(cap, kern, dim3(2 * (most < clusters ? (unsigned)most : clusters)),
                                  dim3(MG_THREADS), (size_t)smem, st, p, tw, tx));
  dlti_count_launch();
  return 0;
}
