// Mixtures of experts and gated activations.
//
//   moe_route        one warp per token: sigmoid scores, groups, the top experts and their weights; every (token, choice) pair
//                    = token * top + choice is appended to its expert's list. Further blocks of the same launch apply a gated
//                    activation to other columns of the same projection (the shared expert).
//   moe_gemm         grouped GEMM over the lists, bf16: weights are the 128-row operand of tcgen05.mma and the pairs of a list its
//                    columns (16 to 256 of them), so one kernel serves one decoded token and whole prompts. Source rows come by
//                    TMA gather (four rows a copy), results go to row `pair` of the output. Two accumulators share a tile's
//                    columns: the gate and the up rows, whose activation is the epilogue, or two neighbouring row tiles.
//   moe_gemm_f32     the same in fp32 FMAs
//
// Pair lists are filled with atomics, so their order differs from run to run; a pair's result does not depend on its place.
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
  float* wgt; int *lists, *counts;                         // [T, top]; [E, T]; [E]
  const void* p; long long p_ld; int og, ou, ff; float limit;      // projection columns of the activation (ff 0: none)
  void* h; long long h_ld;
  long long T;
};
constexpr int ROUTE_WARPS = 4;

template <bool ACC>
__device__ void route_token(const RouteParams& p, long long t, float* sc, float* sp, float* sg, int* sel) {
  const int lane = threadIdx.x & 31, n = p.E / p.groups;
  const float* zr = p.z + t * p.z_ld + p.col;
  for (int e = lane; e < p.E; e += 32) {
    float v = zr[e];
    if (ACC) const_cast<float*>(zr)[e] = 0.f;
    v = sigmoid_f(v);
    sp[e] = v;
    sc[e] = v + p.corr[e];
  }
  __syncwarp();
  if (p.keep < p.groups) {
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
    for (int g = lane; g < p.groups; g += 32) {
      int better = 0;
      for (int o = 0; o < p.groups; ++o) better += sg[o] > sg[g] || (sg[o] == sg[g] && o < g);
      if (better >= p.keep)
        for (int e = g * n; e < (g + 1) * n; ++e) sc[e] = -INFINITY;
    }
    __syncwarp();
  }
  float sum = 0.f;
  for (int k = 0; k < p.top; ++k) {
    float best = -INFINITY;
    int bi = p.E;
    for (int e = lane; e < p.E; e += 32)
      if (sc[e] > best) { best = sc[e]; bi = e; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float v = __shfl_xor_sync(0xffffffffu, best, o);
      const int i = __shfl_xor_sync(0xffffffffu, bi, o);
      if (v > best || (v == best && i < bi)) { best = v; bi = i; }
    }
    if (bi >= p.E) bi = k;                                 // only where the scores are not numbers
    if (lane == 0) {
      sel[k] = bi;
      sc[bi] = -INFINITY;
    }
    sum += sp[bi];
    __syncwarp();
  }
  const float f = p.scale / (sum + 1e-20f);
  for (int k = lane; k < p.top; k += 32) {
    const int e = sel[k];
    p.wgt[t * p.top + k] = sp[e] * f;
    const int r = atomicAdd(p.counts + e, 1);
    if (r < p.T) p.lists[e * p.T + r] = (int)(t * p.top + k);
  }
}

template <typename T, bool ACC, int W>
__global__ void __launch_bounds__(32 * ROUTE_WARPS) moe_route_kernel(const RouteParams p, int route_blocks) {
  extern __shared__ float route_s[];
  griddep_wait();
  griddep_launch();
  if ((int)blockIdx.x < route_blocks) {
    const int warp = threadIdx.x >> 5;
    const long long t = (long long)blockIdx.x * ROUTE_WARPS + warp;
    float* s = route_s + warp * (2 * p.E + p.groups + p.top);
    if (t < p.T) route_token<ACC>(p, t, s, s + p.E, s + 2 * p.E, reinterpret_cast<int*>(s + 2 * p.E + p.groups));
    return;
  }
  const int per = p.ff / W;
  const long long total = p.T * per, step = (long long)(gridDim.x - route_blocks) * blockDim.x;
  for (long long i = (long long)(blockIdx.x - route_blocks) * blockDim.x + threadIdx.x; i < total; i += step) {
    const long long t = i / per;
    const int c = (int)(i - t * per) * W;
    const void* row = reinterpret_cast<const uint8_t*>(p.p) + t * p.p_ld * (ACC ? 4 : sizeof(T));
    T* o = reinterpret_cast<T*>(p.h) + t * p.h_ld + c;
    if constexpr (W == 1) {
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
  int rows, wrows, up, K;                                  // output columns; weight rows of an expert; up > 0: row offset of the up part
  float limit;
  void* out; long long o_ld;
  int x_rows, o_rows;                                      // list entries outside these are not followed (counters of an aborted step)
  int NT, MT, stages, accs;                                // columns of a tile (multiple of 32, at most 256), weight tiles of an expert
};
constexpr int MG_THREADS = 320, MG_W_BYTES = 32768, MG_MAX_STAGES = 8;
constexpr long long MG_WAIT_LIMIT = 4000000000LL;

__device__ __forceinline__ void tma_gather4(uint32_t dst, const CUtensorMap* m, uint32_t bar, int c, int r0, int r1, int r2, int r3) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile::gather4.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6, %7}], [%2];" ::"r"(dst),
               "l"(reinterpret_cast<uint64_t>(m)), "r"(bar), "r"(c), "r"(r0), "r"(r1), "r"(r2), "r"(r3)
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
  const int nt = (c + p.NT - 1) / p.NT, per = ((c + nt - 1) / nt + 15) & ~15;
  const int n0 = (r / p.MT) * per;
  return MoeTile{lo, r % p.MT, n0, min(c - n0, per)};
}

// warp 0: copies (lane 0 the weights, every lane its rows), warp 1: MMAs, warps 2-9: epilogue. Waits are bounded: a CTA that gives
// up writes NaN.
__global__ void __launch_bounds__(MG_THREADS, 1) moe_gemm_kernel(const MoeGemmParams p, const __grid_constant__ CUtensorMap tw,
                                                                 const __grid_constant__ CUtensorMap tx) {
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t stage_bytes = MG_W_BYTES + p.NT * 128;
  const uint32_t bars = base + p.stages * stage_bytes;     // full[stages], empty[stages], acc_full[2], acc_empty[2], TMEM address
  const uint32_t full = bars, empty = full + 8 * MG_MAX_STAGES, acc_full = empty + 8 * MG_MAX_STAGES, acc_empty = acc_full + 16, slot = acc_empty + 16;
  uint8_t* tail = smem_raw + (slot - smem_u32(smem_raw)) + 16;
  volatile uint32_t* slot_ptr = reinterpret_cast<volatile uint32_t*>(tail - 16);
  int* s_dst = reinterpret_cast<int*>(tail);               // [2][256]
  int* s_first = s_dst + 512;                              // [E + 1]
  int* s_cnt = s_first + p.E + 1;                          // [E]
  __shared__ int s_scan[32], s_fail;
  const int warp = __shfl_sync(0xffffffffu, threadIdx.x >> 5, 0), lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tw);
    tma_prefetch_desc(&tx);
    s_fail = 0;
    for (int s = 0; s < p.stages; ++s) {
      mbar_init(full + 8 * s, 1);
      mbar_init(empty + 8 * s, 1);
    }
    for (int a = 0; a < 2; ++a) {
      mbar_init(acc_full + 8 * a, 1);
      mbar_init(acc_empty + 8 * a, 8);
    }
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(slot, 512);
    tmem_relinquish();
  }
  griddep_wait();
  griddep_launch();
  // tiles before every expert: a block-wide prefix sum, MG_THREADS experts at a time
  int carry = 0;
  for (int e0 = 0; e0 < p.E; e0 += MG_THREADS) {
    const int e = e0 + threadIdx.x;
    const int c = e < p.E ? min(p.counts[e], p.cap) : 0;
    const int v = (c + p.NT - 1) / p.NT * p.MT;
    int x = v;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int y = __shfl_up_sync(0xffffffffu, x, o);
      if (lane >= o) x += y;
    }
    if (lane == 31) s_scan[warp] = x;
    __syncthreads();
    int before = carry, all = 0;
    for (int w = 0; w < MG_THREADS / 32; ++w) {
      if (w < warp) before += s_scan[w];
      all += s_scan[w];
    }
    if (e < p.E) {
      s_cnt[e] = c;
      s_first[e] = before + x - v;
    }
    carry += all;
    __syncthreads();
  }
  const int total = carry;
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = __shfl_sync(0xffffffffu, *slot_ptr, 0);
  const int nkb = (p.K + 63) / 64, off1 = p.accs == 2 ? 128 : 256;
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

  if (warp == 0) {
    int it = 0;                                            // k blocks so far
    for (int t = blockIdx.x; t < total; t += gridDim.x) {
      const MoeTile x = moe_tile(p, s_first, s_cnt, t);
      if (x.nn <= 0) continue;
      const int groups = (x.nn + 3) >> 2;
      int r[2][4];
#pragma unroll
      for (int y = 0; y < 2; ++y)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int i = min((lane + 32 * y) * 4 + j, x.nn - 1);
          r[y][j] = min((unsigned)p.lists[(long long)x.e * p.cap + x.n0 + i] / p.div, (unsigned)p.x_rows - 1);
        }
      const int w0 = x.e * p.wrows + x.m * (p.up ? 128 : 256), w1 = w0 + (p.up ? p.up : 128);
      for (int kb = 0; kb < nkb; ++kb, ++it) {
        const int s = it % p.stages;
        if (it >= p.stages && !wait(empty + 8 * s, (it / p.stages - 1) & 1)) break;
        const uint32_t dst = base + s * stage_bytes, bar = full + 8 * s;
        if (lane == 0) {
          mbar_expect_tx(bar, MG_W_BYTES + groups * 512);
          tma_load_2d(dst, &tw, bar, kb * 64, w0);
          tma_load_2d(dst + 16384, &tw, bar, kb * 64, w1);
        }
        __syncwarp();
#pragma unroll
        for (int y = 0; y < 2; ++y)
          if (lane + 32 * y < groups)
            tma_gather4(dst + MG_W_BYTES + (lane + 32 * y) * 512, &tx, bar, kb * 64, r[y][0], r[y][1], r[y][2], r[y][3]);
      }
      if (*fail) break;
    }
  } else if (warp == 1) {
    const bool leader = elect_one_sync();
    int it = 0, tile = 0;
    for (int t = blockIdx.x; t < total; t += gridDim.x) {
      const MoeTile x = moe_tile(p, s_first, s_cnt, t);
      if (x.nn <= 0) continue;
      const int a = p.accs == 2 ? tile & 1 : 0, use = p.accs == 2 ? tile >> 1 : tile;
      if (use > 0 && !wait(acc_empty + 8 * a, (use - 1) & 1)) break;
      tc_fence_after();
      const uint32_t idesc = umma_idesc_f16(DLTI_BF16, 128, (x.nn + 15) & ~15, false, false);
      const uint32_t d0 = tmem + a * 256, d1 = d0 + off1;
      for (int kb = 0; kb < nkb; ++kb, ++it) {
        const int s = it % p.stages;
        if (!wait(full + 8 * s, (it / p.stages) & 1)) break;
        tc_fence_after();
        const uint32_t sm = base + s * stage_bytes;
        const DescLoHi da = desc_split(sm, 0, 1024), dc = desc_split(sm + 16384, 0, 1024), db = desc_split(sm + MG_W_BYTES, 0, 1024);
        if (leader) {
#pragma unroll
          for (int kk = 0; kk < 4; ++kk) umma_f16_ss(d0, da.at(kk * 32), db.at(kk * 32), idesc, kb > 0 || kk > 0);
#pragma unroll
          for (int kk = 0; kk < 4; ++kk) umma_f16_ss(d1, dc.at(kk * 32), db.at(kk * 32), idesc, kb > 0 || kk > 0);
          umma_commit(empty + 8 * s);
        }
        __syncwarp();
      }
      if (*fail) break;
      if (leader) umma_commit(acc_full + 8 * a);
      __syncwarp();
      ++tile;
    }
  } else {
    const int quarter = warp & 3, half = (warp - 2) >> 2;
    int tile = 0;
    for (int t = blockIdx.x; t < total; t += gridDim.x) {
      const MoeTile x = moe_tile(p, s_first, s_cnt, t);
      if (x.nn <= 0) continue;
      const int a = p.accs == 2 ? tile & 1 : 0, use = p.accs == 2 ? tile >> 1 : tile;
      int* dst = s_dst + (tile & 1) * 256;
      const int i0 = threadIdx.x - 64;
      if (i0 < x.nn) dst[i0] = p.lists[(long long)x.e * p.cap + x.n0 + i0];
      asm volatile("bar.sync 1, 256;" ::: "memory");
      const bool ok = wait(acc_full + 8 * a, use & 1);
      tc_fence_after();
      const uint32_t d0 = tmem + ((uint32_t)(quarter * 32) << 16) + a * 256;
      const int row0 = x.m * (p.up ? 128 : 256) + quarter * 32 + lane;
      __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + row0;
      const bool ok0 = row0 < p.rows, ok1 = row0 + 128 < p.rows;
      for (int c = half * 16; c < x.nn; c += 32) {
        uint32_t g[16], u[16];
        if (ok) {
          tmem_ld_32x32b_x16(d0 + c, g);
          tmem_ld_32x32b_x16(d0 + off1 + c, u);
          tmem_wait_ld();
        } else {
#pragma unroll
          for (int j = 0; j < 16; ++j) g[j] = u[j] = 0x7fffffffu;
        }
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          if (c + j >= x.nn) break;
          if ((unsigned)dst[c + j] >= (unsigned)p.o_rows) continue;
          __nv_bfloat16* o = out + (long long)dst[c + j] * p.o_ld;
          const float fg = __uint_as_float(g[j]), fu = __uint_as_float(u[j]);
          if (p.up) {
            if (ok0) *o = __float2bfloat16(gated_fast(fg, fu, p.limit));
          } else {
            if (ok0) *o = __float2bfloat16(fg);
            if (ok1) o[128] = __float2bfloat16(fu);
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(acc_empty + 8 * a);
      ++tile;
    }
  }
  if (*fail) {                                             // copies may still be in flight: leave their shared memory alone for a while
    const long long t0 = clock64();
    while (clock64() - t0 < 20000000LL) {
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// CTA = (64 weight rows, expert), 16 pairs at a time; thread = one row of 4 pairs
__global__ void __launch_bounds__(256) moe_gemm_f32_kernel(const float* __restrict__ X, long long x_ld, const float* __restrict__ Wt, long long w_ld,
                                                           const MoeGemmParams p) {
  __shared__ float sw[2][16][65], sx[16][17];
  __shared__ int s_pair[16];
  const int e = blockIdx.y, r0 = blockIdx.x * 64, cnt = min(p.counts[e], p.cap);
  const int r = threadIdx.x & 63, tg = threadIdx.x >> 6;
  const int parts = p.up ? 2 : 1;
  for (int n0 = 0; n0 < cnt; n0 += 16) {
    __syncthreads();
    if (threadIdx.x < 16) s_pair[threadIdx.x] = p.lists[(long long)e * p.cap + min(n0 + (int)threadIdx.x, cnt - 1)];
    __syncthreads();
    float acc[2][4] = {};
    for (int k0 = 0; k0 < p.K; k0 += 16) {
      for (int i = threadIdx.x; i < parts * 64 * 16; i += 256) {
        const int q = i / (64 * 16), rr = (i / 16) % 64, k = i % 16;
        sw[q][k][rr] = (r0 + rr < p.rows && k0 + k < p.K) ? Wt[((long long)e * p.wrows + q * p.up + r0 + rr) * w_ld + k0 + k] : 0.f;
      }
      {
        const int i = threadIdx.x, tt = i / 16, k = i % 16;
        const unsigned src = min((unsigned)s_pair[tt] / p.div, (unsigned)p.x_rows - 1);
        sx[tt][k] = k0 + k < p.K ? X[(long long)src * x_ld + k0 + k] : 0.f;
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
      if (n0 + i < cnt && r0 + r < p.rows && (unsigned)s_pair[i] < (unsigned)p.o_rows)
        reinterpret_cast<float*>(p.out)[(long long)s_pair[i] * p.o_ld + r0 + r] = p.up ? gated(acc[0][j], acc[1][j], p.limit) : acc[0][j];
    }
  }
}

template <typename T, bool ACC, int W>
int launch_route(const RouteParams& p, cudaStream_t st) {
  const int rb = p.E ? (int)((p.T + ROUTE_WARPS - 1) / ROUTE_WARPS) : 0;
  const int ab = p.ff ? grid_for(p.T * (p.ff / W), 32 * ROUTE_WARPS) : 0;
  const size_t smem = p.E ? (size_t)ROUTE_WARPS * (2 * p.E + p.groups + p.top) * 4 : 0;
  DLTI_CUDA_CHECK(dlti_launch_pdl(p.T, moe_route_kernel<T, ACC, W>, dim3(rb + ab), dim3(32 * ROUTE_WARPS), smem, st, p, rb));
  dlti_count_launch();
  return 0;
}

}  // namespace

// experts 0: no routing; ff 0: no activation. acc: z and p are the decode GEMM's accumulator (zero on return in the columns read).
DLTI_API int dlti_moe_route(const float* z, long long z_ld, int col, const float* corr, int E, int top, int groups, int keep, float scale,
                            float* wgt, int* lists, int* counts, const void* p, long long p_ld, int og, int ou, int ff, float limit, void* h,
                            long long h_ld, long long T, int acc, int dtype, cudaStream_t st) {
  if (T <= 0) return 0;
  if (E && (!z || !corr || !wgt || !lists || !counts || groups < 1 || E % groups || keep < 1 || keep > groups || top < 1 || top > E / groups * keep))
    return DLTI_ERR_BAD_ARG;
  if (E > 1024 || T * (top > 1 ? top : 1) > 0x7fffffffLL) { dlti_set_error("moe_route: up to 1024 experts"); return DLTI_ERR_TOO_LARGE; }
  if (ff && (!p || !h)) return DLTI_ERR_BAD_ARG;
  if (!E && !ff) return 0;
  const RouteParams r{z, z_ld, col, corr, E, top, groups, keep, scale, wgt, lists, counts, p, p_ld, og, ou, ff, limit, h, h_ld, T};
  using B = __nv_bfloat16;
  if (dtype == DLTI_BF16) {
    const bool vec = ((ff | og | ou) & 7) == 0 && ((p_ld | h_ld) & 7) == 0 && ((reinterpret_cast<uintptr_t>(p) | reinterpret_cast<uintptr_t>(h)) & 15) == 0;
    if (vec) return acc ? launch_route<B, true, 8>(r, st) : launch_route<B, false, 8>(r, st);
    return acc ? launch_route<B, true, 1>(r, st) : launch_route<B, false, 1>(r, st);
  }
  if (dtype != DLTI_FP32) return DLTI_ERR_UNSUPPORTED;
  return acc ? launch_route<float, true, 1>(r, st) : launch_route<float, false, 1>(r, st);
}

// out[pair, 0 .. rows) = X[pair / div] · W_e^T over the pairs lists[e, 0 .. counts[e]) of every expert; W_e = rows e * wrows ... of W.
// up > 0: gate rows first, up rows `up` further on, out = clipped activation. X: x_rows rows, out: o_rows rows. cap: capacity of a list.
DLTI_API int dlti_moe_gemm(const void* X, long long x_ld, long long x_rows, int div, const void* Wt, long long w_ld, int wrows, int E,
                           const int* lists, const int* counts, int cap, int rows, int up, int K, float limit, void* out, long long o_ld,
                           int o_rows, int dtype, cudaStream_t st) {
  if (o_rows <= 0 || E <= 0) return 0;
  if (x_rows < 1 || x_rows > 0x7fffffffLL || rows < 1 || K < 1 || div < 1 || (up && up < rows) || (up ? up : 0) + rows > wrows) return DLTI_ERR_BAD_ARG;
  MoeGemmParams p{lists, counts, E, cap, div, rows, wrows, up, K, limit, out, o_ld, (int)x_rows, o_rows, 0, 0, 0, 0};
  if (dtype == DLTI_FP32) {
    moe_gemm_f32_kernel<<<dim3((rows + 63) / 64, E), 256, 0, st>>>((const float*)X, x_ld, (const float*)Wt, w_ld, p);
    dlti_count_launch();
    return (int)cudaGetLastError();
  }
  if (dtype != DLTI_BF16) return DLTI_ERR_UNSUPPORTED;
  if (E > 1024) { dlti_set_error("moe_gemm: up to 1024 experts"); return DLTI_ERR_TOO_LARGE; }
  const long long avg = (o_rows + E - 1) / E;              // pairs of an expert, were they spread evenly
  p.NT = avg > 96 ? 256 : avg > 40 ? 128 : avg > 12 ? 64 : 32;
  const int tile_rows = up ? 128 : 256;
  p.MT = (rows + tile_rows - 1) / tile_rows;
  p.accs = p.NT <= 128 ? 2 : 1;
  const int stage = MG_W_BYTES + p.NT * 128, tail = 16 * MG_MAX_STAGES + 48 + 2048 + (2 * E + 1) * 4 + 16;
  p.stages = (226 * 1024 - 1024 - tail) / stage;
  if (p.stages > MG_MAX_STAGES) p.stages = MG_MAX_STAGES;
  const int smem = p.stages * stage + tail + 1024;
  CUtensorMap tw, tx;
  int rc;
  if ((rc = dlti_get_tmap(&tw, Wt, K, (uint64_t)E * wrows, w_ld, 64, 128))) return rc;
  if ((rc = dlti_get_tmap(&tx, X, K, x_rows, x_ld, 64, 1))) return rc;
  static bool done[64] = {};
  int dev = 0;
  DLTI_CUDA_CHECK(cudaGetDevice(&dev));
  if (!done[dev & 63]) {
    DLTI_CUDA_CHECK(cudaFuncSetAttribute(moe_gemm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024));
    done[dev & 63] = true;
  }
  // at most one tile per pair and weight tile
  const long long most = (long long)p.MT * (E < o_rows ? E + (o_rows - E) / p.NT + 1 : o_rows);
  const int sms = dlti_num_sms();
  DLTI_CUDA_CHECK(dlti_launch_pdl(cap, moe_gemm_kernel, dim3(most < sms ? (unsigned)most : sms), dim3(MG_THREADS), (size_t)smem, st, p, tw, tx));
  dlti_count_launch();
  return 0;
}
