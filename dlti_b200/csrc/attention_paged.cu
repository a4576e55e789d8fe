// Attention over the paged cache for the layer-stack models: any head size, grouped key/value heads, causal, chunked
// (position i sees keys of its own chunk of `chunk` positions only) or windowed (itself and the window - 1 positions before
// it), optional soft cap on the scores, bias by distance, per-head sink, gates on head outputs or on every output element.
//
//   attn_prefill_kernel  portions of prompts, bf16: a CTA owns 128 (token, head of a group) rows and streams key / value
//                        tiles of 64 from the pages through shared memory into mma.sync
//   attn_decode_kernel   one new token per sequence, bf16: the query heads of a group share every key and value (rows of
//                        one m16 fragment), keys are split over CTAs and the splits combined by attn_combine_kernel
//   attn_rows_kernel     one warp per (row, head), fp32 arithmetic throughout: the fp32 mode, and heads above 256
//
// Scores, softmax weights and sums are fp32. The weights enter the P*V product as two bf16 terms (hi + lo, 16 mantissa
// bits), so the product is that of the fp32 weights with the bf16 values.
#include "mma_sync.cuh"
#include "rows.cuh"

namespace {

struct PagedParams {
  const void* q; long long q_ld; int q_hd;         // queries: row pitch, head pitch
  const void *kc, *vc; int kd, vd;                 // cache row pitches of a head
  const int* tables; int max_blocks; int bs;
  const int *ctx, *cu, *rseq, *pos; int nd;
  int H, G, dim, vdim, chunk, window;
  float scale, cap;                                // cap > 0: scores become cap tanh(score / cap)
  const float* gate;                               // [rows, H] factors or null
  void* out; long long o_ld;                       // head h at column h * vdim
  long long rows;
  const float* sink;                               // [H] or null: one more term exp(sink) in the softmax denominator, without a value
  const float* bias; int span;                     // [H, span] or null: added to the scores at the distances 0 ... span - 1
  const void* ogate; long long og_ld;              // [rows, H * vdim] or null: outputs times sigmoid of it
};
// factor of output element c of head h
template <typename T>
__device__ __forceinline__ float gate_at(const PagedParams& p, long long row, int h, int c) {
  if (!p.ogate) return 1.f;
  const float z = Cvt<T>::to_f(reinterpret_cast<const T*>(p.ogate)[row * p.og_ld + (long long)h * p.vdim + c]);
  return sizeof(T) == 4 ? sigmoid_f(z) : fast_sigmoid(z);
}

// softmax denominator of head h with its sink: l is a sum of 2^(score - m), m in log2 (natural: of e^(score - m))
__device__ __forceinline__ float with_sink(const PagedParams& p, int h, float m, float l, bool natural = false) {
  if (!p.sink) return l;
  const float r = m == -INFINITY ? 0.f : m;
  return l + (natural ? expf(p.sink[h] - r) : ex2(p.sink[h] * 1.4426950408889634f - r));
}
__device__ __forceinline__ int first_key(const PagedParams& p, int pos) {
  return p.chunk > 0 ? pos / p.chunk * p.chunk : p.window > 0 ? max(0, pos - p.window + 1) : 0;
}
// a product q . k as the score in log2 units
__device__ __forceinline__ float score_log2(const PagedParams& p, float s, float sl2) {
  return p.cap > 0.f ? capped_log2(s, p.scale, p.cap) : s * sl2;
}

// ROWS_MAXV: value dims per lane
template <typename T, int ROWS_MAXV>
__global__ void __launch_bounds__(128) attn_rows_kernel(const PagedParams p) {
  extern __shared__ float sq_all[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* sq = sq_all + warp * p.dim;
  const long long w = (long long)blockIdx.x * 4 + warp;
  if (w >= p.rows * p.H) return;
  const long long t = w / p.H;
  const int h = (int)(w - t * p.H), g = h / (p.H / p.G);
  const int seq = p.rseq[t], ps = p.pos[t];
  const int nkeys = min(ps + 1, p.ctx[seq]);       // padding rows of a decode graph have no keys
  const int* tab = p.tables + (long long)seq * p.max_blocks;
  const T* qr = reinterpret_cast<const T*>(p.q) + t * p.q_ld + (long long)h * p.q_hd;
  for (int c = lane; c < p.dim; c += 32) sq[c] = Cvt<T>::to_f(qr[c]);
  __syncwarp();
  float m = -INFINITY, l = 0.f, o[ROWS_MAXV];
#pragma unroll
  for (int i = 0; i < ROWS_MAXV; ++i) o[i] = 0.f;
  for (int j0 = first_key(p, ps); j0 < nkeys; j0 += 32) {
    const int j = j0 + lane;
    float s = -INFINITY;
    long long slot = 0;
    if (j < nkeys) {
      slot = (long long)tab[j / p.bs] * p.bs + j % p.bs;
      const T* kr = reinterpret_cast<const T*>(p.kc) + (slot * p.G + g) * p.kd;
      float a = 0.f;
      for (int c0 = 0; c0 < p.dim; c0 += 16) {             // short partial sums keep the rounding error small
        float b = 0.f;
        for (int c = c0; c < min(p.dim, c0 + 16); ++c) b = fmaf(sq[c], Cvt<T>::to_f(kr[c]), b);
        a += b;
      }
      s = a * p.scale;
      if (p.cap > 0.f) s = p.cap * tanhf(s / p.cap);
      if (p.bias && ps - j < p.span) s += p.bias[(long long)h * p.span + ps - j];
    }
    const float nm = fmaxf(m, warp_max(s));
    const float alpha = expf(m - nm);
    const float pj = expf(s - nm);
    l = l * alpha + warp_sum(pj);
    m = nm;
#pragma unroll
    for (int i = 0; i < ROWS_MAXV; ++i) o[i] *= alpha;
    const int nj = min(32, nkeys - j0);
    for (int jj = 0; jj < nj; ++jj) {
      const float pp = __shfl_sync(0xffffffffu, pj, jj);
      const long long sl = __shfl_sync(0xffffffffu, slot, jj);
      const T* vr = reinterpret_cast<const T*>(p.vc) + (sl * p.G + g) * p.vd;
#pragma unroll
      for (int i = 0; i < ROWS_MAXV; ++i) {
        const int c = lane + 32 * i;
        if (c < p.vdim) o[i] = fmaf(pp, Cvt<T>::to_f(vr[c]), o[i]);
      }
    }
  }
  l = with_sink(p, h, m, l, true);
  float f = l > 0.f ? 1.f / l : 0.f;
  if (p.gate) f *= p.gate[t * p.H + h];
  T* orow = reinterpret_cast<T*>(p.out) + t * p.o_ld + (long long)h * p.vdim;
#pragma unroll
  for (int i = 0; i < ROWS_MAXV; ++i) {
    const int c = lane + 32 * i;
    if (c < p.vdim) orow[c] = Cvt<T>::from_f(o[i] * f * gate_at<T>(p, t, h, c));
  }
}

template <typename T>
int launch_rows(const PagedParams& p, cudaStream_t st) {
  const size_t smem = (size_t)4 * p.dim * 4;
  (p.vdim <= 256 ? attn_rows_kernel<T, 8> : attn_rows_kernel<T, 32>)<<<(unsigned)((p.rows * p.H + 3) / 4), 128, smem, st>>>(p);
  dlti_count_launch();
  return (int)cudaGetLastError();
}

using bf16 = __nv_bfloat16;
constexpr int KT = 64;                             // keys per tile
constexpr float LOG2E_F = 1.4426950408889634f;

template <int DK, int DV>
struct Tile {                                      // one stage: K [64][DK + 8] then V [64][DV + 8]; +8 keeps ldmatrix free of conflicts
  static constexpr int KP = DK + 8, VP = DV + 8;
  static constexpr int K_BYTES = KT * KP * 2, BYTES = K_BYTES + KT * VP * 2;
};

// zero the padding columns [kd, DK) and [vd, DV) of both stages: the copies never write them
template <int DK, int DV>
__device__ __forceinline__ void zero_pads(uint8_t* smem, int kd, int vd) {
  using L = Tile<DK, DV>;
  for (int st = 0; st < 2; ++st) {
    bf16* k = reinterpret_cast<bf16*>(smem + st * L::BYTES);
    bf16* v = reinterpret_cast<bf16*>(smem + st * L::BYTES + L::K_BYTES);
    if (kd < DK)
      for (int i = threadIdx.x; i < KT * (DK - kd); i += blockDim.x) k[(i / (DK - kd)) * L::KP + kd + i % (DK - kd)] = __float2bfloat16(0.f);
    if (vd < DV)
      for (int i = threadIdx.x; i < KT * (DV - vd); i += blockDim.x) v[(i / (DV - vd)) * L::VP + vd + i % (DV - vd)] = __float2bfloat16(0.f);
  }
}
// A thread's first 16-byte piece of a tile's keys / values and its step to the next one: no divisions in the loops
struct Walk {
  int kn, kr, kc, kdr, kdc, vn, vr, vc, vdr, vdc;
  __device__ __forceinline__ explicit Walk(const PagedParams& p) {
    const int t = threadIdx.x, n = blockDim.x;
    kn = p.kd >> 3; kr = t / kn; kc = t % kn; kdr = n / kn; kdc = n % kn;
    vn = p.vd >> 3; vr = t / vn; vc = t % vn; vdr = n / vn; vdc = n % vn;
  }
};
// cp.async of keys and values [j0, j0 + 64) of one head of the sequence; rows at or past jend become zeros
template <int DK, int DV>
__device__ __forceinline__ void load_tile(uint32_t stage, const PagedParams& p, const Walk& w, const int* slots, int g, int j0, int jend) {
  using L = Tile<DK, DV>;
  const bf16* K = reinterpret_cast<const bf16*>(p.kc) + g * p.kd;
  const bf16* V = reinterpret_cast<const bf16*>(p.vc) + g * p.vd;
  const int ks = p.G * p.kd, vs = p.G * p.vd;
  for (int r = w.kr, c = w.kc; r < KT;) {
    cp_async16(stage + (r * L::KP + c * 8) * 2, K + (long long)slots[r] * ks + c * 8, j0 + r < jend);
    r += w.kdr;
    c += w.kdc;
    if (c >= w.kn) { c -= w.kn; ++r; }
  }
  for (int r = w.vr, c = w.vc; r < KT;) {
    cp_async16(stage + L::K_BYTES + (r * L::VP + c * 8) * 2, V + (long long)slots[r] * vs + c * 8, j0 + r < jend);
    r += w.vdr;
    c += w.vdc;
    if (c >= w.vn) { c -= w.vn; ++r; }
  }
  cp_async_commit();
}
__device__ __forceinline__ void tile_slots(int* slots, const PagedParams& p, const int* tab, int j0, int jend) {
  if (threadIdx.x < KT) {
    const int j = min(j0 + (int)threadIdx.x, jend - 1);
    const int b = (p.bs & (p.bs - 1)) ? j / p.bs : j >> (31 - __clz(p.bs));
    slots[threadIdx.x] = tab[b] * p.bs + j - b * p.bs;
  }
}
// this thread's elements of query rows as A fragments; q0 / q1: rows lane / 4 and lane / 4 + 8 (null: zeros)
template <int DK>
__device__ __forceinline__ void load_q(uint32_t (&qf)[DK / 16][4], const bf16* q0, const bf16* q1, int dim) {
  const int c0 = (threadIdx.x & 3) * 2;
#pragma unroll
  for (int kk = 0; kk < DK / 16; ++kk)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const bf16* q = (x & 1) ? q1 : q0;
      const int c = kk * 16 + c0 + (x >> 1) * 8;
      uint32_t v = 0;
      if (q && c + 1 < dim) v = *reinterpret_cast<const uint32_t*>(q + c);
      else if (q && c < dim) v = *reinterpret_cast<const uint16_t*>(q + c);
      qf[kk][x] = v;
    }
}
// S[16 x 16 keys] of keys kt .. kt + 15 of the tile
template <int DK>
__device__ __forceinline__ void scores16(float (&s0)[4], float (&s1)[4], const uint32_t (&qf)[DK / 16][4], uint32_t k_base, int kt) {
  const int lane = threadIdx.x & 31;
  const uint32_t addr = k_base + ((kt + (lane & 7) + ((lane >> 4) << 3)) * (DK + 8) + ((lane >> 3) & 1) * 8) * 2;
#pragma unroll
  for (int kk = 0; kk < DK / 16; ++kk) {
    uint32_t b[4];
    ldsm4(b, addr + kk * 32);
    mma_bf16(s0, qf[kk], b[0], b[1]);
    mma_bf16(s1, qf[kk], b[2], b[3]);
  }
}
// O += P[16 x 16 keys] V, the weights as hi + lo
template <int DV>
__device__ __forceinline__ void weighted16(float (&o)[DV / 8][4], const float (&p0)[4], const float (&p1)[4], uint32_t v_base, int kt) {
  const int lane = threadIdx.x & 31;
  uint32_t hi[4], lo[4];
  split_pair(p0[0], p0[1], hi[0], lo[0]);
  split_pair(p0[2], p0[3], hi[1], lo[1]);
  split_pair(p1[0], p1[1], hi[2], lo[2]);
  split_pair(p1[2], p1[3], hi[3], lo[3]);
  const uint32_t addr = v_base + ((kt + (lane & 15)) * (DV + 8) + (lane >> 4) * 8) * 2;
#pragma unroll
  for (int d = 0; d < DV / 16; ++d) {
    uint32_t b[4];
    ldsm4_t(b, addr + d * 32);
    mma_bf16(o[2 * d], hi, b[0], b[1]);
    mma_bf16(o[2 * d], lo, b[0], b[1]);
    mma_bf16(o[2 * d + 1], hi, b[2], b[3]);
    mma_bf16(o[2 * d + 1], lo, b[2], b[3]);
  }
}

constexpr int PF_ROWS = 128;                       // (token, head) rows of a prefill CTA
template <int DK, int DV, bool EXTRA>              // EXTRA: biases by distance and / or gates on output elements
__global__ void __launch_bounds__(256) attn_prefill_kernel(const PagedParams p) {
  using L = Tile<DK, DV>;
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ int s_slots[2][KT];
  const int seq = p.nd + blockIdx.z, g = blockIdx.y, rep = p.H / p.G;
  const int n = p.cu[blockIdx.z + 1] - p.cu[blockIdx.z];
  const long long row0 = p.nd + p.cu[blockIdx.z];
  const int start = p.ctx[seq] - n;
  const long long total = (long long)n * rep;
  // late tiles first: they see the most keys
  const long long tile = (total + PF_ROWS - 1) / PF_ROWS - 1 - blockIdx.x;
  if (tile < 0) return;
  const long long r_first = tile * PF_ROWS, r_last = min(total, r_first + PF_ROWS) - 1;
  const int jbeg = first_key(p, start + (int)(r_first / rep)), jend = start + (int)(r_last / rep) + 1;
  const int* tab = p.tables + (long long)seq * p.max_blocks;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  int pos[2], jlo[2], head[2];
  long long row[2];
  const bf16* qp[2];
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const long long r = r_first + warp * 16 + (lane >> 2) + 8 * x;
    const bool ok = r < total;
    const int i = ok ? (int)(r / rep) : 0;
    head[x] = g * rep + (int)(r % rep);
    row[x] = row0 + i;
    pos[x] = ok ? start + i : -1;
    jlo[x] = ok ? first_key(p, pos[x]) : 0;
    qp[x] = ok ? reinterpret_cast<const bf16*>(p.q) + row[x] * p.q_ld + (long long)head[x] * p.q_hd : nullptr;
  }
  // key range of this warp's 16 rows
  const long long wr0 = r_first + warp * 16, wr1 = min(total, wr0 + 16) - 1;
  const bool warp_on = wr0 < total;
  const int wlo = warp_on ? first_key(p, start + (int)(wr0 / rep)) : 0, whi = warp_on ? start + (int)(wr1 / rep) : -1;

  uint32_t qf[DK / 16][4];
  load_q<DK>(qf, qp[0], qp[1], p.dim);
  float o[DV / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
#pragma unroll
    for (int x = 0; x < 4; ++x) o[i][x] = 0.f;
  const float sl2 = p.scale * LOG2E_F;
  const uint32_t sbase = smem_u32(smem);
  const Walk walk(p);
  zero_pads<DK, DV>(smem, p.kd, p.vd);
  tile_slots(s_slots[0], p, tab, jbeg, jend);
  __syncthreads();
  load_tile<DK, DV>(sbase, p, walk, s_slots[0], g, jbeg, jend);
  int it = 0;
  for (int j0 = jbeg; j0 < jend; j0 += KT, ++it) {
    const bool more = j0 + KT < jend;
    if (more) tile_slots(s_slots[(it + 1) & 1], p, tab, j0 + KT, jend);
    __syncthreads();                               // the other stage is free, its slots are written
    if (more) {
      load_tile<DK, DV>(sbase + ((it + 1) & 1) * L::BYTES, p, walk, s_slots[(it + 1) & 1], g, j0 + KT, jend);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    if (j0 > whi || j0 + KT <= wlo) continue;      // nothing here for this warp (barriers above are CTA-wide)
    const uint32_t kb = sbase + (it & 1) * L::BYTES, vb = kb + L::K_BYTES;
    float s[KT / 8][4];
#pragma unroll
    for (int i = 0; i < KT / 8; ++i)
#pragma unroll
      for (int x = 0; x < 4; ++x) s[i][x] = 0.f;
#pragma unroll
    for (int i = 0; i < KT / 16; ++i) scores16<DK>(s[2 * i], s[2 * i + 1], qf, kb, i * 16);
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int i = 0; i < KT / 8; ++i)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const int j = j0 + i * 8 + (lane & 3) * 2 + (x & 1), y = x >> 1;
        s[i][x] = (j <= pos[y] && j >= jlo[y]) ? score_log2(p, s[i][x], sl2) : -INFINITY;
        if (!EXTRA) mx[y] = fmaxf(mx[y], s[i][x]);
      }
    if constexpr (EXTRA) {
      if (p.bias && start + (int)(wr0 / rep) - (j0 + KT - 1) < p.span) {
        const float* tab[2] = {p.bias + (long long)head[0] * p.span, p.bias + (long long)head[1] * p.span};
#pragma unroll
        for (int i = 0; i < KT / 8; ++i)
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const int n = pos[x >> 1] - (j0 + i * 8 + (lane & 3) * 2 + (x & 1));
            if ((unsigned)n < (unsigned)p.span) s[i][x] = fmaf(LOG2E_F, tab[x >> 1][n], s[i][x]);
          }
      }
#pragma unroll
      for (int i = 0; i < KT / 8; ++i)
#pragma unroll
        for (int x = 0; x < 4; ++x) mx[x >> 1] = fmaxf(mx[x >> 1], s[i][x]);
    }
    float base[2];
#pragma unroll
    for (int y = 0; y < 2; ++y) {
      mx[y] = fmaxf(mx[y], __shfl_xor_sync(0xffffffffu, mx[y], 1));
      mx[y] = fmaxf(mx[y], __shfl_xor_sync(0xffffffffu, mx[y], 2));
      const float nm = fmaxf(m[y], mx[y]);
      base[y] = nm == -INFINITY ? 0.f : nm;
      const float alpha = ex2(m[y] - base[y]);
      m[y] = nm;
      l[y] *= alpha;
#pragma unroll
      for (int i = 0; i < DV / 8; ++i) {
        o[i][2 * y] *= alpha;
        o[i][2 * y + 1] *= alpha;
      }
    }
#pragma unroll
    for (int i = 0; i < KT / 8; ++i)
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        s[i][x] = ex2(s[i][x] - base[x >> 1]);
        l[x >> 1] += s[i][x];
      }
#pragma unroll
    for (int i = 0; i < KT / 16; ++i) weighted16<DV>(o, s[2 * i], s[2 * i + 1], vb, i * 16);
  }
#pragma unroll
  for (int y = 0; y < 2; ++y) {
    l[y] += __shfl_xor_sync(0xffffffffu, l[y], 1);
    l[y] += __shfl_xor_sync(0xffffffffu, l[y], 2);
    if (pos[y] < 0) continue;
    l[y] = with_sink(p, head[y], m[y], l[y]);
    float f = l[y] > 0.f ? 1.f / l[y] : 0.f;
    if (p.gate) f *= p.gate[row[y] * p.H + head[y]];
    bf16* orow = reinterpret_cast<bf16*>(p.out) + row[y] * p.o_ld + (long long)head[y] * p.vdim;
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) {
      const int c = i * 8 + (lane & 3) * 2;
      if (EXTRA && p.ogate) {
        if (c < p.vdim) o[i][2 * y] *= gate_at<bf16>(p, row[y], head[y], c);
        if (c + 1 < p.vdim) o[i][2 * y + 1] *= gate_at<bf16>(p, row[y], head[y], c + 1);
      }
      if (c + 1 < p.vdim && (p.vdim & 1) == 0) {
        *reinterpret_cast<__nv_bfloat162*>(orow + c) = __floats2bfloat162_rn(o[i][2 * y] * f, o[i][2 * y + 1] * f);
      } else {
        if (c < p.vdim) orow[c] = __float2bfloat16(o[i][2 * y] * f);
        if (c + 1 < p.vdim) orow[c + 1] = __float2bfloat16(o[i][2 * y + 1] * f);
      }
    }
  }
}

// grid (splits, G * head blocks of 16, sequences), 4 warps; warp w takes keys 16 w .. 16 w + 15 of every tile.
template <int DK, int DV>
__global__ void __launch_bounds__(128) attn_decode_kernel(const PagedParams p, int splits, float* __restrict__ part_o,
                                                         float* __restrict__ part_ml) {
  using L = Tile<DK, DV>;
  extern __shared__ __align__(128) uint8_t smem[];
  __shared__ int s_slots[2][KT];
  __shared__ float s_m[4][16], s_l[4][16];
  griddep_wait();
  griddep_launch();
  const int rep = p.H / p.G, hblocks = (rep + 15) / 16;
  const int split = blockIdx.x, b = blockIdx.z, g = blockIdx.y / hblocks, h0 = (blockIdx.y % hblocks) * 16;
  const int nh = min(16, rep - h0);
  const int ctx = p.ctx[b];
  const int kbeg = ctx > 0 ? first_key(p, ctx - 1) : 0;
  const int tiles = (ctx - kbeg + KT - 1) / KT, per = (tiles + splits - 1) / splits;
  const int jbeg = kbeg + split * per * KT, jend = min(ctx, jbeg + per * KT);
  const int* tab = p.tables + (long long)b * p.max_blocks;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float o[DV / 8][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
#pragma unroll
    for (int x = 0; x < 4; ++x) o[i][x] = 0.f;
  const uint32_t sbase = smem_u32(smem);
  if (jbeg < jend) {
    const Walk walk(p);
    zero_pads<DK, DV>(smem, p.kd, p.vd);
    tile_slots(s_slots[0], p, tab, jbeg, jend);
    __syncthreads();
    load_tile<DK, DV>(sbase, p, walk, s_slots[0], g, jbeg, jend);
    uint32_t qf[DK / 16][4];
    const bf16* q = reinterpret_cast<const bf16*>(p.q) + (long long)b * p.q_ld + (long long)(g * rep + h0) * p.q_hd;
    const int r0 = lane >> 2, r1 = r0 + 8;
    load_q<DK>(qf, r0 < nh ? q + (long long)r0 * p.q_hd : nullptr, r1 < nh ? q + (long long)r1 * p.q_hd : nullptr, p.dim);
    const float sl2 = p.scale * LOG2E_F;
    int it = 0;
    for (int j0 = jbeg; j0 < jend; j0 += KT, ++it) {
      const bool more = j0 + KT < jend;
      if (more) tile_slots(s_slots[(it + 1) & 1], p, tab, j0 + KT, jend);
      __syncthreads();
      if (more) {
        load_tile<DK, DV>(sbase + ((it + 1) & 1) * L::BYTES, p, walk, s_slots[(it + 1) & 1], g, j0 + KT, jend);
        cp_async_wait<1>();
      } else {
        cp_async_wait<0>();
      }
      __syncthreads();
      if (j0 + warp * 16 >= jend) continue;
      const uint32_t kb = sbase + (it & 1) * L::BYTES, vb = kb + L::K_BYTES;
      float s[2][4] = {};
      const bool near = p.bias && ctx - (j0 + KT) < p.span;
      scores16<DK>(s[0], s[1], qf, kb, warp * 16);
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          const int j = j0 + warp * 16 + i * 8 + (lane & 3) * 2 + (x & 1), hr = (lane >> 2) + 8 * (x >> 1);
          s[i][x] = j < jend ? score_log2(p, s[i][x], sl2) : -INFINITY;
          if (near && j < jend && ctx - 1 - j < p.span && hr < nh) s[i][x] += LOG2E_F * p.bias[(long long)(g * rep + h0 + hr) * p.span + ctx - 1 - j];
          mx[x >> 1] = fmaxf(mx[x >> 1], s[i][x]);
        }
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        mx[y] = fmaxf(mx[y], __shfl_xor_sync(0xffffffffu, mx[y], 1));
        mx[y] = fmaxf(mx[y], __shfl_xor_sync(0xffffffffu, mx[y], 2));
        const float nm = fmaxf(m[y], mx[y]);         // finite: the warp has a visible key in this tile
        const float alpha = ex2(m[y] - nm);
        m[y] = nm;
        l[y] *= alpha;
#pragma unroll
        for (int i = 0; i < DV / 8; ++i) {
          o[i][2 * y] *= alpha;
          o[i][2 * y + 1] *= alpha;
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int x = 0; x < 4; ++x) {
          s[i][x] = ex2(s[i][x] - m[x >> 1]);
          l[x >> 1] += s[i][x];
        }
      weighted16<DV>(o, s[0], s[1], vb, warp * 16);
    }
  }
  // merge the four warps; the stages are free after the barrier
#pragma unroll
  for (int y = 0; y < 2; ++y) {
    l[y] += __shfl_xor_sync(0xffffffffu, l[y], 1);
    l[y] += __shfl_xor_sync(0xffffffffu, l[y], 2);
    if ((lane & 3) == 0) {
      s_m[warp][(lane >> 2) + 8 * y] = m[y];
      s_l[warp][(lane >> 2) + 8 * y] = l[y];
    }
  }
  __syncthreads();
  float* so = reinterpret_cast<float*>(smem);      // [4][16][DV]
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
#pragma unroll
    for (int x = 0; x < 4; ++x)
      so[(warp * 16 + (lane >> 2) + 8 * (x >> 1)) * DV + i * 8 + (lane & 3) * 2 + (x & 1)] = o[i][x];
  __syncthreads();
  for (int i = threadIdx.x; i < nh * p.vdim; i += 128) {
    const int r = i / p.vdim, c = i - r * p.vdim;
    float gm = -INFINITY, a = 0.f, gl = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) gm = fmaxf(gm, s_m[w][r]);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float f = s_m[w][r] == -INFINITY ? 0.f : ex2(s_m[w][r] - gm);
      a += so[(w * 16 + r) * DV + c] * f;
      gl += s_l[w][r] * f;
    }
    const int h = g * rep + h0 + r;
    if (splits == 1) {
      gl = with_sink(p, h, gm, gl);
      float f = gl > 0.f ? 1.f / gl : 0.f;
      if (p.gate) f *= p.gate[(long long)b * p.H + h];
      reinterpret_cast<bf16*>(p.out)[(long long)b * p.o_ld + (long long)h * p.vdim + c] = __float2bfloat16(a * f * gate_at<bf16>(p, b, h, c));
    } else {
      const long long idx = ((long long)b * p.H + h) * splits + split;
      part_o[idx * p.vdim + c] = a;
      if (c == 0) {
        part_ml[idx * 2] = gm;
        part_ml[idx * 2 + 1] = gl;
      }
    }
  }
}

__global__ void __launch_bounds__(128) attn_combine_kernel(const PagedParams p, int splits, const float* __restrict__ part_o,
                                                          const float* __restrict__ part_ml) {
  griddep_wait();
  griddep_launch();
  const int h = blockIdx.x, b = blockIdx.y;
  const long long base = ((long long)b * p.H + h) * splits;
  float gm = -INFINITY, gl = 0.f;
  for (int s = 0; s < splits; ++s) gm = fmaxf(gm, part_ml[(base + s) * 2]);
  for (int s = 0; s < splits; ++s) {
    const float ms = part_ml[(base + s) * 2];
    gl += ms == -INFINITY ? 0.f : part_ml[(base + s) * 2 + 1] * ex2(ms - gm);
  }
  gl = with_sink(p, h, gm, gl);
  float f = gl > 0.f ? 1.f / gl : 0.f;
  if (p.gate) f *= p.gate[(long long)b * p.H + h];
  for (int c = threadIdx.x; c < p.vdim; c += 128) {
    float a = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float ms = part_ml[(base + s) * 2];
      if (ms != -INFINITY) a += part_o[(base + s) * p.vdim + c] * ex2(ms - gm);
    }
    reinterpret_cast<bf16*>(p.out)[(long long)b * p.o_ld + (long long)h * p.vdim + c] = __float2bfloat16(a * f * gate_at<bf16>(p, b, h, c));
  }
}

template <typename K>
int allow_smem(K kernel, int bytes, bool* done) {
  int dev = 0;
  DLTI_CUDA_CHECK(cudaGetDevice(&dev));
  if (!done[dev & 63]) {
    DLTI_CUDA_CHECK(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes));
    done[dev & 63] = true;
  }
  return 0;
}

template <int DK, int DV>
int launch_prefill(const PagedParams& p, int nseq, int max_rows, cudaStream_t st) {
  static bool done[2][64] = {};
  const int smem = 2 * Tile<DK, DV>::BYTES;
  const bool extra = p.bias || p.ogate;
  auto kern = extra ? attn_prefill_kernel<DK, DV, true> : attn_prefill_kernel<DK, DV, false>;
  if (int rc = allow_smem(kern, smem, done[extra])) return rc;
  const long long tiles = ((long long)max_rows * (p.H / p.G) + PF_ROWS - 1) / PF_ROWS;
  kern<<<dim3((unsigned)tiles, p.G, nseq), 256, smem, st>>>(p);
  dlti_count_launch();
  return (int)cudaGetLastError();
}

template <int DK, int DV>
int launch_decode(const PagedParams& p, int splits, float* ws, cudaStream_t st) {
  static bool done[64] = {};
  const int merge = 4 * 16 * DV * 4, smem = 2 * Tile<DK, DV>::BYTES > merge ? 2 * Tile<DK, DV>::BYTES : merge;
  if (int rc = allow_smem(attn_decode_kernel<DK, DV>, smem, done)) return rc;
  const int rep = p.H / p.G;
  float* part_ml = ws + (long long)p.rows * p.H * splits * p.vdim;
  DLTI_CUDA_CHECK(dlti_launch_pdl(p.rows, attn_decode_kernel<DK, DV>, dim3(splits, p.G * ((rep + 15) / 16), (unsigned)p.rows), dim3(128),
                                  (size_t)smem, st, p, splits, ws, part_ml));
  dlti_count_launch();
  if (splits > 1) {
    DLTI_CUDA_CHECK(dlti_launch_pdl(p.rows, attn_combine_kernel, dim3(p.H, (unsigned)p.rows), dim3(128), 0, st, p, splits,
                                    (const float*)ws, (const float*)part_ml));
    dlti_count_launch();
  }
  return 0;
}

#define HEAD_DISPATCH(dim, vdim, F, ...)                                \
  do {                                                                  \
    const int dk_ = (dim) <= 64 ? 0 : ((dim) <= 128 ? 1 : 2);           \
    const int dv_ = (vdim) <= 64 ? 0 : ((vdim) <= 128 ? 1 : 2);         \
    switch (dk_ * 3 + dv_) {                                            \
      case 0: return F<64, 64>(__VA_ARGS__);                            \
      case 1: return F<64, 128>(__VA_ARGS__);                           \
      case 2: return F<64, 256>(__VA_ARGS__);                           \
      case 3: return F<128, 64>(__VA_ARGS__);                           \
      case 4: return F<128, 128>(__VA_ARGS__);                          \
      case 5: return F<128, 256>(__VA_ARGS__);                          \
      case 6: return F<256, 64>(__VA_ARGS__);                           \
      case 7: return F<256, 128>(__VA_ARGS__);                          \
      default: return F<256, 256>(__VA_ARGS__);                         \
    }                                                                   \
  } while (0)

}  // namespace

// rows of decode sequences (row s = sequence s < nd) and of prompts (sequence nd + i: rows nd + cu[i] ... nd + cu[i+1]).
DLTI_API int dlti_attn_rows(const void* q, long long q_ld, int q_hd, const void* kc, const void* vc, int kd, int vd, const int* tables,
                            int max_blocks, int bs, const int* ctx, const int* rseq, const int* pos, int H, int G, int dim, int vdim,
                            int chunk, int window, float scale, float cap, const float* gate, const float* sink, const float* bias, int span,
                            const void* ogate, long long og_ld, void* out, long long o_ld, long long rows, int dtype,
                            cudaStream_t st) {
  if (rows <= 0) return 0;
  if (H % G || dim < 1 || vdim < 1 || (chunk > 0 && window > 0)) return DLTI_ERR_BAD_ARG;
  if (dim > 2048 || vdim > 1024) { dlti_set_error("attn_rows: queries of up to 2048 and values of up to 1024 dimensions"); return DLTI_ERR_TOO_LARGE; }
  PagedParams p{q, q_ld, q_hd, kc, vc, kd, vd, tables, max_blocks, bs, ctx, nullptr, rseq, pos, 0, H, G, dim, vdim, chunk, window, scale, cap,
                gate, out, o_ld, rows, sink, bias, span, ogate, og_ld};
  if (dtype == DLTI_BF16) return launch_rows<__nv_bfloat16>(p, st);
  if (dtype == DLTI_FP32) return launch_rows<float>(p, st);
  return DLTI_ERR_UNSUPPORTED;
}

static int check_mma(int H, int G, int dim, int vdim, int kd, int vd, int q_hd) {
  if (H % G || dim < 1 || vdim < 1 || kd % 8 || vd % 8 || dim > kd || vdim > vd || q_hd % 2) return DLTI_ERR_BAD_ARG;
  if (kd > 256 || vd > 256) { dlti_set_error("paged attention: heads of up to 256 dimensions"); return DLTI_ERR_TOO_LARGE; }
  return 0;
}

// bf16. Prompt sequences nd ... nd + nseq - 1 (rows nd + cu[i] ...), at most max_rows rows each; the keys and values of
// the rows themselves must be in the pages already.
DLTI_API int dlti_attn_paged_prefill(const void* q, long long q_ld, int q_hd, const void* kc, const void* vc, int kd, int vd,
                                     const int* tables, int max_blocks, int bs, const int* ctx, const int* cu, int nd, int nseq,
                                     int max_rows, int H, int G, int dim, int vdim, int chunk, int window, float scale, float cap, const float* gate, const float* sink, const float* bias, int span,
                                     const void* ogate, long long og_ld, void* out, long long o_ld, cudaStream_t st) {
  if (nseq <= 0 || max_rows <= 0) return 0;
  if (int rc = check_mma(H, G, dim, vdim, kd, vd, q_hd)) return rc;
  if (q_ld % 2 || nseq > 65535) return DLTI_ERR_BAD_ARG;
  PagedParams p{q, q_ld, q_hd, kc, vc, kd, vd, tables, max_blocks, bs, ctx, cu, nullptr, nullptr, nd, H, G, dim, vdim, chunk, window, scale, cap,
                gate, out, o_ld, 0, sink, bias, span, ogate, og_ld};
  HEAD_DISPATCH(kd, vd, launch_prefill, p, nseq, max_rows, st);
}

// bf16. Row b = the newest token of sequence b, whose context is ctx[b] tokens. ws: batch * H * splits * (vdim + 2) floats.
DLTI_API int dlti_attn_paged_decode(const void* q, long long q_ld, int q_hd, const void* kc, const void* vc, int kd, int vd,
                                    const int* tables, int max_blocks, int bs, const int* ctx, int batch, int H, int G, int dim, int vdim,
                                    int chunk, int window, float scale, float cap, const float* gate, const float* sink, const float* bias, int span,
                                    const void* ogate, long long og_ld, int splits, float* ws, void* out, long long o_ld,
                                    cudaStream_t st) {
  if (batch <= 0) return 0;
  if (int rc = check_mma(H, G, dim, vdim, kd, vd, q_hd)) return rc;
  if (q_ld % 2 || splits < 1 || batch > 65535) return DLTI_ERR_BAD_ARG;
  PagedParams p{q, q_ld, q_hd, kc, vc, kd, vd, tables, max_blocks, bs, ctx, nullptr, nullptr, nullptr, 0, H, G, dim, vdim, chunk, window, scale, cap,
                gate, out, o_ld, batch, sink, bias, span, ogate, og_ld};
  HEAD_DISPATCH(kd, vd, launch_decode, p, splits, ws, st);
}
