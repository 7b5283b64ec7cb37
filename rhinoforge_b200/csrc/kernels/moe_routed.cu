// Mixture of experts of the mixed-layer decoders: the router (logits in fp32; group-limited choice, weights, and the plan of
// which expert gets which rows), the row gather of prefill-sized batches, and the expert GEMMs of small batches,
// whose work is reading the chosen experts' weights once.
//
// Sorted rows: the picks of an expert are neighbours; row k * T + t behind them belongs to the shared expert's token t.  A tile
// list entry {expert, first row, end row, 0} is one block of at most tile_rows sorted rows of one expert (expert number E: the
// shared one).
#include "../common/dtype.cuh"
#include "../common/host_util.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"
#include "../rf_api.h"

namespace rf {

constexpr int kRtLane = 8;            // experts per lane: up to 256

constexpr int kRtTokens = 32;         // tokens (warps) per CTA of the choice
constexpr int kRtOneCta = 64;         // up to this many tokens one CTA chooses for all of them and plans in shared memory

struct BestPick { uint32_t v; int i; };
// floats in an order that unsigned comparison keeps
__device__ __forceinline__ uint32_t ordered(float f) {
  const uint32_t u = __float_as_uint(f);
  return u ^ ((u >> 31) ? 0xffffffffu : 0x80000000u);
}
// largest of the lanes' values x[s] (index s * 32 + lane), ties to the lower index
template <int S>
__device__ __forceinline__ BestPick warp_argmax(const float (&x)[S], int lane) {
  BestPick b = {0u, 0x7fffffff};
#pragma unroll
  for (int s = 0; s < S; ++s) {
    const uint32_t v = ordered(x[s]);
    if (v > b.v) { b.v = v; b.i = s * 32 + lane; }
  }
  const uint32_t top = __reduce_max_sync(0xffffffffu, b.v);
  return BestPick{top, (int)__reduce_min_sync(0xffffffffu, b.v == top ? (unsigned)b.i : 0x7fffffffu)};
}

// One warp routes one token.  sc[s]: this lane's logits (expert s * 32 + lane); keys: shared scratch of E floats.  Lane j < k
// leaves with the j-th expert and its weight.
template <int S>
__device__ __forceinline__ void route_token(const RfMoeRouter& p, int lane, float (&sc)[S], float* keys, int* my_id, float* my_w) {
  const int E = p.experts;
  float mx = -INFINITY;
#pragma unroll
  for (int s = 0; s < S; ++s) mx = fmaxf(mx, s * 32 + lane < E ? sc[s] : -INFINITY);
  if (p.score_fn == RF_MOE_CHOSEN) {
#pragma unroll
    for (int s = 0; s < S; ++s)
      if (p.correction && s * 32 + lane < E) sc[s] += p.correction[s * 32 + lane];
  } else if (p.score_fn == RF_MOE_SOFTMAX) {
    mx = warp_max(mx);
    float sum = 0.f;
#pragma unroll
    for (int s = 0; s < S; ++s) {
      sc[s] = s * 32 + lane < E ? expf(sc[s] - mx) : 0.f;
      sum += sc[s];
    }
    sum = warp_sum(sum);
#pragma unroll
    for (int s = 0; s < S; ++s) sc[s] /= sum;
  } else {
#pragma unroll
    for (int s = 0; s < S; ++s) sc[s] = s * 32 + lane < E ? 1.f / (1.f + expf(-sc[s])) : 0.f;
  }
  float key[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    const int e = s * 32 + lane;
    key[s] = e < E ? sc[s] + (p.correction && p.score_fn != RF_MOE_CHOSEN ? p.correction[e] : 0.f) : -INFINITY;
  }
  if (p.keep < p.groups) {
    // a group counts as much as its best expert; experts outside the best groups cannot be chosen
    const int size = E / p.groups;
    __syncwarp();
#pragma unroll
    for (int s = 0; s < S; ++s)
      if (s * 32 + lane < E) keys[s * 32 + lane] = key[s];
    __syncwarp();
    float gs[S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
      const int g = s * 32 + lane;
      gs[s] = -INFINITY;
      if (g < p.groups)
        for (int i = 0; i < size; ++i) gs[s] = fmaxf(gs[s], keys[g * size + i]);
    }
    __syncwarp();
#pragma unroll
    for (int s = 0; s < S; ++s)
      if (s * 32 + lane < p.groups) keys[s * 32 + lane] = 0.f;      // now: is this group kept?
    __syncwarp();
    for (int j = 0; j < p.keep; ++j) {
      const BestPick b = warp_argmax<S>(gs, lane);
      if (b.i < p.groups && (b.i & 31) == lane) {
#pragma unroll
        for (int s = 0; s < S; ++s)
          if (s == (b.i >> 5)) gs[s] = -INFINITY;
        keys[b.i] = 1.f;
      }
    }
    __syncwarp();
#pragma unroll
    for (int s = 0; s < S; ++s) {
      const int e = s * 32 + lane;
      if (e < E && keys[e / size] == 0.f) key[s] = -INFINITY;
    }
  }
  float sum = 0.f;
  *my_w = 0.f;
  *my_id = -1;
  for (int j = 0; j < p.k; ++j) {
    const BestPick b = warp_argmax<S>(key, lane);
    float w = 0.f;
    if (b.i < E && (b.i & 31) == lane) {
#pragma unroll
      for (int s = 0; s < S; ++s)
        if (s == (b.i >> 5)) { w = sc[s]; key[s] = -INFINITY; }
    }
    w = __shfl_sync(0xffffffffu, w, b.i & 31);
    sum += w;
    if (lane == j) { *my_id = b.i < E ? b.i : -1; *my_w = w; }
  }
  if (p.score_fn == RF_MOE_CHOSEN) {                      // the first pick has the largest logit
    const float top = __shfl_sync(0xffffffffu, *my_w, 0), e = lane < p.k ? expf(*my_w - top) : 0.f;
    *my_w = e / warp_sum(e) * p.scale;
    return;
  }
  *my_w *= (p.norm_topk ? 1.f / (sum + 1e-20f) : 1.f) * p.scale;
}

struct PlanSmem { int32_t cnt[256], rows_at[257], tiles_at[257]; };

// Exclusive sums of the experts' counts (sm.cnt) and the tile list; all threads of the CTA.
__device__ __forceinline__ void plan_tiles(const RfMoeRouter& p, PlanSmem& sm) {
  const int tid = threadIdx.x, E = p.experts - p.identity, R = p.tile_rows;
  if (tid < 32) {
    int rows = 0, tiles = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int n = e0 + tid < E ? sm.cnt[e0 + tid] : 0, nt = (n + R - 1) / R;
      int ri = n, ti = nt;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int ro = __shfl_up_sync(0xffffffffu, ri, o), to = __shfl_up_sync(0xffffffffu, ti, o);
        if (tid >= o) { ri += ro; ti += to; }
      }
      if (e0 + tid < E) { sm.rows_at[e0 + tid] = rows + ri - n; sm.tiles_at[e0 + tid] = tiles + ti - nt; }
      rows += __shfl_sync(0xffffffffu, ri, 31);
      tiles += __shfl_sync(0xffffffffu, ti, 31);
    }
    if (tid == 0) { sm.rows_at[E] = rows; sm.tiles_at[E] = tiles; }
  }
  __syncthreads();
  for (int e = tid; e < E; e += blockDim.x) {
    const int r0 = sm.rows_at[e], n = sm.cnt[e];
    p.start[e] = r0;
    for (int i = 0; i * R < n; ++i)
      reinterpret_cast<int4*>(p.tiles)[1 + sm.tiles_at[e] + i] = make_int4(e, r0 + i * R, r0 + n, 0);
  }
  const int pairs = p.rows * p.k, shared = p.shared_tiles ? (p.rows + R - 1) / R : 0;
  for (int i = tid; i < shared; i += blockDim.x)
    reinterpret_cast<int4*>(p.tiles)[1 + sm.tiles_at[E] + i] = make_int4(E, pairs + i * R, pairs + p.rows, 0);
  if (tid == 0) p.tiles[0] = p.tiles[3] = sm.tiles_at[E] + shared;   // words 3.. are the list as rf_moe_grouped_gemm takes it
  if (p.scatter && p.has_shared)
    for (int t = tid; t < p.rows; t += blockDim.x) {
      p.slot_of[(size_t)t * p.slot_ld + p.k] = pairs + t;
      p.token_of_slot[pairs + t] = t;
      if (!p.shared_gate) p.slot_w[pairs + t] = 1.f;
    }
}

__device__ __forceinline__ void place_pick(const RfMoeRouter& p, const PlanSmem& sm, int i, int e, int rank, float w) {
  const int t = i / p.k, slot = e >= 0 ? sm.rows_at[e] + rank : -1;
  p.slot_of[(size_t)t * p.slot_ld + i % p.k] = slot;
  if (slot >= 0) {
    p.token_of_slot[slot] = t;
    p.slot_w[slot] = w;
  }
}

// Scores, choice and plan over the logits [splits][rows][experts] (partial sums, added in order).  One CTA: everything stays in
// shared memory.  Several: a CTA counts its own picks, takes its places among the experts' rows with one atomic per expert, and
// the last one to finish plans.
template <int S>
__global__ void __launch_bounds__(kRtTokens * 32) moe_choose_kernel(const RfMoeRouter p, int splits) {
  pdl_prologue();
  extern __shared__ __align__(16) float ch_sm[];          // [warps][E] keys, then the picks of one CTA's tokens
  __shared__ PlanSmem sm;
  __shared__ int32_t base[256];
  __shared__ int last;
  const int E = p.experts, real = E - p.identity, columns = E + p.shared_gate, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const bool alone = gridDim.x == 1;
  const int per_cta = alone ? kRtOneCta : kRtTokens, first = blockIdx.x * per_cta;
  const int here = min(per_cta, p.rows - first);
  float* keys = ch_sm + warp * E;
  int32_t* s_id = reinterpret_cast<int32_t*>(ch_sm + kRtTokens * E);
  int32_t* s_rank = s_id + per_cta * p.k;
  float* s_w = reinterpret_cast<float*>(s_rank + per_cta * p.k);
  for (int e = tid; e < real; e += blockDim.x) sm.cnt[e] = 0;
  __syncthreads();
  for (int t = warp; t < here; t += kRtTokens) {
    float sc[S];
#pragma unroll
    for (int s = 0; s < S; ++s) {
      const int e = s * 32 + lane;
      sc[s] = 0.f;
      if (e < E)
        for (int z = 0; z < splits; ++z) sc[s] += p.logits[((size_t)z * p.rows + first + t) * columns + e];
    }
    if (p.shared_gate && lane == 0) {
      float v = 0.f;
      for (int z = 0; z < splits; ++z) v += p.logits[((size_t)z * p.rows + first + t) * columns + E];
      p.slot_w[(size_t)p.rows * p.k + first + t] = 1.f / (1.f + expf(-v));
    }
    int id;
    float w;
    route_token<S>(p, lane, sc, keys, &id, &w);
    if (p.identity > 0) {
      const bool self = lane < p.k && id >= real;
      const float sum = warp_sum(self ? w : 0.f);
      if (lane == 0) p.self_w[first + t] = sum;
      if (self) id = -1;
    }
    if (lane < p.k) {
      const int i = t * p.k + lane;
      s_id[i] = id;
      s_w[i] = w;
      s_rank[i] = id >= 0 ? atomicAdd(&sm.cnt[id], 1) : -1;
    }
  }
  __syncthreads();
  if (!alone) {
    for (int e = tid; e < real; e += blockDim.x) base[e] = sm.cnt[e] ? atomicAdd(p.counters + e, sm.cnt[e]) : 0;
    __syncthreads();
  }
  for (int i = tid; i < here * p.k; i += blockDim.x) {
    const size_t at = (size_t)first * p.k + i;
    const int id = s_id[i];
    p.ids[at] = id;
    p.weights[at] = s_w[i];
    p.rank[at] = alone || id < 0 ? s_rank[i] : base[id] + s_rank[i];
  }
  if (alone) {
    plan_tiles(p, sm);
    if (p.scatter)
      for (int i = tid; i < here * p.k; i += blockDim.x) place_pick(p, sm, i, s_id[i], s_rank[i], s_w[i]);
    return;
  }
  __threadfence();
  __syncthreads();
  if (tid == 0) {
    last = atomicAdd(p.counters + real, 1) == (int)gridDim.x - 1;
    if (last) p.counters[real] = 0;
  }
  __syncthreads();
  if (!last) return;
  __threadfence();
  for (int e = tid; e < real; e += blockDim.x) {          // the counters are left at zero for the next launch
    sm.cnt[e] = __ldcg(p.counters + e);
    p.counters[e] = 0;
  }
  __syncthreads();
  plan_tiles(p, sm);
  if (p.scatter)
    for (int i = tid; i < p.rows * p.k; i += blockDim.x) place_pick(p, sm, i, __ldcg(p.ids + i), __ldcg(p.rank + i), __ldcg(p.weights + i));
}

// Logits in fp32: 16 * MT * TW tokens times 64 experts per CTA; TW warps along the tokens, the others and blockIdx.z split the
// width.  A lane's operand fragment is eight consecutive columns (the order of the columns inside a product does not matter as
// long as both operands agree), so fragments come straight from global memory as 16-byte loads.
template <typename T, int MT, int TW>
__global__ void __launch_bounds__(256, 2) moe_logits_kernel(const RfMoeRouter p) {
  pdl_prologue();
  constexpr int KW = 8 / TW, ROWS = 16 * MT * TW, LD = 68;
  extern __shared__ __align__(16) float lg[];             // [KW][ROWS][LD]
  const int E = p.experts + p.shared_gate, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q = lane & 3;
  const int tw = warp % TW, kw = warp / TW, t0 = blockIdx.x * ROWS + tw * 16 * MT, e0 = blockIdx.y * 64;
  const T* x = reinterpret_cast<const T*>(p.x);
  const T* w = reinterpret_cast<const T*>(p.w) + (size_t)(e0 + g) * p.width;
  const int kb_n = (p.width + 31) / 32, step = KW * gridDim.z;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  float acc[MT][8][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[m][n][i] = 0.f;
  for (int kb = blockIdx.z * KW + kw; kb < kb_n; kb += step) {
    const int k = kb * 32 + q * 8;
    const bool kin = k < p.width;
    uint4 b[8], a[MT][2];
#pragma unroll
    for (int n = 0; n < 8; ++n) b[n] = kin && e0 + n * 8 + g < E ? *reinterpret_cast<const uint4*>(w + (size_t)(n * 8) * p.width + k) : zero;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int t = t0 + m * 16 + h * 8 + g;
        a[m][h] = kin && t < p.rows ? *reinterpret_cast<const uint4*>(x + (size_t)t * p.ldx + k) : zero;
      }
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const uint32_t a0[4] = {a[m][0].x, a[m][1].x, a[m][0].y, a[m][1].y}, a1[4] = {a[m][0].z, a[m][1].z, a[m][0].w, a[m][1].w};
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        MmaOp<T>::mma(acc[m][n], a0, b[n].x, b[n].y);
        MmaOp<T>::mma(acc[m][n], a1, b[n].z, b[n].w);
      }
    }
  }
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      float* o = lg + ((size_t)kw * ROWS + tw * 16 * MT + m * 16 + g) * LD + n * 8 + q * 2;
      *reinterpret_cast<float2*>(o) = make_float2(acc[m][n][0], acc[m][n][1]);
      *reinterpret_cast<float2*>(o + 8 * LD) = make_float2(acc[m][n][2], acc[m][n][3]);
    }
  __syncthreads();
  for (int i = tid; i < ROWS * 64; i += 256) {
    const int r = i >> 6, e = i & 63, t = blockIdx.x * ROWS + r;
    if (t >= p.rows || e0 + e >= E) continue;
    float s = 0.f;
#pragma unroll
    for (int z = 0; z < KW; ++z) s += lg[((size_t)z * ROWS + r) * LD + e];       // the warps' parts in order: the same sum every time
    p.logits[((size_t)blockIdx.z * p.rows + t) * E + e0 + e] = s;
  }
}

// 32-bit models: one CTA per token, a warp per expert.
__global__ void __launch_bounds__(256) moe_logits_f32_kernel(const RfMoeRouter p) {
  pdl_prologue();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x;
  const float* x = reinterpret_cast<const float*>(p.x) + (size_t)t * p.ldx;
  const int columns = p.experts + p.shared_gate;
  for (int e = warp; e < columns; e += 8) {
    const float* w = reinterpret_cast<const float*>(p.w) + (size_t)e * p.width;
    float s = 0.f;
    for (int i = lane; i < p.width; i += 32) s += x[i] * w[i];
    s = warp_sum(s);
    if (lane == 0) p.logits[(size_t)t * columns + e] = s;
  }
}

// Prefill-sized batches: every token's row is copied to its sorted rows.
template <typename T>
__global__ void __launch_bounds__(256) moe_gather_kernel(const RfMoeRouter p, T* __restrict__ out, int64_t ldo, int cols) {
  pdl_prologue();
  __shared__ int32_t slots[32];
  const int t = blockIdx.x, pairs = p.rows * p.k;
  if (threadIdx.x < (unsigned)p.k) {
    const size_t i = (size_t)t * p.k + threadIdx.x;
    const int e = p.ids[i], slot = e >= 0 ? p.start[e] + p.rank[i] : -1;
    slots[threadIdx.x] = slot;
    p.slot_of[(size_t)t * p.slot_ld + threadIdx.x] = slot;
    if (slot >= 0) {
      p.token_of_slot[slot] = t;
      p.slot_w[slot] = p.weights[i];
    }
  }
  if (threadIdx.x == 32 && p.has_shared) {
    p.slot_of[(size_t)t * p.slot_ld + p.k] = pairs + t;
    p.token_of_slot[pairs + t] = t;
    if (!p.shared_gate) p.slot_w[pairs + t] = 1.f;
  }
  __syncthreads();
  const T* x = reinterpret_cast<const T*>(p.x) + (size_t)t * p.ldx;
  for (int c = threadIdx.x * 8; c < cols; c += blockDim.x * 8) {
    const Vec8<T> v = *reinterpret_cast<const Vec8<T>*>(x + c);
    for (int j = 0; j < p.k; ++j)
      if (slots[j] >= 0) *reinterpret_cast<Vec8<T>*>(out + (size_t)slots[j] * ldo + c) = v;
  }
}

// --------------------------------------------------------------------------------- expert GEMMs, few rows ----
__device__ __forceinline__ uint4 ld_weight(const uint8_t* p) {       // read once: no allocation in L1
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

// One CTA: up to 16 * MT sorted rows of one expert times FW * NT * 8 of its features.  KW warps split the contraction, FW the
// features.  Weights come from the tile-major image (128 rows x 64 columns, 16-byte pieces swizzled inside a row) straight into
// the fragments: no staging, no barriers until the warps add up.
template <typename T, int MT, bool DUAL, int KW, int NT>
__global__ void __launch_bounds__(256, MT == 1 ? 2 : 1) moe_small_kernel(const RfMoeExperts p) {
  pdl_prologue();
  constexpr int FW = 8 / KW, FEAT = FW * NT * 8, D = DUAL ? 2 : 1;
  extern __shared__ __align__(16) float red[];                       // [KW][D][16 * MT][FEAT + 4]
  constexpr int LD = FEAT + 4;
  if ((int)blockIdx.y >= p.tiles[0]) return;
  const int4 tile = reinterpret_cast<const int4*>(p.tiles)[1 + blockIdx.y];
  const bool sh = tile.x == p.experts;
  const int N = sh ? p.shared_n : p.n, K = sh ? p.shared_k : p.k, f0 = blockIdx.x * FEAT;
  if (f0 >= N) return;
  const int row0 = tile.y, rows = min(tile.z - tile.y, 16 * MT);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3, kw = warp / FW, fw = warp % FW;
  const uint8_t* w = reinterpret_cast<const uint8_t*>(sh ? p.w_shared : p.w);
  const int kb_total = sh ? p.shared_kb_total : p.bank_kb_total, section = sh ? p.shared_section_row_tiles : p.bank_section_row_tiles;
  const int rt0 = sh ? 0 : tile.x * p.rt_per_expert, kb0 = sh ? 0 : tile.x * p.kb_per_expert;
  // this lane's row of the first feature eight; the warp's features lie in one 128-row tile of the image, whose rows behind the
  // last feature are zero
  static_assert(128 % FEAT == 0, "features of a CTA lie in one row tile");
  const int f = f0 + fw * NT * 8 + g;
  const uint8_t* wrow[D];
  wrow[0] = w + ((size_t)(rt0 + (f >> 7)) * kb_total + kb0) * 16384 + (size_t)(f & 127) * 128;
  if (DUAL) wrow[D - 1] = wrow[0] + (size_t)section * kb_total * 16384;
  const T* xrow[MT][2];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = m * 16 + h * 8 + g;
      const int s = row0 + r;
      xrow[m][h] = r < rows ? reinterpret_cast<const T*>(p.x) + (size_t)(p.token_of_slot ? p.token_of_slot[s] : s) * p.ldx : nullptr;
    }
  float acc[D][MT][NT][4];
#pragma unroll
  for (int d = 0; d < D; ++d)
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[d][m][n][i] = 0.f;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  const int kn = (K + 31) / 32;
#pragma unroll 2
  for (int kb = kw; kb < kn; kb += KW) {
    const size_t off = (size_t)(kb >> 1) * 16384 + (((((kb & 1) << 2) | q) ^ g) << 4);     // f & 7 == g
    uint4 b[D][NT], a[MT][2];
#pragma unroll
    for (int d = 0; d < D; ++d)
#pragma unroll
      for (int n = 0; n < NT; ++n) b[d][n] = ld_weight(wrow[d] + off + n * 1024);
    const int k = kb * 32 + q * 8;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int h = 0; h < 2; ++h) a[m][h] = xrow[m][h] && k < K ? *reinterpret_cast<const uint4*>(xrow[m][h] + k) : zero;
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const uint32_t a0[4] = {a[m][0].x, a[m][1].x, a[m][0].y, a[m][1].y}, a1[4] = {a[m][0].z, a[m][1].z, a[m][0].w, a[m][1].w};
#pragma unroll
      for (int d = 0; d < D; ++d)
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          MmaOp<T>::mma(acc[d][m][n], a0, b[d][n].x, b[d][n].y);
          MmaOp<T>::mma(acc[d][m][n], a1, b[d][n].z, b[d][n].w);
        }
    }
  }
#pragma unroll
  for (int d = 0; d < D; ++d)
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        float* o = red + ((size_t)(kw * D + d) * 16 * MT + m * 16 + g) * LD + (fw * NT + n) * 8 + q * 2;
        *reinterpret_cast<float2*>(o) = make_float2(acc[d][m][n][0], acc[d][m][n][1]);
        *reinterpret_cast<float2*>(o + 8 * LD) = make_float2(acc[d][m][n][2], acc[d][m][n][3]);
      }
  __syncthreads();
  for (int i = threadIdx.x; i < rows * (FEAT / 8); i += 256) {
    const int r = i / (FEAT / 8), c = (i % (FEAT / 8)) * 8;
    if (f0 + c >= N) continue;
    float v[D][8];
#pragma unroll
    for (int d = 0; d < D; ++d) {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[d][j] = 0.f;
#pragma unroll
      for (int z = 0; z < KW; ++z) {
        float f[8];
        load8(red + ((size_t)(z * D + d) * 16 * MT + r) * LD + c, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[d][j] += f[j];
      }
    }
    const float ws = p.slot_w ? p.slot_w[row0 + r] : 1.f;
    if constexpr (DUAL) {
      if (p.act == kActClippedGlu) {
        const ActArgs a = {sh ? p.shared_limit : p.act_limit, p.act_alpha};
#pragma unroll
        for (int j = 0; j < 8; ++j) v[0][j] = clipped_glu_f(v[0][j], v[D - 1][j], a);
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) v[0][j] = silu_f(v[0][j]) * v[D - 1][j];
      }
    } else if (p.act != kActNone && !act_is_dual(p.act)) {
      apply_act_n<8>(p.act, v[0], v[0], v[0], ActArgs{p.act_limit, p.act_alpha});
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) v[0][j] *= ws;
    store8(reinterpret_cast<T*>(p.out) + (size_t)(row0 + r) * p.ldo + f0 + c, v[0]);
  }
}

// 32-bit models: 64 x 64 tiles on the CUDA cores; weights are plain row-major matrices per expert.
template <bool DUAL>
__global__ void __launch_bounds__(256) moe_f32_kernel(const RfMoeExperts p) {
  pdl_prologue();
  constexpr int BM = 64, BN = 64, BK = 16, D = DUAL ? 2 : 1;
  __shared__ __align__(16) float sx[BK][BM + 4], sw[D][BK][BN + 4];
  if ((int)blockIdx.y >= p.tiles[0]) return;
  const int4 tile = reinterpret_cast<const int4*>(p.tiles)[1 + blockIdx.y];
  const bool sh = tile.x == p.experts;
  const int N = sh ? p.shared_n : p.n, K = sh ? p.shared_k : p.k, n0 = blockIdx.x * BN;
  if (n0 >= N) return;
  const float* w = reinterpret_cast<const float*>(sh ? p.w_shared : p.w) + (sh ? 0 : (size_t)tile.x * N * K);
  const size_t second = sh ? (size_t)N * K : (size_t)p.experts * N * K;
  const int row0 = tile.y, rows = min(tile.z - tile.y, BM), tid = threadIdx.x;
  const int tx = tid % 16, ty = tid / 16, lr = tid / 4, lk = (tid % 4) * 4;
  const float* x = nullptr;
  if (lr < rows) x = reinterpret_cast<const float*>(p.x) + (size_t)(p.token_of_slot ? p.token_of_slot[row0 + lr] : row0 + lr) * p.ldx;
  float acc[D][4][4] = {};
  for (int k0 = 0; k0 < K; k0 += BK) {
    const bool kin = k0 + lk < K;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    if (kin && x) a = *reinterpret_cast<const float4*>(x + k0 + lk);
    sx[lk][lr] = a.x; sx[lk + 1][lr] = a.y; sx[lk + 2][lr] = a.z; sx[lk + 3][lr] = a.w;
#pragma unroll
    for (int d = 0; d < D; ++d) {
      float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
      if (kin && n0 + lr < N) b = *reinterpret_cast<const float4*>(w + d * second + (size_t)(n0 + lr) * K + k0 + lk);
      sw[d][lk][lr] = b.x; sw[d][lk + 1][lr] = b.y; sw[d][lk + 2][lr] = b.z; sw[d][lk + 3][lr] = b.w;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < BK; ++k)
#pragma unroll
      for (int d = 0; d < D; ++d)
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[d][i][j] = fmaf(sx[k][ty * 4 + i], sw[d][k][tx * 4 + j], acc[d][i][j]);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int r = ty * 4 + i, n = n0 + tx * 4 + j;
      if (r >= rows || n >= N) continue;
      const float g = acc[0][i][j];
      float v = g;
      if constexpr (DUAL) {
        const float u = acc[D - 1][i][j], limit = sh ? p.shared_limit : p.act_limit, gc = fminf(g, limit);
        v = p.act == kActClippedGlu ? gc / (1.f + expf(-p.act_alpha * gc)) * (fminf(fmaxf(u, -limit), limit) + 1.f) : g / (1.f + expf(-g)) * u;
      } else if (p.act == kActGeluErf) {
        v = 0.5f * g * (1.f + erff(g * 0.7071067811865476f));
      }
      reinterpret_cast<float*>(p.out)[(size_t)(row0 + r) * p.ldo + n] = v * (p.slot_w ? p.slot_w[row0 + r] : 1.f);
    }
}

// CTAs that share the width of one tile of tokens: about two 32-column blocks per warp, as long as the GPU has room
static int router_splits(int rows, int experts, int width) {
  if (rows > 1024) return 1;
  const int tiles = ceil_div(rows, 16) * ceil_div(experts, 64);
  return std::max(1, std::min({16, width / (32 * 8 * 2), 2 * sm_count() / tiles}));
}

template <typename T, int MT, int TW>
static int launch_logits(const RfMoeRouter* a, int splits, cudaStream_t s) {
  constexpr int ROWS = 16 * MT * TW;
  const size_t smem = (size_t)(8 / TW) * ROWS * 68 * sizeof(float);
  RF_ALLOW_SMEM_PER_DEVICE((moe_logits_kernel<T, MT, TW>), 80 * 1024);
  RF_CUDA_CHECK(::rf::launch_k(moe_logits_kernel<T, MT, TW>, dim3(ceil_div(a->rows, ROWS), ceil_div(a->experts + a->shared_gate, 64), splits), dim3(256), smem, s, 1, *a));
  ::rf::count_launch();
  return RF_OK;
}

template <int S>
static int launch_choose(const RfMoeRouter* a, int splits, cudaStream_t s) {
  const bool alone = a->rows <= kRtOneCta;
  const int per_cta = alone ? kRtOneCta : kRtTokens;
  const size_t smem = ((size_t)kRtTokens * a->experts + 3 * per_cta * a->k) * sizeof(float);
  RF_ALLOW_SMEM_PER_DEVICE(moe_choose_kernel<S>, 64 * 1024);
  RF_CUDA_CHECK(::rf::launch_k(moe_choose_kernel<S>, dim3(alone ? 1 : ceil_div(a->rows, kRtTokens)), dim3(kRtTokens * 32), smem, s, 1, *a, splits));
  ::rf::count_launch();
  return RF_OK;
}

template <typename T, int MT, bool DUAL, int KW, int NT>
static int launch_small(const RfMoeExperts* a, cudaStream_t s) {
  constexpr int FEAT = 8 / KW * NT * 8;
  const size_t smem = (size_t)KW * (DUAL ? 2 : 1) * 16 * MT * (FEAT + 4) * sizeof(float);
  RF_ALLOW_SMEM_PER_DEVICE((moe_small_kernel<T, MT, DUAL, KW, NT>), 160 * 1024);
  const dim3 grid(ceil_div(std::max(a->n, a->shared_n), FEAT), a->max_tiles);
  RF_CUDA_CHECK(::rf::launch_k(moe_small_kernel<T, MT, DUAL, KW, NT>, grid, dim3(256), smem, s, 1, *a));
  ::rf::count_launch();
  return RF_OK;
}

template <typename T>
static int dispatch_small(const RfMoeExperts* a, cudaStream_t s) {
  // one operand: CTAs of 128 features, or of 32 where those would not fill the GPU
  const bool narrow = (long)ceil_div(std::max(a->n, a->shared_n), 128) * a->max_tiles < 2 * sm_count();
  if (a->tile_rows <= 16) {
    if (a->dual) return launch_small<T, 1, true, 8, 4>(a, s);
    return narrow ? launch_small<T, 1, false, 8, 4>(a, s) : launch_small<T, 1, false, 4, 8>(a, s);
  }
  if (a->dual) return launch_small<T, 2, true, 8, 4>(a, s);
  return narrow ? launch_small<T, 2, false, 8, 4>(a, s) : launch_small<T, 2, false, 4, 8>(a, s);
}

static int check_router(const RfMoeRouter* a) {
  RF_REQUIRE(a && a->x && a->ids && a->weights && a->rank && a->counters && a->start && a->tiles && a->slot_of && a->token_of_slot && a->slot_w,
             "moe_router: missing buffers");
  RF_REQUIRE(a->experts > 0 && a->experts <= 32 * kRtLane && a->k > 0 && a->k <= 32 && a->groups > 0 && a->experts % a->groups == 0 &&
                 a->keep > 0 && a->keep <= a->groups && a->k <= a->experts / a->groups * a->keep,
             "moe_router: %d experts in %d groups, %d groups kept, %d experts chosen", a->experts, a->groups, a->keep, a->k);
  RF_REQUIRE(a->width > 0 && a->width % 8 == 0 && a->ldx % 8 == 0 && a->tile_rows > 0 && a->slot_ld >= a->k + (a->has_shared ? 1 : 0),
             "moe_router: width %d, tile of %d rows", a->width, a->tile_rows);
  RF_REQUIRE(a->dtype >= 0 && a->dtype <= 2 && (int64_t)a->rows * (a->k + 1) < (1ll << 30), "moe_router: dtype %d", a->dtype);
  RF_REQUIRE(a->score_fn >= RF_MOE_SIGMOID && a->score_fn <= RF_MOE_CHOSEN && (a->shared_gate == 0 || (a->shared_gate == 1 && a->has_shared)),
             "moe_router: score function %d, gate of the shared expert %d", a->score_fn, a->shared_gate);
  RF_REQUIRE(a->identity >= 0 && a->identity < a->experts && (a->identity == 0 || a->self_w), "moe_router: %d identity experts of %d", a->identity, a->experts);
  return RF_OK;
}

}  // namespace rf

using namespace rf;

extern "C" int rf_moe_router(const RfMoeRouter* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  int rc = check_router(a);
  if (rc) return rc;
  RF_REQUIRE(a->w && a->logits, "moe_router: weights and logits");
  if (a->rows == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  int splits = 1, rc2;
  if (a->dtype == kF32) {
    RF_CUDA_CHECK(::rf::launch_k(moe_logits_f32_kernel, dim3(a->rows), dim3(256), 0, s, 1, *a));
    ::rf::count_launch();
  } else {
    const bool many = a->rows > 1024;
    splits = router_splits(a->rows, a->experts + a->shared_gate, a->width);
    if (a->dtype == kF16) rc2 = many ? launch_logits<__half, 2, 2>(a, 1, s) : launch_logits<__half, 1, 1>(a, splits, s);
    else rc2 = many ? launch_logits<__nv_bfloat16, 2, 2>(a, 1, s) : launch_logits<__nv_bfloat16, 1, 1>(a, splits, s);
    if (rc2) return rc2;
  }
  if (a->experts <= 64) return launch_choose<2>(a, splits, s);
  return a->experts <= 128 ? launch_choose<4>(a, splits, s) : launch_choose<kRtLane>(a, splits, s);
}

extern "C" uint64_t rf_moe_router_scratch_bytes(int rows, int experts) {
  // rows x splits stays below two waves of 16-row tiles unless there is one split only
  return ((uint64_t)std::max(rows, 2 * sm_count() * 16 + 16)) * experts * sizeof(float);
}

extern "C" int rf_moe_gather(const RfMoeRouter* a, void* out, int64_t ldo, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  int rc = check_router(a);
  if (rc) return rc;
  RF_REQUIRE(out && ldo % 8 == 0 && ldo >= a->width, "moe_gather: output");
  if (a->rows == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (a->dtype == kF16) RF_CUDA_CHECK(::rf::launch_k(moe_gather_kernel<__half>, dim3(a->rows), dim3(256), 0, s, 1, *a, (__half*)out, ldo, a->width));
  else if (a->dtype == kBF16) RF_CUDA_CHECK(::rf::launch_k(moe_gather_kernel<__nv_bfloat16>, dim3(a->rows), dim3(256), 0, s, 1, *a, (__nv_bfloat16*)out, ldo, a->width));
  else RF_CUDA_CHECK(::rf::launch_k(moe_gather_kernel<float>, dim3(a->rows), dim3(256), 0, s, 1, *a, (float*)out, ldo, a->width));
  ::rf::count_launch();
  return RF_OK;
}

extern "C" int rf_moe_experts(const RfMoeExperts* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_REQUIRE(a && a->x && a->w && a->out && a->tiles && a->max_tiles > 0 && a->max_tiles <= 65535, "moe_experts: missing buffers");
  RF_REQUIRE(a->n > 0 && a->k > 0 && a->n % 8 == 0 && a->k % 8 == 0 && a->ldx % 8 == 0 && a->ldo % 8 == 0, "moe_experts: %d x %d", a->n, a->k);
  RF_REQUIRE((a->shared_n > 0) == (a->w_shared != nullptr) && a->shared_n % 8 == 0 && a->shared_k % 8 == 0, "moe_experts: shared expert");
  RF_REQUIRE(a->dtype >= 0 && a->dtype <= 2, "moe_experts: dtype %d", a->dtype);
  RF_REQUIRE(a->act == 0 || a->act == kActSiluMul || (a->act == kActGeluErf && !a->dual) || (a->act == kActClippedGlu && a->act_limit > 0.f && (!a->w_shared || a->shared_limit > 0.f)),
             "moe_experts: activation %d", a->act);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (a->dtype == kF32) {
    RF_REQUIRE(a->tile_rows == 64, "moe_experts: 32-bit tiles have 64 rows");
    const dim3 grid(ceil_div(std::max(a->n, a->shared_n), 64), a->max_tiles);
    if (a->dual) RF_CUDA_CHECK(::rf::launch_k(moe_f32_kernel<true>, grid, dim3(256), 0, s, 1, *a));
    else RF_CUDA_CHECK(::rf::launch_k(moe_f32_kernel<false>, grid, dim3(256), 0, s, 1, *a));
    ::rf::count_launch();
    return RF_OK;
  }
  RF_REQUIRE(a->tile_rows == 16 || a->tile_rows == 32, "moe_experts: tiles of %d rows", a->tile_rows);
  RF_REQUIRE(a->bank_kb_total > 0 && (!a->w_shared || a->shared_kb_total > 0), "moe_experts: bank geometry");
  return a->dtype == kF16 ? dispatch_small<__half>(a, s) : dispatch_small<__nv_bfloat16>(a, s);
}
