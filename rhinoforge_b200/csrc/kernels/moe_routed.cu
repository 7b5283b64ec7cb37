// Mixture of experts of the mixed-layer decoders: the router as one launch (logits in fp32, group-limited choice, weights, and
// the plan of which expert gets which rows), the row gather of prefill-sized batches, and the expert GEMMs of small batches,
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

struct BestPick { float v; int i; };
__device__ __forceinline__ BestPick warp_argmax(BestPick b) {       // ties go to the lower index
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, b.v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, b.i, o);
    if (ov > b.v || (ov == b.v && oi < b.i)) { b.v = ov; b.i = oi; }
  }
  return b;
}

// One warp routes one token.  sc[s]: this lane's logits (expert s * 32 + lane); keys: shared scratch of E floats.
__device__ __forceinline__ void route_token(const RfMoeRouter& p, int t, int lane, float (&sc)[kRtLane], float* keys) {
  const int E = p.experts;
  float mx = -INFINITY;
#pragma unroll
  for (int s = 0; s < kRtLane; ++s) mx = fmaxf(mx, s * 32 + lane < E ? sc[s] : -INFINITY);
  if (p.score_fn == RF_MOE_SOFTMAX) {
    mx = warp_max(mx);
    float sum = 0.f;
#pragma unroll
    for (int s = 0; s < kRtLane; ++s) {
      sc[s] = s * 32 + lane < E ? expf(sc[s] - mx) : 0.f;
      sum += sc[s];
    }
    sum = warp_sum(sum);
#pragma unroll
    for (int s = 0; s < kRtLane; ++s) sc[s] /= sum;
  } else {
#pragma unroll
    for (int s = 0; s < kRtLane; ++s) sc[s] = s * 32 + lane < E ? 1.f / (1.f + expf(-sc[s])) : 0.f;
  }
  float key[kRtLane];
#pragma unroll
  for (int s = 0; s < kRtLane; ++s) {
    const int e = s * 32 + lane;
    key[s] = e < E ? sc[s] + (p.correction ? p.correction[e] : 0.f) : -INFINITY;
  }
  if (p.keep < p.groups) {
    // a group counts as much as its best expert; experts outside the best groups cannot be chosen
    const int size = E / p.groups;
    __syncwarp();
#pragma unroll
    for (int s = 0; s < kRtLane; ++s)
      if (s * 32 + lane < E) keys[s * 32 + lane] = key[s];
    __syncwarp();
    float gs[kRtLane];
#pragma unroll
    for (int s = 0; s < kRtLane; ++s) {
      const int g = s * 32 + lane;
      gs[s] = -INFINITY;
      if (g < p.groups)
        for (int i = 0; i < size; ++i) gs[s] = fmaxf(gs[s], keys[g * size + i]);
    }
    __syncwarp();
#pragma unroll
    for (int s = 0; s < kRtLane; ++s)
      if (s * 32 + lane < p.groups) keys[s * 32 + lane] = 0.f;      // now: is this group kept?
    __syncwarp();
    for (int j = 0; j < p.keep; ++j) {
      BestPick b = {-INFINITY, 0x7fffffff};
#pragma unroll
      for (int s = 0; s < kRtLane; ++s)
        if (gs[s] > b.v) b = {gs[s], s * 32 + lane};
      b = warp_argmax(b);
      if (b.i < p.groups && (b.i & 31) == lane) {
#pragma unroll
        for (int s = 0; s < kRtLane; ++s)
          if (s == (b.i >> 5)) gs[s] = -INFINITY;
        keys[b.i] = 1.f;
      }
    }
    __syncwarp();
#pragma unroll
    for (int s = 0; s < kRtLane; ++s) {
      const int e = s * 32 + lane;
      if (e < E && keys[e / size] == 0.f) key[s] = -INFINITY;
    }
  }
  float sum = 0.f, my_w = 0.f;
  int my_id = -1;
  for (int j = 0; j < p.k; ++j) {
    BestPick b = {-INFINITY, 0x7fffffff};
#pragma unroll
    for (int s = 0; s < kRtLane; ++s)
      if (key[s] > b.v) b = {key[s], s * 32 + lane};
    b = warp_argmax(b);
    float w = 0.f;
    if (b.i < E && (b.i & 31) == lane) {
#pragma unroll
      for (int s = 0; s < kRtLane; ++s)
        if (s == (b.i >> 5)) { w = sc[s]; key[s] = -INFINITY; }
    }
    w = __shfl_sync(0xffffffffu, w, b.i & 31);
    sum += w;
    if (lane == j) { my_id = b.i < E ? b.i : -1; my_w = w; }
  }
  const float mul = (p.norm_topk ? 1.f / (sum + 1e-20f) : 1.f) * p.scale;
  if (lane < p.k) {
    const size_t at = (size_t)t * p.k + lane;
    p.ids[at] = my_id;
    p.weights[at] = my_w * mul;
    p.rank[at] = my_id >= 0 ? atomicAdd(&p.counters[my_id], 1) : -1;
  }
}

// Exclusive sums over the experts and the tile list; by the CTA whose ticket is the last (all of the router's results are
// visible to it then).  Leaves the counters at zero for the next launch.
__device__ __forceinline__ void router_plan(const RfMoeRouter& p) {
  __shared__ int32_t rows_at[257], tiles_at[257], cnt[256];
  const int tid = threadIdx.x, E = p.experts, R = p.tile_rows;
  for (int e = tid; e < E; e += blockDim.x) {
    cnt[e] = __ldcg(p.counters + e);
    p.counters[e] = 0;
  }
  __syncthreads();
  if (tid < 32) {
    int rows = 0, tiles = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int n = e0 + tid < E ? cnt[e0 + tid] : 0, nt = (n + R - 1) / R;
      int ri = n, ti = nt;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int ro = __shfl_up_sync(0xffffffffu, ri, o), to = __shfl_up_sync(0xffffffffu, ti, o);
        if (tid >= o) { ri += ro; ti += to; }
      }
      if (e0 + tid < E) { rows_at[e0 + tid] = rows + ri - n; tiles_at[e0 + tid] = tiles + ti - nt; }
      rows += __shfl_sync(0xffffffffu, ri, 31);
      tiles += __shfl_sync(0xffffffffu, ti, 31);
    }
    if (tid == 0) { rows_at[E] = rows; tiles_at[E] = tiles; }
  }
  __syncthreads();
  for (int e = tid; e < E; e += blockDim.x) {
    const int r0 = rows_at[e], n = cnt[e];
    p.start[e] = r0;
    for (int i = 0; i * R < n; ++i)
      reinterpret_cast<int4*>(p.tiles)[1 + tiles_at[e] + i] = make_int4(e, r0 + i * R, r0 + n, 0);
  }
  const int pairs = p.rows * p.k, shared = p.shared_tiles ? (p.rows + R - 1) / R : 0;
  for (int i = tid; i < shared; i += blockDim.x)
    reinterpret_cast<int4*>(p.tiles)[1 + tiles_at[E] + i] = make_int4(E, pairs + i * R, pairs + p.rows, 0);
  if (tid == 0) p.tiles[0] = p.tiles[3] = tiles_at[E] + shared;    // words 3.. are the list as rf_moe_grouped_gemm takes it
  if (p.scatter) {
    for (int i = tid; i < pairs; i += blockDim.x) {
      const int e = __ldcg(p.ids + i), t = i / p.k;
      const int slot = e >= 0 ? rows_at[e] + __ldcg(p.rank + i) : -1;
      p.slot_of[(size_t)t * p.slot_ld + i % p.k] = slot;
      if (slot >= 0) {
        p.token_of_slot[slot] = t;
        p.slot_w[slot] = __ldcg(p.weights + i);
      }
    }
    if (p.has_shared)
      for (int t = tid; t < p.rows; t += blockDim.x) {
        p.slot_of[(size_t)t * p.slot_ld + p.k] = pairs + t;
        p.token_of_slot[pairs + t] = t;
        p.slot_w[pairs + t] = 1.f;
      }
  }
}

__device__ __forceinline__ void router_ticket(const RfMoeRouter& p) {
  __shared__ int last;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) {
    const int n = (int)(gridDim.x * gridDim.y * gridDim.z);
    last = atomicAdd(p.counters + p.experts, 1) == n - 1;
    if (last) p.counters[p.experts] = 0;
  }
  __syncthreads();
  if (!last) return;
  __threadfence();
  router_plan(p);
}

// MT * 16 tokens per cluster.  Warps and cluster CTAs split the width; a lane's operand fragment is eight consecutive columns
// (the order of the columns inside a product does not matter as long as both operands agree), so fragments come straight from
// global memory as 16-byte loads.
template <typename T, int MT>
__global__ void __launch_bounds__(256) moe_router_kernel(const RfMoeRouter p) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float lg[];             // [16 * MT][E] logits, then one row of keys per warp
  const int E = p.experts, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q = lane & 3;
  const int splits = gridDim.z, rank = blockIdx.z, t0 = blockIdx.x * 16 * MT;
  const T* x = reinterpret_cast<const T*>(p.x);
  const T* w = reinterpret_cast<const T*>(p.w);
  pdl_wait();
  const int kb_n = (p.width + 31) / 32;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  for (int e0 = 0; e0 < E; e0 += 64) {
    float acc[MT][8][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[m][n][i] = 0.f;
#pragma unroll 2
    for (int kb = rank * 8 + warp; kb < kb_n; kb += 8 * splits) {
      const int k = kb * 32 + q * 8;
      const bool kin = k < p.width;
      uint4 b[8], a[MT][2];
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        const int e = e0 + n * 8 + g;
        b[n] = kin && e < E ? *reinterpret_cast<const uint4*>(w + (size_t)e * p.width + k) : zero;
      }
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
    for (int v = 0; v < 8; ++v) {                          // the warps add in order: the same sum every time
      if (warp == v) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int n = 0; n < 8; ++n)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              const int e = e0 + n * 8 + q * 2 + (i & 1), r = m * 16 + g + (i >> 1) * 8;
              if (e < E) lg[r * E + e] = (v ? lg[r * E + e] : 0.f) + acc[m][n][i];
            }
      }
      __syncthreads();
    }
  }
  if (splits > 1) cluster_sync_all();
  float* keys = lg + 16 * MT * E + warp * E;
  for (int r = rank + splits * warp; r < 16 * MT; r += splits * 8) {
    if (t0 + r >= p.rows) break;
    float sc[kRtLane];
#pragma unroll
    for (int s = 0; s < kRtLane; ++s) {
      const int e = s * 32 + lane;
      sc[s] = 0.f;
      if (e < E) {
        if (splits == 1) sc[s] = lg[r * E + e];
        else
          for (int z = 0; z < splits; ++z) sc[s] += ld_dsmem_f32(dsmem_addr(smem_u32(lg + r * E + e), (uint32_t)z));
      }
    }
    route_token(p, t0 + r, lane, sc, keys);
  }
  if (splits > 1) cluster_sync_all();                      // nobody leaves while its logits are read
  router_ticket(p);
}

// 32-bit models: one CTA per token, a warp per expert.
__global__ void __launch_bounds__(256) moe_router_f32_kernel(const RfMoeRouter p) {
  pdl_prologue();
  extern __shared__ __align__(16) float lg[];
  const int E = p.experts, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x;
  const float* x = reinterpret_cast<const float*>(p.x) + (size_t)t * p.ldx;
  for (int e = warp; e < E; e += 8) {
    const float* w = reinterpret_cast<const float*>(p.w) + (size_t)e * p.width;
    float s = 0.f;
    for (int i = lane; i < p.width; i += 32) s += x[i] * w[i];
    s = warp_sum(s);
    if (lane == 0) lg[e] = s;
  }
  __syncthreads();
  if (warp == 0) {
    float sc[kRtLane];
#pragma unroll
    for (int s = 0; s < kRtLane; ++s) sc[s] = s * 32 + lane < E ? lg[s * 32 + lane] : 0.f;
    route_token(p, t, lane, sc, lg + E);
  }
  router_ticket(p);
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
    p.slot_w[pairs + t] = 1.f;
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
#pragma unroll
    for (int j = 0; j < 8; ++j) v[0][j] = (DUAL ? silu_f(v[0][j]) * v[D - 1][j] : v[0][j]) * ws;
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
      const float v = DUAL ? g / (1.f + expf(-g)) * acc[D - 1][i][j] : g;
      reinterpret_cast<float*>(p.out)[(size_t)(row0 + r) * p.ldo + n] = v * (p.slot_w ? p.slot_w[row0 + r] : 1.f);
    }
}

template <typename T, int MT>
static int launch_router(const RfMoeRouter* a, int splits, cudaStream_t s) {
  const size_t smem = (size_t)(16 * MT + 8) * a->experts * sizeof(float);
  RF_ALLOW_SMEM_PER_DEVICE((moe_router_kernel<T, MT>), 128 * 1024);
  RF_CUDA_CHECK(::rf::launch_k(moe_router_kernel<T, MT>, dim3(ceil_div(a->rows, 16 * MT), 1, splits), dim3(256), smem, s, splits, *a));
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
  if (a->tile_rows <= 16) return a->dual ? launch_small<T, 1, true, 8, 4>(a, s) : launch_small<T, 1, false, 4, 8>(a, s);
  return a->dual ? launch_small<T, 2, true, 8, 4>(a, s) : launch_small<T, 2, false, 4, 8>(a, s);
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
  return RF_OK;
}

}  // namespace rf

using namespace rf;

extern "C" int rf_moe_router(const RfMoeRouter* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  int rc = check_router(a);
  if (rc) return rc;
  RF_REQUIRE(a->w, "moe_router: weights");
  if (a->rows == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (a->dtype == kF32) {
    RF_CUDA_CHECK(::rf::launch_k(moe_router_f32_kernel, dim3(a->rows), dim3(256), 2 * a->experts * sizeof(float), s, 1, *a));
    ::rf::count_launch();
    return RF_OK;
  }
  // few tokens: the width is split over clusters of eight CTAs; many: 64 tokens share one pass over the router's weights
  const bool many = a->rows > 1024;
  const int tiles = ceil_div(a->rows, 16), splits = many || a->width < 512 ? 1 : (tiles > 32 ? 2 : (tiles > 16 ? 4 : 8));
  if (a->dtype == kF16) return many ? launch_router<__half, 4>(a, 1, s) : launch_router<__half, 1>(a, splits, s);
  return many ? launch_router<__nv_bfloat16, 4>(a, 1, s) : launch_router<__nv_bfloat16, 1>(a, splits, s);
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
