// HGRN2 linear attention: one gate per key channel sets how much of the state is kept and, as its complement, how much is added,
//   S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T,   o_t = S_t^T q_t,
// with an fp32 state per (slot, head), q = silu(.), f = lower + (1 - lower) sigmoid(. + bias), and an RMSNorm per head on o.
//   * rf_hgrn2_recurrent: token by token (decode steps, short portions, everything in fp32),
//   * rf_hgrn2_chunked: block by block on the tensor cores (prefill-sized portions).
#include "../common/dtype.cuh"
#include "../common/host_util.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"
#include "../common/status.h"
#include "../rf_api.h"

namespace rf {

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.f / (1.f + expf(-x)); }
// for inputs that were rounded to 16 bits: a few ulp, on the special-function unit
__device__ __forceinline__ float sigmoid_fast(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
template <typename T> __device__ __forceinline__ float sigmoid_t(float x) {
  if constexpr (sizeof(T) == 4) return sigmoid_f32(x);
  else return sigmoid_fast(x);
}

// One CTA owns `cols` state columns (value channels) of one head of one sequence; thread = (column, row group), RPT state rows
// per thread in registers (RPT = 0: the state stays in global memory, any head size).  When the value channels of a head are
// split over several CTAs they form a cluster and exchange the sums of squares of the head norm.
template <typename T, int RPT>
__global__ void __launch_bounds__(RPT == 64 ? 512 : 1024) hgrn2_recurrent_kernel(const RfHgrn2 p, int cols, int col_tiles) {
  pdl_prologue();
  extern __shared__ float sm[];
  const int groups = blockDim.x / cols, col = threadIdx.x % cols, rg = threadIdx.x / cols;
  float* sq = sm;                              // [2][dim]
  float* sf = sq + 2 * p.dim;                  // [2][dim]
  float* red = sf + 2 * p.dim;                 // [groups][cols]
  float* wsum = red + groups * cols;           // [2][32] warp sums
  float* csum = wsum + 64;                     // [2] this CTA's sum of squares, read by its cluster
  const int head = blockIdx.y, seq = blockIdx.x, j = blockIdx.z * cols + col;
  const bool on = j < p.vdim;
  const int q0 = p.rows.q_start ? p.rows.q_start[seq] : seq, n = p.rows.q_len ? p.rows.q_len[seq] : 1;
  const int slot = p.rows.slot ? p.rows.slot[seq] : seq;
  const bool fresh = p.rows.pos[q0] == 0;
  float* S = p.state + ((size_t)slot * p.heads + head) * p.dim * p.vdim;
  const T* x = reinterpret_cast<const T*>(p.x);
  T* out = reinterpret_cast<T*>(p.out);
  const int per = RPT > 0 ? RPT : (p.dim + groups - 1) / groups, row0 = rg * per;
  constexpr int NR = RPT > 0 ? RPT : 1;
  float st[NR];
  if constexpr (RPT > 0) {
#pragma unroll
    for (int r = 0; r < RPT; ++r) st[r] = (on && row0 + r < p.dim) ? __ldcs(S + (size_t)(row0 + r) * p.vdim + j) : 0.f;
    if (fresh) {                               // checked after the loads are in flight
#pragma unroll
      for (int r = 0; r < RPT; ++r) st[r] = 0.f;
    }
  }
  const float nw = (p.norm_w && on) ? p.norm_w[j] : 1.f;
  for (int t = 0; t < n; ++t) {
    const int buf = t & 1;
    const T* xr = x + (size_t)(q0 + t) * p.ldx;
    for (int i = threadIdx.x; i < p.dim; i += blockDim.x) {
      const int ch = head * p.dim + i;
      const float qv = Num<T>::to_f(xr[ch]);
      sq[buf * p.dim + i] = qv * sigmoid_t<T>(qv);
      const float lo = p.lower[ch];
      sf[buf * p.dim + i] = lo + (1.f - lo) * sigmoid_t<T>(Num<T>::to_f(xr[p.f_off + ch]) + p.f_bias[ch]);
    }
    const float v = on ? Num<T>::to_f(xr[p.v_off + head * p.vdim + j]) : 0.f;
    __syncthreads();
    const float* fq = sq + buf * p.dim;
    const float* ff = sf + buf * p.dim;
    float part = 0.f;
    if constexpr (RPT > 0) {
#pragma unroll
      for (int r = 0; r < RPT; ++r) {
        const bool in = row0 + r < p.dim;
        const float f = in ? ff[row0 + r] : 1.f;
        st[r] = f * st[r] + (1.f - f) * v;
        part = fmaf(st[r], in ? fq[row0 + r] : 0.f, part);
      }
    } else if (on) {
      for (int r = row0; r < min(p.dim, row0 + per); ++r) {
        const float f = ff[r], old = (fresh && t == 0) ? 0.f : S[(size_t)r * p.vdim + j];
        const float s = f * old + (1.f - f) * v;
        S[(size_t)r * p.vdim + j] = s;
        part = fmaf(s, fq[r], part);
      }
    }
    red[rg * cols + col] = part;
    __syncthreads();
    float o = 0.f;
    for (int g = 0; g < groups; ++g) o += red[g * cols + col];
    if (p.norm_w) {
      // every row group holds the same o: sum over the columns of group 0's warps
      const float s = warp_sum(rg == 0 && on ? o * o : 0.f);
      float* ws = wsum + buf * 32;
      if ((threadIdx.x & 31) == 0) ws[threadIdx.x >> 5] = s;
      __syncthreads();
      float tot = 0.f;
      for (int w = 0; w < cols / 32; ++w) tot += ws[w];        // row group 0's warps
      if (col_tiles > 1) {
        if (threadIdx.x == 0) csum[buf] = tot;
        cluster_sync_all();
        tot = 0.f;
        for (int c = 0; c < col_tiles; ++c) tot += ld_dsmem_f32(dsmem_addr(smem_u32(csum + buf), (uint32_t)c));
      }
      o *= rsqrtf(tot / (float)p.vdim_true + p.eps) * nw;
    }
    if (rg == 0 && on) out[(size_t)(q0 + t) * p.ldo + head * p.vdim + j] = Num<T>::from_f(o);
  }
  if constexpr (RPT > 0) {
    if (on) {
#pragma unroll
      for (int r = 0; r < RPT; ++r)
        if (row0 + r < p.dim) __stcs(S + (size_t)(row0 + r) * p.vdim + j, st[r]);
    }
  }
  if (col_tiles > 1) cluster_sync_all();       // no CTA leaves while its sum may still be read
}

template <typename T>
static int launch_recurrent(const RfHgrn2* a, cudaStream_t s) {
  // up to 128 columns per CTA; eight CTAs at most share a head (portable cluster size)
  int cols = std::min(128, round_up(a->vdim, 32)), tiles = ceil_div(a->vdim, cols);
  while (tiles > 8 && cols < 1024) {
    cols *= 2;
    tiles = ceil_div(a->vdim, cols);
  }
  RF_REQUIRE(tiles <= 8, "hgrn2: value heads of %d are too wide", a->vdim);
  int threads = 0, rpt = 0;
  static const int sizes[] = {4, 8, 16, 32, 64};
  for (int r : sizes) {
    const int t = cols * ceil_div(a->dim, r);
    if (t <= (r <= 32 ? 1024 : 512)) { rpt = r; threads = t; break; }
  }
  if (!rpt) threads = cols * std::max(1, std::min(512 / cols, ceil_div(a->dim, 8)));
  const int groups = threads / cols;
  const size_t smem = ((size_t)4 * a->dim + (size_t)groups * cols + 64 + 8) * sizeof(float);
  RF_REQUIRE(smem <= 48 * 1024, "hgrn2: heads of %d do not fit", a->dim);
  const dim3 grid(a->rows.num_seqs, a->heads, tiles);
#define RF_HG(N) RF_CUDA_CHECK(::rf::launch_k(hgrn2_recurrent_kernel<T, N>, grid, dim3(threads), smem, s, tiles, *a, cols, tiles))
  switch (rpt) {
    case 4: RF_HG(4); break;
    case 8: RF_HG(8); break;
    case 16: RF_HG(16); break;
    case 32: RF_HG(32); break;
    case 64: RF_HG(64); break;
    default: RF_HG(0); break;
  }
#undef RF_HG
  ::rf::count_launch();
  return RF_OK;
}

// ------------------------------------------------------- one token per sequence ----
// A decode step reads and writes every state once, so it is a copy with a little arithmetic.  Persistent CTAs walk over the
// (sequence, head) states: a ring of three shared-memory buffers keeps bulk loads of the next states and the bulk store of the
// last one in flight while one is updated in place; the row of a state's token is fetched one state ahead.
constexpr int kHdThreads = 512, kHdRing = 3;

struct Hgrn2DecodeGeom {
  int quads, groups;                     // 4-column groups per state row, rows updated side by side
  uint32_t bytes, sq, sf, red, wsum, bar, total;
};
__host__ __device__ inline Hgrn2DecodeGeom hgrn2_decode_geom(int dim, int vdim) {
  Hgrn2DecodeGeom g;
  g.quads = vdim / 4;
  g.groups = kHdThreads / g.quads;
  g.bytes = (uint32_t)dim * vdim * 4;
  uint32_t o = kHdRing * g.bytes;
  g.sq = o; o += dim * 4;
  g.sf = o; o += dim * 4;
  g.red = o; o += g.groups * vdim * 4;
  g.wsum = o; o += 32 * 4;
  o = (o + 15) & ~15u;
  g.bar = o; o += kHdRing * 8;
  g.total = o;
  return g;
}

template <typename T>
__global__ void __launch_bounds__(kHdThreads) hgrn2_decode_kernel(const RfHgrn2 p) {
  pdl_launch_dependents();
  extern __shared__ __align__(128) uint8_t dsm[];
  const Hgrn2DecodeGeom G = hgrn2_decode_geom(p.dim, p.vdim);
  float* sq = reinterpret_cast<float*>(dsm + G.sq);
  float* sf = reinterpret_cast<float*>(dsm + G.sf);
  float* red = reinterpret_cast<float*>(dsm + G.red);
  float* wsum = reinterpret_cast<float*>(dsm + G.wsum);
  uint64_t* full = reinterpret_cast<uint64_t*>(dsm + G.bar);
  const int tid = threadIdx.x, items = p.rows.num_seqs * p.heads, step = gridDim.x;
  const int quad = tid % G.quads, rg = tid / G.quads;      // rg >= groups: no state rows
  const T* x = reinterpret_cast<const T*>(p.x);
  T* out = reinterpret_cast<T*>(p.out);
  const size_t per_head = (size_t)p.dim * p.vdim;
  auto state_of = [&](int item) {
    const int seq = item / p.heads, slot = p.rows.slot ? p.rows.slot[seq] : seq;
    return p.state + ((size_t)slot * p.heads + item % p.heads) * per_head;
  };
  if (tid == 0) {
    for (int s = 0; s < kHdRing; ++s) mbar_init(&full[s], 1);
    fence_barrier_init();
  }
  __syncthreads();
  pdl_wait();
  int loaded = 0;                        // thread 0: states whose load was issued
  auto load_state = [&](int item, int stage) {
    mbar_arrive_expect_tx(&full[stage], G.bytes);
    bulk_load_1d(dsm + stage * G.bytes, state_of(item), G.bytes, &full[stage]);
    ++loaded;
  };
  if (tid == 0) {
    if (blockIdx.x < items) load_state(blockIdx.x, 0);
    if (blockIdx.x + step < items) load_state(blockIdx.x + step, 1);
  }
  // the token row of one state: this thread's channel of q and f, its four values, and whether the sequence starts here
  float rq = 0.f, rf = 0.f, lo = 1.f, fb = 0.f;
  float4 rv = make_float4(0.f, 0.f, 0.f, 0.f);
  bool fresh = false;
  auto fetch = [&](int item) {
    const int seq = item / p.heads, head = item % p.heads;
    const T* xr = x + (size_t)seq * p.ldx;
    if (tid < p.dim) {
      const int ch = head * p.dim + tid;
      rq = Num<T>::to_f(xr[ch]);
      rf = Num<T>::to_f(xr[p.f_off + ch]);
      lo = p.lower[ch];
      fb = p.f_bias[ch];
    }
    const T* vr = xr + p.v_off + head * p.vdim + quad * 4;
    rv = make_float4(Num<T>::to_f(vr[0]), Num<T>::to_f(vr[1]), Num<T>::to_f(vr[2]), Num<T>::to_f(vr[3]));
    fresh = p.rows.pos[seq] == 0;
  };
  if (blockIdx.x < items) fetch(blockIdx.x);

  bool ok = true;
  for (int item = blockIdx.x, it = 0; item < items; item += step, ++it) {
    const int stage = it % kHdRing;
    if (tid < p.dim) {
      sq[tid] = rq * sigmoid_t<T>(rq);
      sf[tid] = lo + (1.f - lo) * sigmoid_t<T>(rf + fb);
    }
    const float4 v = rv;
    const bool start = fresh;
    if (item + step < items) fetch(item + step);
    const bool have = mbar_wait(&full[stage], (uint32_t)(it / kHdRing) & 1u);
    if (__syncthreads_or(!have)) {
      ok = false;
      if (tid == 0) report_status(p.status, kStatusTmaTimeout, kTagHgrn2, item);
      break;
    }
    float4 part = make_float4(0.f, 0.f, 0.f, 0.f);
    if (rg < G.groups) {
      float4* S = reinterpret_cast<float4*>(dsm + stage * G.bytes) + quad;
#pragma unroll 4
      for (int r = rg; r < p.dim; r += G.groups) {
        const float f = sf[r], w = 1.f - f, q = sq[r];
        float4 s = S[(size_t)r * G.quads];
        if (start) s = make_float4(0.f, 0.f, 0.f, 0.f);
        s.x = f * s.x + w * v.x; s.y = f * s.y + w * v.y; s.z = f * s.z + w * v.z; s.w = f * s.w + w * v.w;
        S[(size_t)r * G.quads] = s;
        part.x = fmaf(s.x, q, part.x); part.y = fmaf(s.y, q, part.y); part.z = fmaf(s.z, q, part.z); part.w = fmaf(s.w, q, part.w);
      }
      *reinterpret_cast<float4*>(red + rg * p.vdim + quad * 4) = part;
    }
    fence_proxy_async();
    __syncthreads();
    if (tid == 0) {
      bulk_store_1d(state_of(item), dsm + stage * G.bytes, G.bytes);
      bulk_commit_group();
      if (item + 2 * step < items) {
        bulk_wait_read_1();              // the store before this one has left its buffer
        load_state(item + 2 * step, (it + 2) % kHdRing);
      }
    }
    const int seq = item / p.heads, head = item % p.heads;
    float o = 0.f;
    if (tid < p.vdim)
      for (int g = 0; g < G.groups; ++g) o += red[g * p.vdim + tid];
    const float ss = warp_sum(o * o);
    if ((tid & 31) == 0) wsum[tid >> 5] = ss;
    __syncthreads();
    if (tid < p.vdim) {
      float r = 1.f;
      if (p.norm_w) {
        float tot = 0.f;
        for (int w = 0; w < (p.vdim + 31) / 32; ++w) tot += wsum[w];
        r = rsqrtf(tot / (float)p.vdim_true + p.eps) * p.norm_w[tid];
      }
      out[(size_t)seq * p.ldo + head * p.vdim + tid] = Num<T>::from_f(o * r);
    }
  }
  if (tid == 0) {
    if (!ok) {                           // let every load that was issued land before the CTA exits
      for (int s = max(0, loaded - kHdRing); s < loaded; ++s) mbar_wait(&full[s % kHdRing], (uint32_t)(s / kHdRing) & 1u, 20ull * 1000 * 1000);
    }
    bulk_wait_all();
  }
}

static bool hgrn2_decode_eligible(const RfHgrn2* a) {
  return !a->rows.q_start && a->dim <= kHdThreads && a->vdim <= kHdThreads && a->vdim % 4 == 0 &&
         hgrn2_decode_geom(a->dim, a->vdim).total <= 220 * 1024;
}

template <typename T>
static int launch_decode(const RfHgrn2* a, cudaStream_t s) {
  const Hgrn2DecodeGeom g = hgrn2_decode_geom(a->dim, a->vdim);
  RF_ALLOW_SMEM_PER_DEVICE(hgrn2_decode_kernel<T>, 220 * 1024);
  const int per_sm = std::max(1, std::min(4, (int)(227 * 1024 / (g.total + 1024))));
  const int grid = std::min(a->rows.num_seqs * a->heads, per_sm * sm_count());
  RF_CUDA_CHECK(::rf::launch_k(hgrn2_decode_kernel<T>, dim3(grid), dim3(kHdThreads), g.total, s, 1, *a));
  ::rf::count_launch();
  return RF_OK;
}

// ------------------------------------------------------- block form (prefill) ----
// Sixteen tokens per step.  With G_t the product of the gates from the block's start to t (inclusive), E_t the product of the
// gates behind t to the block's end and S the state ahead of the block:
//     O = (q * G) S + tril(P) V,   P[t, s] = sum_c q_t[c] (1 - f_s[c]) prod_{s < r <= t} f_r[c]
//     S' = G_last * S + ((1 - f) * E)^T V
// Every factor is a product of gates in [0, 1], built by running products: no logarithms, no exponentials of differences, and
// nothing can overflow however fast a channel forgets.  P is evaluated in fp32 on the CUDA cores (its cost does not grow with
// the sequence), the three matrix products run on the tensor cores with their fp32 operands as bf16 pairs (value + remainder,
// about 16 mantissa bits; the values V are bf16 already).  The transposed state lives in the accumulator registers of the
// warps - 16 value channels x a share of the key channels each - where the product with it reads it as an operand.
// A CTA owns VG * 16 value channels of one head of one sequence; the CTAs of a head form a cluster that exchanges the sums of
// squares of the head norm one step behind the computation.
constexpr int kHcTok = 16, kHcThreads = 256, kHcWarps = 8, kHcRing = 4;

// Shared memory of a CTA with DP (padded) key channels and VT value channels, in bytes from the base.
template <int DP, int VT> struct Hgrn2Geom {
  static constexpr int kRawLd = 2 * DP + VT + 8, kQLd = DP + 4, kBLd = DP + 8, kPLd = 24, kOLd = VT + 4;
  static constexpr int kDG = kHcWarps / (VT / 16);
  static constexpr int raw = 0;                                   // [ring][16] rows q | f | v as they come
  static constexpr int sq = raw + kHcRing * kHcTok * kRawLd * 2;  // [16][DP] silu(q), gates
  static constexpr int sf = sq + kHcTok * kQLd * 4;
  static constexpr int qh = sf + kHcTok * kQLd * 4;               // bf16 pairs of q * G and (1 - f) * E
  static constexpr int ql = qh + kHcTok * kBLd * 2;
  static constexpr int kh = ql + kHcTok * kBLd * 2;
  static constexpr int kl = kh + kHcTok * kBLd * 2;
  static constexpr int gt = kl + kHcTok * kBLd * 2;               // gate product of the whole block
  static constexpr int ph = gt + DP * 4;
  static constexpr int pl = ph + kHcTok * kPLd * 2;
  static constexpr int so = pl + kHcTok * kPLd * 2;               // [warps of a value group][16][VT] partial outputs
  static constexpr int csum = so + kDG * kHcTok * kOLd * 4;
  static constexpr int total = csum + 2 * 8 * kHcTok * 4;         // [2][cluster rank][16]
};

__device__ __forceinline__ void hc_cp16(uint32_t dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void hc_split(float v, __nv_bfloat16& hi, __nv_bfloat16& lo) {
  hi = __float2bfloat16_rn(v);
  lo = __float2bfloat16_rn(v - __bfloat162float(hi));
}
// value and remainder of two floats, packed
__device__ __forceinline__ void hc_split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<uint32_t*>(&h);
  lo = *reinterpret_cast<uint32_t*>(&l);
}

// VG: groups of 16 value channels per CTA; the 8 / VG warps of a group share its key channels, DT 16-channel tiles each.
template <int VG, int DP>
__global__ void __launch_bounds__(kHcThreads, DP == 256 ? 1 : 2) hgrn2_chunked_kernel(const RfHgrn2 p, int col_tiles) {
  pdl_prologue();
  using T = __nv_bfloat16;
  constexpr int VT = VG * 16, DG = kHcWarps / VG, NV = VT / 16, DT = DP / 16 / DG;
  using L = Hgrn2Geom<DP, VT>;
  extern __shared__ __align__(16) uint8_t csm[];
  T* raw = reinterpret_cast<T*>(csm + L::raw);
  float* sq = reinterpret_cast<float*>(csm + L::sq);
  float* sf = reinterpret_cast<float*>(csm + L::sf);
  T* qh = reinterpret_cast<T*>(csm + L::qh);
  T* ql = reinterpret_cast<T*>(csm + L::ql);
  T* kh = reinterpret_cast<T*>(csm + L::kh);
  T* kl = reinterpret_cast<T*>(csm + L::kl);
  float* gt = reinterpret_cast<float*>(csm + L::gt);
  T* ph = reinterpret_cast<T*>(csm + L::ph);
  T* pl = reinterpret_cast<T*>(csm + L::pl);
  float* so = reinterpret_cast<float*>(csm + L::so);
  float* csum = reinterpret_cast<float*>(csm + L::csum);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q4 = lane & 3;
  const int vg = warp % VG, dg = warp / VG, head = blockIdx.y, seq = blockIdx.x, v0 = blockIdx.z * VT;
  const int q0 = p.rows.q_start[seq], n = p.rows.q_len[seq], slot = p.rows.slot ? p.rows.slot[seq] : seq;
  const bool fresh = p.rows.pos[q0] == 0;
  float* S = p.state + ((size_t)slot * p.heads + head) * p.dim * p.vdim;
  const T* x = reinterpret_cast<const T*>(p.x);
  T* out = reinterpret_cast<T*>(p.out);

  // transposed state: tile j covers key channels (j * DG + dg) * 16 .. + 15 as two accumulator tiles of eight
  float st[DT][8];
#pragma unroll
  for (int j = 0; j < DT; ++j)
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const int d = (j * DG + dg) * 16 + (e >> 2) * 8 + q4 * 2 + (e & 1), v = v0 + vg * 16 + g + ((e >> 1) & 1) * 8;
      st[j][e] = (!fresh && d < p.dim && v < p.vdim) ? S[(size_t)d * p.vdim + v] : 0.f;
    }

  auto prefetch = [&](int b) {
    constexpr int kChunks = (2 * DP + VT) / 8, kAll = kHcTok * kChunks;
    if (b * kHcTok < n) {
#pragma unroll
      for (int k = 0; k < (kAll + kHcThreads - 1) / kHcThreads; ++k) {
        const int i = tid + k * kHcThreads, t = i / kChunks, c = (i % kChunks) * 8, tok = b * kHcTok + t;
        if (i < kAll) {
          int src;
          bool ok = tok < n;
          if (c < DP) { src = head * p.dim + c; ok = ok && c < p.dim; }
          else if (c < 2 * DP) { src = p.f_off + head * p.dim + c - DP; ok = ok && c - DP < p.dim; }
          else { src = p.v_off + head * p.vdim + v0 + c - 2 * DP; ok = ok && v0 + c - 2 * DP < p.vdim; }
          hc_cp16(smem_u32(raw + ((b % kHcRing) * kHcTok + t) * L::kRawLd + c), ok ? x + (size_t)(q0 + tok) * p.ldx + src : x, ok);
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // this thread's share of the gates: two neighbouring key channels of every (512 / DP)-th token
  constexpr int kGateStep = 2 * kHcThreads / DP;
  const int gc = (tid % (DP / 2)) * 2, gtok = tid / (DP / 2);
  float g_lo[2] = {1.f, 1.f}, g_b[2] = {0.f, 0.f};
  if (gc < p.dim) {
    g_lo[0] = p.lower[head * p.dim + gc]; g_lo[1] = p.lower[head * p.dim + gc + 1];
    g_b[0] = p.f_bias[head * p.dim + gc]; g_b[1] = p.f_bias[head * p.dim + gc + 1];
  }
  const int steps = (n + kHcTok - 1) / kHcTok;
  // output of the step before, still to be normalised: token row `orow`, values ov of channels ocol ..
  float ov[NV];
  int orow = -1;
  const int otok = tid >> 4, ocol = (tid & 15) * NV;
  float nw[NV];
#pragma unroll
  for (int i = 0; i < NV; ++i) nw[i] = (p.norm_w && v0 + ocol + i < p.vdim) ? p.norm_w[v0 + ocol + i] : 1.f;
  auto finish = [&](int buf, float own) {
    float tot = own;
    if (col_tiles > 1) {
      tot = 0.f;
      for (int c = 0; c < col_tiles; ++c) tot += csum[(buf * 8 + c) * kHcTok + otok];
    }
    const int v = v0 + ocol;
    if (orow < 0 || v >= p.vdim) return;
    const float r = p.norm_w ? rsqrtf(tot / (float)p.vdim_true + p.eps) : 1.f;
    T* dst = out + (size_t)orow * p.ldo + head * p.vdim + v;
#pragma unroll
    for (int i = 0; i < NV; i += 2) *reinterpret_cast<uint32_t*>(dst + i) = MmaOp<T>::pack(ov[i] * r * nw[i], ov[i + 1] * r * nw[i + 1]);
  };
  for (int b = 0; b < kHcRing - 1; ++b) prefetch(b);

  for (int b = 0; b < steps; ++b) {
    asm volatile("cp.async.wait_group %0;" ::"n"(kHcRing - 2) : "memory");
    __syncthreads();
    prefetch(b + kHcRing - 1);
    const T* rw = raw + (b % kHcRing) * kHcTok * L::kRawLd;
    const int valid = n - b * kHcTok;
    // ---- gates
#pragma unroll
    for (int k = 0; k < kHcTok / kGateStep; ++k) {
      const int t = gtok + k * kGateStep;
      const float2 z = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(rw + t * L::kRawLd + gc));
      const float2 y = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(rw + t * L::kRawLd + DP + gc));
      const bool in = t < valid && gc < p.dim;
      float2 q, f;
      q.x = in ? z.x * sigmoid_fast(z.x) : 0.f;
      q.y = in ? z.y * sigmoid_fast(z.y) : 0.f;
      f.x = in ? g_lo[0] + (1.f - g_lo[0]) * sigmoid_fast(y.x + g_b[0]) : 1.f;
      f.y = in ? g_lo[1] + (1.f - g_lo[1]) * sigmoid_fast(y.y + g_b[1]) : 1.f;
      *reinterpret_cast<float2*>(sq + t * L::kQLd + gc) = q;
      *reinterpret_cast<float2*>(sf + t * L::kQLd + gc) = f;
    }
    __syncthreads();
    if (warp < 4) {
      // ---- P: source tokens warp, warp + 4, .. of this warp, the lanes over the key channels
      float acc[4 * kHcTok];
#pragma unroll
      for (int i = 0; i < 4 * kHcTok; ++i) acc[i] = 0.f;
      for (int c = lane * 4; c < DP; c += 128) {
        float4 w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 f0 = *reinterpret_cast<const float4*>(sf + (warp + 4 * i) * L::kQLd + c);
          w[i] = make_float4(1.f - f0.x, 1.f - f0.y, 1.f - f0.z, 1.f - f0.w);
        }
#pragma unroll
        for (int t = 0; t < kHcTok; ++t) {
          const float4 f = *reinterpret_cast<const float4*>(sf + t * L::kQLd + c), q = *reinterpret_cast<const float4*>(sq + t * L::kQLd + c);
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if (t >= 4 * i) {                    // source token s = warp + 4 i cannot be later than t otherwise
              const int s = warp + 4 * i;
              if (t > s) { w[i].x *= f.x; w[i].y *= f.y; w[i].z *= f.z; w[i].w *= f.w; }
              if (t >= s) acc[i * kHcTok + t] += fmaf(q.x, w[i].x, fmaf(q.y, w[i].y, fmaf(q.z, w[i].z, q.w * w[i].w)));
            }
          }
        }
      }
      // sum over the lanes: halves of the 64 sums change sides until a lane holds two of them, index lane * 2 (+ 1)
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const bool up = (lane & o) != 0;
#pragma unroll
        for (int i = 0; i < 2 * kHcTok; ++i) {
          if (i < 2 * o) {
            const float send = up ? acc[i] : acc[i + 2 * o], keep = up ? acc[i + 2 * o] : acc[i];
            acc[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
          }
        }
      }
      const int s = warp + 4 * (lane >> 3), t = (lane & 7) * 2;
      hc_split(acc[0], ph[t * L::kPLd + s], pl[t * L::kPLd + s]);
      hc_split(acc[1], ph[(t + 1) * L::kPLd + s], pl[(t + 1) * L::kPLd + s]);
    } else {
      // ---- running products per key channel
      for (int c = tid - 128; c < DP; c += 128) {
        float f[kHcTok], q[kHcTok];
#pragma unroll
        for (int t = 0; t < kHcTok; ++t) { f[t] = sf[t * L::kQLd + c]; q[t] = sq[t * L::kQLd + c]; }
        float G = 1.f, E = 1.f;
#pragma unroll
        for (int t = 0; t < kHcTok; ++t) {
          G *= f[t];
          hc_split(q[t] * G, qh[t * L::kBLd + c], ql[t * L::kBLd + c]);
          const int r = kHcTok - 1 - t;
          hc_split((1.f - f[r]) * E, kh[r * L::kBLd + c], kl[r * L::kBLd + c]);
          E *= f[r];
        }
        gt[c] = G;
      }
    }
    if (b > 0 && col_tiles > 1) {
      __syncwarp();
      asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
      finish((b - 1) & 1, 0.f);
    }
    __syncthreads();
    // ---- tensor cores
    {
      uint32_t va[4];                            // V^T of this warp's value channels (rows) over the sixteen tokens
      ldsm_x4_t(smem_u32(rw + ((lane >> 4) * 8 + (lane & 7)) * L::kRawLd + 2 * DP + vg * 16 + ((lane >> 3) & 1) * 8), va[0], va[1], va[2], va[3]);
      float o[2][4] = {}, o1[2][4] = {}, o2[2][4] = {};      // separate sums: no chain of dependent products
      if (dg == 0) {
        uint32_t bh[4], bl[4];
        const int off = ((lane >> 4) * 8 + (lane & 7)) * L::kPLd + ((lane >> 3) & 1) * 8;
        ldsm_x4(smem_u32(ph + off), bh[0], bh[1], bh[2], bh[3]);
        ldsm_x4(smem_u32(pl + off), bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
        for (int nt = 0; nt < 2; ++nt) {
          MmaOp<T>::mma(o[nt], va, bh[nt * 2], bh[nt * 2 + 1]);
          MmaOp<T>::mma(o[nt], va, bl[nt * 2], bl[nt * 2 + 1]);
        }
      }
#pragma unroll
      for (int j = 0; j < DT; ++j) {
        const int d = (j * DG + dg) * 16;
        {
          uint32_t ah[4], al[4], bh[4], bl[4];
          hc_split2(st[j][0], st[j][1], ah[0], al[0]);
          hc_split2(st[j][2], st[j][3], ah[1], al[1]);
          hc_split2(st[j][4], st[j][5], ah[2], al[2]);
          hc_split2(st[j][6], st[j][7], ah[3], al[3]);
          const int qoff = ((lane >> 4) * 8 + (lane & 7)) * L::kBLd + d + ((lane >> 3) & 1) * 8;      // [token][channel], no transpose
          ldsm_x4(smem_u32(qh + qoff), bh[0], bh[1], bh[2], bh[3]);
          ldsm_x4(smem_u32(ql + qoff), bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
          for (int nt = 0; nt < 2; ++nt) {
            MmaOp<T>::mma(o[nt], ah, bh[nt * 2], bh[nt * 2 + 1]);
            MmaOp<T>::mma(o1[nt], al, bh[nt * 2], bh[nt * 2 + 1]);
            MmaOp<T>::mma(o2[nt], ah, bl[nt * 2], bl[nt * 2 + 1]);
          }
          const int koff = (lane & 15) * L::kBLd + d + (lane >> 4) * 8;                              // transposed: tokens are the k axis
          ldsm_x4_t(smem_u32(kh + koff), bh[0], bh[1], bh[2], bh[3]);
          ldsm_x4_t(smem_u32(kl + koff), bl[0], bl[1], bl[2], bl[3]);
#pragma unroll
          for (int h8 = 0; h8 < 2; ++h8) {
            const float2 G = *reinterpret_cast<const float2*>(gt + d + h8 * 8 + q4 * 2);
            float (&c)[4] = *reinterpret_cast<float (*)[4]>(&st[j][h8 * 4]);
            c[0] *= G.x; c[1] *= G.y; c[2] *= G.x; c[3] *= G.y;
            MmaOp<T>::mma(c, va, bh[h8 * 2], bh[h8 * 2 + 1]);
            MmaOp<T>::mma(c, va, bl[h8 * 2], bl[h8 * 2 + 1]);
          }
        }
      }
      float* dst = so + dg * kHcTok * L::kOLd + vg * 16 + g;
#pragma unroll
      for (int nt = 0; nt < 2; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) dst[(nt * 8 + q4 * 2 + (e & 1)) * L::kOLd + (e >> 1) * 8] = o[nt][e] + (o1[nt][e] + o2[nt][e]);
    }
    __syncthreads();
    // ---- this step's outputs: sixteen threads per token
    {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        float v = 0.f;
#pragma unroll
        for (int k = 0; k < DG; ++k) v += so[(k * kHcTok + otok) * L::kOLd + ocol + i];
        ov[i] = v;
        ss += v * v;
      }
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      orow = otok < valid ? q0 + b * kHcTok + otok : -1;
      if (col_tiles > 1) {
        // lane c of a token's sixteen threads stores the sum into CTA c of the cluster
        if ((tid & 15) < col_tiles)
          st_dsmem_u32(dsmem_addr(smem_u32(csum + ((b & 1) * 8 + (int)cluster_ctarank()) * kHcTok + otok), (uint32_t)(tid & 15)), __float_as_uint(ss));
        __syncwarp();
        asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
      } else {
        finish(0, ss);
      }
    }
  }
  if (col_tiles > 1) {
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
    finish((steps - 1) & 1, 0.f);
  }
#pragma unroll
  for (int j = 0; j < DT; ++j)
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const int d = (j * DG + dg) * 16 + (e >> 2) * 8 + q4 * 2 + (e & 1), v = v0 + vg * 16 + g + ((e >> 1) & 1) * 8;
      if (d < p.dim && v < p.vdim) S[(size_t)d * p.vdim + v] = st[j][e];
    }
}

template <int VG, int DP>
static int launch_chunked_t(const RfHgrn2* a, int tiles, cudaStream_t s) {
  constexpr int smem = Hgrn2Geom<DP, VG * 16>::total;
  RF_ALLOW_SMEM_PER_DEVICE((hgrn2_chunked_kernel<VG, DP>), smem);
  RF_CUDA_CHECK(::rf::launch_k(hgrn2_chunked_kernel<VG, DP>, dim3(a->rows.num_seqs, a->heads, tiles), dim3(kHcThreads), smem, s, tiles, *a, tiles));
  ::rf::count_launch();
  return RF_OK;
}

template <int VG>
static int launch_chunked(const RfHgrn2* a, int tiles, cudaStream_t s) {
  if (a->dim <= 64) return launch_chunked_t<VG, 64>(a, tiles, s);
  if (a->dim <= 128) return launch_chunked_t<VG, 128>(a, tiles, s);
  return launch_chunked_t<VG, 256>(a, tiles, s);
}

}  // namespace rf

using namespace rf;

static int check_hgrn2(const RfHgrn2* a) {
  RF_REQUIRE(a && a->x && a->state && a->out && a->f_bias && a->lower && a->rows.pos, "hgrn2: null argument");
  RF_REQUIRE(a->heads > 0 && a->dim > 0 && a->dim % 8 == 0 && a->vdim > 0 && a->vdim % 8 == 0 && a->vdim_true > 0 &&
                 a->vdim_true <= a->vdim && a->ldx % 8 == 0 && a->ldo % 8 == 0, "hgrn2: head sizes");
  return RF_OK;
}

extern "C" int rf_hgrn2_recurrent(const RfHgrn2* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  int rc = check_hgrn2(a);
  if (rc) return rc;
  if (a->rows.num_seqs == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (hgrn2_decode_eligible(a)) {
    if (a->dtype == kF32) return launch_decode<float>(a, s);
    if (a->dtype == kF16) return launch_decode<__half>(a, s);
    return launch_decode<__nv_bfloat16>(a, s);
  }
  if (a->dtype == kF32) return launch_recurrent<float>(a, s);
  if (a->dtype == kF16) return launch_recurrent<__half>(a, s);
  return launch_recurrent<__nv_bfloat16>(a, s);
}

extern "C" int rf_hgrn2_chunked_supported(int dim, int vdim, int dtype) {
  return dtype == kBF16 && dim > 0 && dim <= 256 && vdim > 0 && vdim <= 1024;
}

extern "C" int rf_hgrn2_chunked(const RfHgrn2* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  int rc = check_hgrn2(a);
  if (rc) return rc;
  if (!rf_hgrn2_chunked_supported(a->dim, a->vdim, a->dtype)) return rf_hgrn2_recurrent(a, stream);
  RF_REQUIRE(a->rows.q_start && a->rows.q_len, "hgrn2: the block form works on portions");
  if (a->rows.num_seqs == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  // value channels per CTA: as few as still share a head between at most eight CTAs, more once the GPU is full
  int vt = a->vdim <= 32 ? 32 : a->vdim <= 64 ? 64 : 128;
  for (int t : {32, 64}) {
    const int tiles = ceil_div(a->vdim, t);
    if (tiles <= 8 && (long)a->rows.num_seqs * a->heads * tiles <= sm_count()) { vt = std::min(vt, t); break; }
  }
  const int tiles = ceil_div(a->vdim, vt);
  if (vt == 32) return launch_chunked<2>(a, tiles, s);
  if (vt == 64) return launch_chunked<4>(a, tiles, s);
  return launch_chunked<8>(a, tiles, s);
}
