// Selective scan (Mamba) layers: causal convolution with carried inputs, the token-by-token recurrence with its step-size
// projection (decode rows and short portions), and the tiled scan of prefill-sized portions.
//
// The state of a channel is a short fp32 vector.  Four neighbouring lanes hold one channel, each lane every fourth quad of its
// states, so that a warp reads and writes the states of eight channels as whole lines.
#include "../common/dtype.cuh"
#include "../common/host_util.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"
#include "../rf_api.h"

namespace rf {

template <typename T> __device__ __forceinline__ float exp2_t(float x);
template <> __device__ __forceinline__ float exp2_t<float>(float x) { return exp2f(x); }
template <> __device__ __forceinline__ float exp2_t<__half>(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <> __device__ __forceinline__ float exp2_t<__nv_bfloat16>(float x) { return exp2_t<__half>(x); }

// log(1 + exp(v)) = max(v, 0) + log1p(exp(-|v|)); in 16-bit models the second term comes from the special-function units, and
// from the first terms of the series where 1 + e would drop the digits of e.
template <typename T> __device__ __forceinline__ float softplus_t(float v) {
  const float e = __expf(-fabsf(v));
  const float series = e * (1.f - e * (0.5f - e * (1.f / 3.f - e * (0.25f - e * 0.2f))));
  return fmaxf(v, 0.f) + (e < 0.0625f ? series : __logf(1.f + e));
}
template <> __device__ __forceinline__ float softplus_t<float>(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
template <typename T> __device__ __forceinline__ float silu_t(float v) { return silu_f(v); }
template <> __device__ __forceinline__ float silu_t<float>(float v) { return v / (1.f + expf(-v)); }

__device__ __forceinline__ void zero8(float (&f)[8]) {
#pragma unroll
  for (int j = 0; j < 8; ++j) f[j] = 0.f;
}

// --------------------------------------------------------------------------------------- causal convolution ----
// A thread owns eight channels over `tile` consecutive rows of one sequence; the thread of the first rows also replaces the
// carried inputs.  TAPS = 0: any number of taps, every input read again for each of them.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) conv_silu_kernel(const RfConvSilu p, int tile) {
  pdl_prologue();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8, seq = blockIdx.z;
  const int q0 = p.rows.q_start ? p.rows.q_start[seq] : seq, n = p.rows.q_len ? p.rows.q_len[seq] : 1;
  const int t0 = blockIdx.y * tile, t1 = min(n, t0 + tile), taps = TAPS > 0 ? TAPS : p.taps, past = taps - 1;
  if (c >= p.channels || t0 >= n) return;
  T* state = reinterpret_cast<T*>(p.state) + (size_t)(p.rows.slot ? p.rows.slot[seq] : seq) * (p.ring ? taps : past) * p.channels + c;
  const int pos0 = p.rows.pos[q0];
  auto carried = [&](int i) -> T* { return state + (size_t)(p.ring ? (pos0 + i) % taps : past + i) * p.channels; };   // input at place i < 0
  const T* x = reinterpret_cast<const T*>(p.x) + (size_t)q0 * p.ldx + c;
  T* y = reinterpret_cast<T*>(p.y) + (size_t)q0 * p.ldy + c;
  // input at place i of this launch's rows; negative places are carried ones
  auto input = [&](int i, float (&f)[8]) {
    if (i >= 0) load8(x + (size_t)i * p.ldx, f);
    else if (pos0 + i >= 0) load8(carried(i), f);
    else zero8(f);
  };
  float bias[8];
  zero8(bias);
  if (p.bias) load8(p.bias + c, bias);
  if constexpr (TAPS > 0) {
    float w[TAPS][8], win[TAPS][8];
#pragma unroll
    for (int k = 0; k < TAPS; ++k) load8(p.w + (size_t)k * p.channels + c, w[k]);
#pragma unroll
    for (int k = 0; k < TAPS - 1; ++k) input(t0 - (TAPS - 1) + k, win[k]);
#pragma unroll 4
    for (int t = t0; t < t1; ++t) {
      load8(x + (size_t)t * p.ldx, win[TAPS - 1]);
      float a[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        a[j] = bias[j];
#pragma unroll
        for (int k = 0; k < TAPS; ++k) a[j] += w[k][j] * win[k][j];
        a[j] = p.add ? win[TAPS - 1][j] + a[j] : silu_t<T>(a[j]);
      }
      store8(y + (size_t)t * p.ldy, a);
#pragma unroll
      for (int k = 0; k < TAPS - 1; ++k)
#pragma unroll
        for (int j = 0; j < 8; ++j) win[k][j] = win[k + 1][j];
    }
  } else {
    for (int t = t0; t < t1; ++t) {
      float a[8], w[8], v[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] = bias[j];
      for (int k = 0; k < taps; ++k) {
        load8(p.w + (size_t)k * p.channels + c, w);
        input(t - past + k, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) a[j] += w[j] * v[j];
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) a[j] = p.add ? v[j] + a[j] : silu_t<T>(a[j]);      // v: the row itself, the last tap's input
      store8(y + (size_t)t * p.ldy, a);
    }
  }
  if (blockIdx.y == 0)
    for (int i = 0; i < past; ++i) {             // ascending: row i comes from a later row of the old state, or from this launch
      const int at = n - past + i;
      if (p.ring && at < 0) continue;            // stays where it is
      float v[8];
      input(at, v);
      store8(p.ring ? state + (size_t)((pos0 + at) % taps) * p.channels : state + (size_t)i * p.channels, v);
    }
}

// ------------------------------------------------------------------------------------------- recurrence ----
constexpr int kMbChannels = 64;       // channels per CTA (256 threads)
constexpr int kMbRows = 8;            // rows staged in shared memory at a time

// Shared memory of a CTA: operands of eight rows for its 64 channels, and what the step-size product needs (16-bit models: the
// inputs of the rows and the two halves of the product; 32-bit models: inputs and the weights of the channels).
template <typename T, int QPL>
struct MbTile {
  static constexpr int CH = kMbChannels, SP = 16 * QPL;             // SP: states per channel in shared memory, zero padded
  static constexpr bool kMma = sizeof(T) == 2;
  int rank_p, wp;
  T* in;              // [rows][wp] step-size inputs
  float* pre;         // [2][rows][CH] halves of the product (16 bits)
  T* w;               // [CH][wp] (32 bits)
  float* b; float* c; // [rows][SP]
  float* x; float* z; // [rows][CH]; x is replaced by the result
  __device__ __forceinline__ MbTile(uint8_t* raw, int rank) {
    rank_p = (rank + 31) & ~31; wp = rank_p + 8;
    in = reinterpret_cast<T*>(raw);
    pre = reinterpret_cast<float*>(in + kMbRows * wp);
    b = pre + (kMma ? 2 * kMbRows * CH : 0);
    c = b + kMbRows * SP;
    x = c + kMbRows * SP;
    z = x + kMbRows * CH;
    w = reinterpret_cast<T*>(z + kMbRows * CH);
  }
  static size_t bytes(int rank) {
    const int rank_p = (rank + 31) & ~31, wp = rank_p + 8;
    return (size_t)kMbRows * wp * sizeof(T) + ((size_t)(kMma ? 2 * kMbRows * CH : 0) + 2 * kMbRows * (SP + CH)) * sizeof(float) +
           (kMma ? 0 : (size_t)CH * wp * sizeof(T));
  }
  // padding columns to zero, and in 32 bits the weights: nothing of this depends on the previous kernel
  __device__ __forceinline__ void prepare(const RfMamba1& p, int c0) {
    const float zero[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    for (int i = threadIdx.x; i < kMbRows * wp / 8; i += 256) store8(in + i * 8, zero);
    for (int i = threadIdx.x; i < 2 * kMbRows * SP; i += 256) b[i] = 0.f;
    if constexpr (!kMma) {
      for (int i = threadIdx.x; i < CH * (wp / 8); i += 256) {
        const int r = i / (wp / 8), k = (i % (wp / 8)) * 8;
        float f[8];
        zero8(f);
        if (c0 + r < p.inner && k < p.rank) load8(reinterpret_cast<const T*>(p.w_dt) + (size_t)(c0 + r) * p.rank + k, f);
        store8(w + (size_t)r * wp + k, f);
      }
    }
  }
  // operands of rows r0 .. r0 + nr - 1
  __device__ __forceinline__ void stage(const RfMamba1& p, int c0, int r0, int nr) {
    for (int i = threadIdx.x; i < nr * (p.rank / 8); i += 256) {
      const int r = i / (p.rank / 8), k = (i % (p.rank / 8)) * 8;
      *reinterpret_cast<Vec8<T>*>(in + r * wp + k) = *reinterpret_cast<const Vec8<T>*>(reinterpret_cast<const T*>(p.bc) + (size_t)(r0 + r) * p.ld_bc + k);
    }
    for (int i = threadIdx.x; i < nr * (p.states / 4); i += 256) {          // B and C: states / 8 pieces each
      const int r = i / (p.states / 4), k = (i % (p.states / 4)) * 8;
      const bool is_c = k >= p.states;
      float f[8];
      load8(reinterpret_cast<const T*>(p.bc) + (size_t)(r0 + r) * p.ld_bc + p.rank + k, f);
      store8((is_c ? c : b) + r * SP + (is_c ? k - p.states : k), f);
    }
    for (int i = threadIdx.x; i < nr * (CH / 8) * 2; i += 256) {
      const int zi = i & 1, r = (i >> 1) / (CH / 8), k = ((i >> 1) % (CH / 8)) * 8;
      float f[8];
      zero8(f);
      if (c0 + k < p.inner) load8((zi ? reinterpret_cast<const T*>(p.z) + (size_t)(r0 + r) * p.ldz : reinterpret_cast<const T*>(p.x) + (size_t)(r0 + r) * p.ldx) + c0 + k, f);
      store8((zi ? z : x) + r * CH + k, f);
    }
  }
  // 16 bits: step sizes of the staged rows on mma.sync - channels on the M axis, rows on the N axis, eight warps as four channel
  // tiles times two halves of the rank, weights straight from L2 into the fragments (a lane's eight consecutive columns)
  __device__ __forceinline__ void project(const RfMamba1& p, int c0) {
    if constexpr (kMma) {
      const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3, mt = warp & 3, half = warp >> 2;
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
      const T* w0 = reinterpret_cast<const T*>(p.w_dt) + (size_t)(c0 + mt * 16 + g) * p.rank;
      const bool in0 = c0 + mt * 16 + g < p.inner, in1 = c0 + mt * 16 + g + 8 < p.inner;
      const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
#pragma unroll 4
      for (int kb = half; kb < rank_p / 32; kb += 2) {
        const int k = kb * 32 + q * 8;
        const uint4 a0 = in0 && k < p.rank ? *reinterpret_cast<const uint4*>(w0 + k) : zero;
        const uint4 a1 = in1 && k < p.rank ? *reinterpret_cast<const uint4*>(w0 + (size_t)8 * p.rank + k) : zero;
        const uint4 bb = *reinterpret_cast<const uint4*>(in + g * wp + k);
        const uint32_t lo[4] = {a0.x, a1.x, a0.y, a1.y}, hi[4] = {a0.z, a1.z, a0.w, a1.w};
        MmaOp<T>::mma(acc, lo, bb.x, bb.y);
        MmaOp<T>::mma(acc, hi, bb.z, bb.w);
      }
      float* o = pre + half * kMbRows * CH + mt * 16 + g;
      o[(q * 2) * CH] = acc[0]; o[(q * 2 + 1) * CH] = acc[1];
      o[(q * 2) * CH + 8] = acc[2]; o[(q * 2 + 1) * CH + 8] = acc[3];
    }
  }
  // step-size product of staged row r and this thread's channel (all four lanes of the channel get it)
  __device__ __forceinline__ float product(int r, int ci, int l) const {
    if constexpr (kMma) return pre[r * CH + ci] + pre[(kMbRows + r) * CH + ci];
    float dot = 0.f;
    for (int k = l * 8; k < rank_p; k += 32) {
      float w8[8], d8[8];
      load8(w + (size_t)ci * wp + k, w8);
      load8(in + r * wp + k, d8);
#pragma unroll
      for (int j = 0; j < 8; ++j) dot += w8[j] * d8[j];
    }
    dot += __shfl_xor_sync(0xffffffffu, dot, 1);
    return dot + __shfl_xor_sync(0xffffffffu, dot, 2);
  }
  // one token of one channel: new state, and the gated result in place of x
  __device__ __forceinline__ void token(int r, int ci, int l, float bias, float D, const float4 (&A)[QPL], float4 (&S)[QPL]) {
    const float dt = softplus_t<T>(product(r, ci, l) + bias), xv = x[r * CH + ci], dx = dt * xv;
    float y = 0.f;
#pragma unroll
    for (int q = 0; q < QPL; ++q) {
      const float4 B = *reinterpret_cast<const float4*>(b + r * SP + (l + 4 * q) * 4), C = *reinterpret_cast<const float4*>(c + r * SP + (l + 4 * q) * 4);
      S[q].x = S[q].x * exp2_t<T>(dt * A[q].x) + dx * B.x; y += S[q].x * C.x;
      S[q].y = S[q].y * exp2_t<T>(dt * A[q].y) + dx * B.y; y += S[q].y * C.y;
      S[q].z = S[q].z * exp2_t<T>(dt * A[q].z) + dx * B.z; y += S[q].z * C.z;
      S[q].w = S[q].w * exp2_t<T>(dt * A[q].w) + dx * B.w; y += S[q].w * C.w;
    }
    y += __shfl_xor_sync(0xffffffffu, y, 1);
    y += __shfl_xor_sync(0xffffffffu, y, 2);
    if (l == 0) x[r * CH + ci] = (y + D * xv) * silu_t<T>(z[r * CH + ci]);   // read by these four lanes only, all of them done
  }
  __device__ __forceinline__ void write(const RfMamba1& p, int c0, int r0, int nr) const {
    for (int i = threadIdx.x; i < nr * (CH / 8); i += 256) {
      const int r = i / (CH / 8), k = (i % (CH / 8)) * 8;
      if (c0 + k >= p.inner) continue;
      float f[8];
      load8(x + r * CH + k, f);
      store8(reinterpret_cast<T*>(p.out) + (size_t)(r0 + r) * p.ldo + c0 + k, f);
    }
  }
};

// Any portions: a CTA owns 64 channels of `seqs_per_cta` neighbouring sequences, whose rows are contiguous.
template <typename T, int QPL>
__global__ void __launch_bounds__(256) mamba_recurrent_kernel(const RfMamba1 p, int seqs_per_cta) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t mb_raw[];
  MbTile<T, QPL> tile(mb_raw, p.rank);
  const int l = threadIdx.x & 3, ci = threadIdx.x >> 2, c0 = blockIdx.x * kMbChannels, c = c0 + ci, nq = p.states / 4;
  const bool live = c < p.inner;
  tile.prepare(p, c0);
  float4 A[QPL];
#pragma unroll
  for (int q = 0; q < QPL; ++q)
    A[q] = live && l + 4 * q < nq ? reinterpret_cast<const float4*>(p.a2 + (size_t)c * p.states)[l + 4 * q] : make_float4(0.f, 0.f, 0.f, 0.f);
  const float bias = live ? p.dt_bias[c] : 0.f, D = live ? p.d[c] : 0.f;
  pdl_wait();
  const int s0 = blockIdx.y * seqs_per_cta, s1 = min(p.rows.num_seqs, s0 + seqs_per_cta);
  const int row_begin = p.rows.q_start ? p.rows.q_start[s0] : s0;
  const int row_end = p.rows.q_start ? p.rows.q_start[s1 - 1] + p.rows.q_len[s1 - 1] : s1;
  auto state_of = [&](int seq) { return p.state + ((size_t)(p.rows.slot ? p.rows.slot[seq] : seq) * p.inner + c) * p.states; };
  auto load_state = [&](int seq, float4 (&S)[QPL]) {
    const bool fresh = p.rows.pos[p.rows.q_start ? p.rows.q_start[seq] : seq] == 0;
    const float4* st = reinterpret_cast<const float4*>(state_of(seq));
#pragma unroll
    for (int q = 0; q < QPL; ++q) S[q] = live && !fresh && l + 4 * q < nq ? st[l + 4 * q] : make_float4(0.f, 0.f, 0.f, 0.f);
  };
  float4 S[QPL], next[QPL];
  int seq = s0, left = p.rows.q_len ? p.rows.q_len[s0] : 1;
  load_state(s0, next);
  bool start = true;
  for (int r0 = row_begin; r0 < row_end; r0 += kMbRows) {
    const int nr = min(kMbRows, row_end - r0);
    __syncthreads();
    tile.stage(p, c0, r0, nr);
    __syncthreads();
    if (MbTile<T, QPL>::kMma) {
      tile.project(p, c0);
      __syncthreads();
    }
    for (int r = 0; r < nr; ++r) {
      if (start) {
#pragma unroll
        for (int q = 0; q < QPL; ++q) S[q] = next[q];
        if (seq + 1 < s1) load_state(seq + 1, next);
        start = false;
      }
      tile.token(r, ci, l, bias, D, A, S);
      if (--left == 0) {
        float4* st = reinterpret_cast<float4*>(state_of(seq));
        if (live) {
#pragma unroll
          for (int q = 0; q < QPL; ++q)
            if (l + 4 * q < nq) st[l + 4 * q] = S[q];
        }
        if (++seq < s1) left = p.rows.q_len ? p.rows.q_len[seq] : 1;
        start = true;
      }
    }
    __syncthreads();
    tile.write(p, c0, r0, nr);
  }
}

// Decode steps, one row per sequence, up to eight of them per CTA: the states of DEPTH sequences are in flight at any time.
template <typename T, int QPL, int DEPTH>
__global__ void __launch_bounds__(256) mamba_decode_kernel(const RfMamba1 p, int seqs_per_cta) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t mb_raw[];
  MbTile<T, QPL> tile(mb_raw, p.rank);
  const int l = threadIdx.x & 3, ci = threadIdx.x >> 2, c0 = blockIdx.x * kMbChannels, c = c0 + ci, nq = p.states / 4;
  const bool live = c < p.inner;
  tile.prepare(p, c0);
  float4 A[QPL], S[DEPTH][QPL];
#pragma unroll
  for (int q = 0; q < QPL; ++q)
    A[q] = live && l + 4 * q < nq ? reinterpret_cast<const float4*>(p.a2 + (size_t)c * p.states)[l + 4 * q] : make_float4(0.f, 0.f, 0.f, 0.f);
  const float bias = live ? p.dt_bias[c] : 0.f, D = live ? p.d[c] : 0.f;
  pdl_wait();
  const int s0 = blockIdx.y * seqs_per_cta, n = min(seqs_per_cta, p.rows.num_seqs - s0);
  auto state_of = [&](int i) { return reinterpret_cast<float4*>(p.state + ((size_t)(p.rows.slot ? p.rows.slot[s0 + i] : s0 + i) * p.inner + c) * p.states); };
  auto fetch = [&](int i, float4 (&s)[QPL]) {
    const bool use = live && i < n && p.rows.pos[min(s0 + i, p.rows.num_seqs - 1)] != 0;
#pragma unroll
    for (int q = 0; q < QPL; ++q) s[q] = use && l + 4 * q < nq ? state_of(i)[l + 4 * q] : make_float4(0.f, 0.f, 0.f, 0.f);
  };
#pragma unroll
  for (int i = 0; i < DEPTH; ++i) fetch(i, S[i]);
  __syncthreads();
  tile.stage(p, c0, s0, n);
  __syncthreads();
  if (MbTile<T, QPL>::kMma) {
    tile.project(p, c0);
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < kMbRows; ++i) {
    if (i >= n) break;
    float4 (&s)[QPL] = S[i % DEPTH];
    tile.token(i, ci, l, bias, D, A, s);
    if (live) {
#pragma unroll
      for (int q = 0; q < QPL; ++q)
        if (l + 4 * q < nq) state_of(i)[l + 4 * q] = s[q];
    }
    if (i + DEPTH < n) fetch(i + DEPTH, s);
  }
  __syncthreads();
  tile.write(p, c0, s0, n);
}

// ------------------------------------------------------------------------------------------------- scan ----
constexpr int kScanRows = 32;

// A CTA owns CH channels of one sequence and walks it in tiles of 32 rows: a thread fetches CPL pieces of eight channels of one
// row (the next tile's while the current one is scanned) and turns the step sizes and gates once per (row, channel).  Four lanes
// run the recurrence of CPL channels, which share what is read of B and C - shared-memory bandwidth is what bounds this kernel -
// and go four rows at a time, so that the sums over lanes cost three shuffles per four rows.
template <typename T, int CH, int QPL, int CPL>
__global__ void __launch_bounds__(CH * 4 / CPL) mamba_scan_kernel(const RfMamba1 p) {
  pdl_prologue();
  extern __shared__ __align__(16) float sc_sm[];
  constexpr int SP = 16 * QPL, NT = CH * 4 / CPL, TR = kScanRows, LD = CH + 8;   // LD: four rows of eight channels in different banks
  float2* s_q = reinterpret_cast<float2*>(sc_sm);       // [TR][CH] step size, step size times input
  float* s_d = reinterpret_cast<float*>(s_q + TR * CH); // [TR][LD] D times input; then the result
  float* s_g = s_d + TR * LD;                           // silu(z)
  float* s_b = s_g + TR * LD;                           // [TR][SP]
  float* s_c = s_b + TR * SP;
  const int tid = threadIdx.x, l = tid & 3, ci = tid >> 2, c0 = blockIdx.x * CH, seq = blockIdx.y;
  const int q0 = p.rows.q_start ? p.rows.q_start[seq] : seq, n = p.rows.q_len ? p.rows.q_len[seq] : 1;
  const int nq = p.states / 4;
  const bool fresh = p.rows.pos[q0] == 0;
  for (int i = tid; i < TR * SP * 2; i += NT) s_b[i] = 0.f;
  float4 A[CPL][QPL], S[CPL][QPL];
  float* st[CPL];
#pragma unroll
  for (int h = 0; h < CPL; ++h) {
    const int c = c0 + ci + h * (CH / CPL);
    const bool live = c < p.inner;
    st[h] = p.state + ((size_t)(p.rows.slot ? p.rows.slot[seq] : seq) * p.inner + (live ? c : 0)) * p.states;
#pragma unroll
    for (int q = 0; q < QPL; ++q) {
      const bool in = live && l + 4 * q < nq;
      A[h][q] = in ? reinterpret_cast<const float4*>(p.a2 + (size_t)c * p.states)[l + 4 * q] : make_float4(0.f, 0.f, 0.f, 0.f);
      S[h][q] = in && !fresh ? reinterpret_cast<const float4*>(st[h])[l + 4 * q] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  // the thread's pieces of a tile: rows lr + u * TR / CPL
  const int lr = tid / (CH / 8), lc = (tid % (CH / 8)) * 8;
  const bool in_c = c0 + lc < p.inner;
  float bias[8], D[8];
  zero8(bias); zero8(D);
  if (in_c) { load8(p.dt_bias + c0 + lc, bias); load8(p.d + c0 + lc, D); }
  const T* xp = reinterpret_cast<const T*>(p.x) + (size_t)q0 * p.ldx + c0 + lc;
  const T* zp = reinterpret_cast<const T*>(p.z) + (size_t)q0 * p.ldz + c0 + lc;
  const T* dp = reinterpret_cast<const T*>(p.dt) + (size_t)q0 * p.ld_dt + c0 + lc;
  const T* bp = reinterpret_cast<const T*>(p.bc) + (size_t)q0 * p.ld_bc + p.rank;
  Vec8<T> vx[CPL], vz[CPL], vd[CPL];
  auto fetch = [&](int t0) {
#pragma unroll
    for (int u = 0; u < CPL; ++u) {
      const int t = t0 + lr + u * (TR / CPL);
      if (t < n && in_c) {
        vx[u] = *reinterpret_cast<const Vec8<T>*>(xp + (size_t)t * p.ldx);
        vz[u] = *reinterpret_cast<const Vec8<T>*>(zp + (size_t)t * p.ldz);
        vd[u] = *reinterpret_cast<const Vec8<T>*>(dp + (size_t)t * p.ld_dt);
      }
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < n; t0 += TR) {
    const int nr = min(TR, n - t0);
    __syncthreads();                       // the previous tile's results have left
#pragma unroll
    for (int u = 0; u < CPL; ++u) {
      const int r = lr + u * (TR / CPL);
      float dd[8], g[8];
      zero8(dd); zero8(g);
      const bool in = r < nr && in_c;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        float4 dq = make_float4(0.f, 0.f, 0.f, 0.f);   // rows behind the end: step size 0 leaves the state as it is
        if (in) {
          const float2 x2 = Num<T>::to_f2(vx[u].v[j]), z2 = Num<T>::to_f2(vz[u].v[j]), d2 = Num<T>::to_f2(vd[u].v[j]);
          dq.x = softplus_t<T>(d2.x + bias[2 * j]); dq.y = dq.x * x2.x;
          dq.z = softplus_t<T>(d2.y + bias[2 * j + 1]); dq.w = dq.z * x2.y;
          dd[2 * j] = D[2 * j] * x2.x; dd[2 * j + 1] = D[2 * j + 1] * x2.y;
          g[2 * j] = silu_t<T>(z2.x); g[2 * j + 1] = silu_t<T>(z2.y);
        }
        *reinterpret_cast<float4*>(s_q + r * CH + lc + 2 * j) = dq;
      }
      store8(s_d + r * LD + lc, dd);
      store8(s_g + r * LD + lc, g);
    }
    for (int i = tid; i < TR * (p.states / 4); i += NT) {
      const int r = i / (p.states / 4), k = (i % (p.states / 4)) * 8;
      const bool is_c = k >= p.states;
      float f[8];
      zero8(f);
      if (r < nr) load8(bp + (size_t)(t0 + r) * p.ld_bc + k, f);
      store8((is_c ? s_c : s_b) + r * SP + (is_c ? k - p.states : k), f);
    }
    __syncthreads();
    if (t0 + TR < n) fetch(t0 + TR);
    for (int t = 0; t < nr; t += 4) {
      float v[CPL][4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        float2 dq[CPL];
#pragma unroll
        for (int h = 0; h < CPL; ++h) {
          dq[h] = s_q[(t + u) * CH + ci + h * (CH / CPL)];
          v[h][u] = 0.f;
        }
#pragma unroll
        for (int q = 0; q < QPL; ++q) {
          const float4 B = *reinterpret_cast<const float4*>(s_b + (t + u) * SP + (l + 4 * q) * 4), C = *reinterpret_cast<const float4*>(s_c + (t + u) * SP + (l + 4 * q) * 4);
#pragma unroll
          for (int h = 0; h < CPL; ++h) {
            float4& s = S[h][q];
            const float dt = dq[h].x, dx = dq[h].y;
            s.x = s.x * exp2_t<T>(dt * A[h][q].x) + dx * B.x; v[h][u] += s.x * C.x;
            s.y = s.y * exp2_t<T>(dt * A[h][q].y) + dx * B.y; v[h][u] += s.y * C.y;
            s.z = s.z * exp2_t<T>(dt * A[h][q].z) + dx * B.z; v[h][u] += s.z * C.z;
            s.w = s.w * exp2_t<T>(dt * A[h][q].w) + dx * B.w; v[h][u] += s.w * C.w;
          }
        }
      }
      // lane l ends with the sum of row t + l: swap halves with the lane two away, then with the neighbour
      const bool hi = l & 2, odd = l & 1;
#pragma unroll
      for (int h = 0; h < CPL; ++h) {
        const float a0 = __shfl_xor_sync(0xffffffffu, hi ? v[h][0] : v[h][2], 2), a1 = __shfl_xor_sync(0xffffffffu, hi ? v[h][1] : v[h][3], 2);
        const float w0 = (hi ? v[h][2] : v[h][0]) + a0, w1 = (hi ? v[h][3] : v[h][1]) + a1;
        const float y = (odd ? w1 : w0) + __shfl_xor_sync(0xffffffffu, odd ? w0 : w1, 1);
        const int at = (t + l) * LD + ci + h * (CH / CPL);
        s_d[at] = (y + s_d[at]) * s_g[at];
      }
    }
    __syncthreads();
#pragma unroll
    for (int u = 0; u < CPL; ++u) {
      const int r = lr + u * (TR / CPL);
      if (r >= nr || !in_c) continue;
      float f[8];
      load8(s_d + r * LD + lc, f);
      store8(reinterpret_cast<T*>(p.out) + (size_t)(q0 + t0 + r) * p.ldo + c0 + lc, f);
    }
  }
#pragma unroll
  for (int h = 0; h < CPL; ++h) {
    if (c0 + ci + h * (CH / CPL) >= p.inner) continue;
#pragma unroll
    for (int q = 0; q < QPL; ++q)
      if (l + 4 * q < nq) reinterpret_cast<float4*>(st[h])[l + 4 * q] = S[h][q];
  }
}

// ------------------------------------------------------------------------------------------------- host ----
static int check_mamba(const RfMamba1* a) {
  RF_REQUIRE(a && a->x && a->z && a->bc && a->dt_bias && a->a2 && a->d && a->state && a->out && a->rows.pos, "mamba: missing buffers");
  RF_REQUIRE(a->inner > 0 && a->inner % 8 == 0 && a->states > 0 && a->states % 8 == 0 && a->states <= 256 && a->rank > 0 && a->rank % 8 == 0,
             "mamba: %d channels, %d states, step rank %d", a->inner, a->states, a->rank);
  RF_REQUIRE(a->ldx % 8 == 0 && a->ldz % 8 == 0 && a->ld_bc % 8 == 0 && a->ldo % 8 == 0, "mamba: pitches must be multiples of 8");
  RF_REQUIRE(a->dtype >= 0 && a->dtype <= 2, "mamba: dtype %d", a->dtype);
  return RF_OK;
}

template <typename T, int QPL>
static int launch_recurrent(const RfMamba1* a, cudaStream_t s) {
  const int tiles = ceil_div(a->inner, kMbChannels), seqs = a->rows.num_seqs;
  const size_t smem = MbTile<T, QPL>::bytes(a->rank);
  RF_REQUIRE(smem <= 200 * 1024, "mamba: a step rank of %d does not fit in shared memory", a->rank);
  // share what a CTA reads for its channels between sequences once there are enough CTAs without that
  const int spc = std::max(1, std::min(kMbRows, seqs * tiles / (4 * sm_count())));
  if (QPL <= 4 && !a->rows.q_start) {
    constexpr int Q = QPL <= 4 ? QPL : 1, DEPTH = QPL == 1 ? 4 : 2;
    RF_ALLOW_SMEM_PER_DEVICE((mamba_decode_kernel<T, Q, DEPTH>), 200 * 1024);
    RF_CUDA_CHECK(::rf::launch_k(mamba_decode_kernel<T, Q, DEPTH>, dim3(tiles, ceil_div(seqs, spc)), dim3(256), smem, s, 1, *a, spc));
    ::rf::count_launch();
    return RF_OK;
  }
  RF_ALLOW_SMEM_PER_DEVICE((mamba_recurrent_kernel<T, QPL>), 200 * 1024);
  RF_CUDA_CHECK(::rf::launch_k(mamba_recurrent_kernel<T, QPL>, dim3(tiles, ceil_div(seqs, spc)), dim3(256), smem, s, 1, *a, spc));
  ::rf::count_launch();
  return RF_OK;
}

template <typename T, int CH, int QPL, int CPL>
static int launch_scan_t(const RfMamba1* a, cudaStream_t s) {
  const size_t smem = (size_t)kScanRows * (2 * CH + 2 * (CH + 8) + 32 * QPL) * sizeof(float);
  RF_ALLOW_SMEM_PER_DEVICE((mamba_scan_kernel<T, CH, QPL, CPL>), 128 * 1024);
  RF_CUDA_CHECK(::rf::launch_k(mamba_scan_kernel<T, CH, QPL, CPL>, dim3(ceil_div(a->inner, CH), a->rows.num_seqs), dim3(CH * 4 / CPL), smem, s, 1, *a));
  ::rf::count_launch();
  return RF_OK;
}

template <typename T, int QPL>
static int launch_scan(const RfMamba1* a, cudaStream_t s) {
  constexpr int CPL = QPL <= 2 ? 2 : 1;              // wider states leave no registers for a second channel
  const int seqs = a->rows.num_seqs;
  if (ceil_div(a->inner, 64) * seqs >= 4 * sm_count()) return launch_scan_t<T, 64, QPL, CPL>(a, s);
  // few sequences: latency counts, so more warps with one channel per four lanes
  if (ceil_div(a->inner, 32) * seqs >= 3 * sm_count()) return launch_scan_t<T, 32, QPL, CPL>(a, s);
  return launch_scan_t<T, 32, QPL, 1>(a, s);
}

}  // namespace rf

using namespace rf;

#define RF_MAMBA_STATES(T, FN)                  \
  {                                             \
    const int q = (a->states + 15) / 16;        \
    if (q <= 1) return FN<T, 1>(a, s);          \
    if (q <= 2) return FN<T, 2>(a, s);          \
    if (q <= 4) return FN<T, 4>(a, s);          \
    if (q <= 8) return FN<T, 8>(a, s);          \
    return FN<T, 16>(a, s);                     \
  }
#define RF_MAMBA_DISPATCH(FN)                                   \
  cudaStream_t s = static_cast<cudaStream_t>(stream);           \
  if (a->dtype == kF16) RF_MAMBA_STATES(__half, FN)             \
  if (a->dtype == kBF16) RF_MAMBA_STATES(__nv_bfloat16, FN)     \
  RF_MAMBA_STATES(float, FN)

extern "C" int rf_mamba1_recurrent(const RfMamba1* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  int rc = check_mamba(a);
  if (rc) return rc;
  RF_REQUIRE(a->w_dt, "mamba recurrence: step-size weights");
  if (a->rows.num_seqs == 0) return RF_OK;
  RF_MAMBA_DISPATCH(launch_recurrent)
}

extern "C" int rf_mamba1_scan(const RfMamba1* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  int rc = check_mamba(a);
  if (rc) return rc;
  RF_REQUIRE(a->dt && a->ld_dt % 8 == 0, "mamba scan: step-size rows");
  RF_REQUIRE(a->rows.num_seqs <= 65535, "mamba scan: %d sequences", a->rows.num_seqs);
  if (a->rows.num_seqs == 0) return RF_OK;
  RF_MAMBA_DISPATCH(launch_scan)
}

extern "C" int rf_conv_silu(const RfConvSilu* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_REQUIRE(a && a->x && a->y && a->w && a->rows.pos && (a->taps == 1 || a->state), "conv_silu: missing buffers");
  RF_REQUIRE(a->channels > 0 && a->channels % 8 == 0 && a->ldx % 8 == 0 && a->ldy % 8 == 0 && a->taps >= 1, "conv_silu: %d channels, %d taps",
             a->channels, a->taps);
  RF_REQUIRE(a->dtype >= 0 && a->dtype <= 2 && a->x != a->y && a->max_q_len >= 1 && a->rows.num_seqs <= 65535, "conv_silu: options");
  if (a->rows.num_seqs == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int tile = std::max(16, a->taps - 1);      // later tiles find their past in the rows of this launch
  const dim3 grid(ceil_div(a->channels, 1024), ceil_div(a->max_q_len, tile), a->rows.num_seqs);
#define RF_CONV(T)                                                                                                       \
  switch (a->taps) {                                                                                                     \
    case 2: RF_CUDA_CHECK(::rf::launch_k(conv_silu_kernel<T, 2>, grid, dim3(128), 0, s, 1, *a, tile)); break;            \
    case 3: RF_CUDA_CHECK(::rf::launch_k(conv_silu_kernel<T, 3>, grid, dim3(128), 0, s, 1, *a, tile)); break;            \
    case 4: RF_CUDA_CHECK(::rf::launch_k(conv_silu_kernel<T, 4>, grid, dim3(128), 0, s, 1, *a, tile)); break;            \
    default: RF_CUDA_CHECK(::rf::launch_k(conv_silu_kernel<T, 0>, grid, dim3(128), 0, s, 1, *a, tile)); break;           \
  }
  if (a->dtype == kF16) { RF_CONV(__half) } else if (a->dtype == kBF16) { RF_CONV(__nv_bfloat16) } else { RF_CONV(float) }
#undef RF_CONV
  ::rf::count_launch();
  return RF_OK;
}
