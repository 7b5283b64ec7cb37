// The fp32 residual stream between sublayers (pending sublayer output added, optionally normalised; RMSNorm; token shift),
// the per-token gate of a side input, and the fp32 GEMM of models served in 32 bits.
#include "../common/dtype.cuh"
#include "../common/host_util.h"
#include "../common/ptx.cuh"
#include "../rf_api.h"

namespace rf {

__device__ __forceinline__ float stream_block_sum(float v, float* red) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = (blockDim.x + 31) >> 5;
  __syncthreads();
  if (l == 0) red[w] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < nw; ++i) t += red[i];       // every thread adds the same values in the same order
  return t;
}

template <typename T> struct alignas(sizeof(T) * 4) Quad { T v[4]; };
template <typename T>
__device__ __forceinline__ float4 load4(const T* p) {
  const Quad<T> q = *reinterpret_cast<const Quad<T>*>(p);
  return make_float4(Num<T>::to_f(q.v[0]), Num<T>::to_f(q.v[1]), Num<T>::to_f(q.v[2]), Num<T>::to_f(q.v[3]));
}
template <typename T>
__device__ __forceinline__ void store4(T* p, float4 f) {
  Quad<T> q;
  q.v[0] = Num<T>::from_f(f.x); q.v[1] = Num<T>::from_f(f.y); q.v[2] = Num<T>::from_f(f.z); q.v[3] = Num<T>::from_f(f.w);
  *reinterpret_cast<Quad<T>*>(p) = q;
}
// four columns of the outstanding output of row `src`: one row, or the sum of the picked ones
template <typename T>
__device__ __forceinline__ float4 pending4(const RfStreamNorm& p, const T* y, int src, int col) {
  if (p.y_picks <= 0) return load4(y + (size_t)src * p.H + col);
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (p.y_self_w) {
    const float w = p.y_self_w[src];
    const float4 v = load4(reinterpret_cast<const T*>(p.y_self) + (size_t)src * p.H + col);
    s = make_float4(w * v.x, w * v.y, w * v.z, w * v.w);
  }
  const int32_t* slots = p.y_slots + (size_t)src * p.y_picks;
#pragma unroll 4
  for (int j = 0; j < p.y_picks; ++j) {
    const int r = slots[j];
    if (r < 0) continue;
    const float4 v = load4(y + (size_t)r * p.H + col);
    s.x += v.x; s.y += v.y; s.z += v.z; s.w += v.w;
  }
  return s;
}
__device__ __forceinline__ float4 mul4(float4 v, float f) { return make_float4(v.x * f, v.y * f, v.z * f, v.w * f); }
__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
// Row of table2 for the token pair (previous token, token) that ends in row r.
__device__ __forceinline__ int64_t pair_row(const RfStreamNorm& p, int r) {
  const int seq = p.rows.seq_of_row ? p.rows.seq_of_row[r] : r, q0 = p.rows.q_start ? p.rows.q_start[seq] : r;
  int64_t prev;
  if (r > q0) prev = p.ids[r - 1];
  else if (p.rows.pos[r] == 0) return p.buckets;
  else prev = p.last_token[p.rows.slot ? p.rows.slot[seq] : seq];
  return (prev * p.mul_prev + p.ids[r] * p.mul_cur) % p.buckets;
}
// The CTA of a sequence's first row, the only reader of the carried token, replaces it (all threads of the CTA, after pair_row).
__device__ __forceinline__ void carry_token(const RfStreamNorm& p, int r) {
  const int seq = p.rows.seq_of_row ? p.rows.seq_of_row[r] : r, q0 = p.rows.q_start ? p.rows.q_start[seq] : r;
  if (r != q0) return;
  __syncthreads();
  if (threadIdx.x == 0) p.last_token[p.rows.slot ? p.rows.slot[seq] : seq] = p.ids[q0 + (p.rows.q_len ? p.rows.q_len[seq] : 1) - 1];
}
__device__ __forceinline__ float sq4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

// A CTA walks rows_per_cta neighbouring rows.  A thread always touches the same columns, so the shared copies of the
// current row (xs) and of the previous token's normalised row (hp) need no barriers of their own.
template <typename T>
__global__ void stream_norm_kernel(const RfStreamNorm p, int rows_per_cta) {
  pdl_prologue();
  extern __shared__ __align__(16) float sm[];
  float* xs = sm;
  float* hp = sm + p.H;
  float* red = hp + (p.shift ? p.H : 0);
  const int H = p.H, step = blockDim.x * 4, c0 = threadIdx.x * 4;
  const float inv_dim = 1.f / (float)p.dim;
  const T* table = reinterpret_cast<const T*>(p.table);
  const T* y = reinterpret_cast<const T*>(p.y);

  // loads row r into xs with the pending output added, returns 1 / rms of it (when the row is normalised)
  auto load_row = [&](int r, bool write) -> float {
    const int src = p.row_idx ? p.row_idx[r] : r;
    float yr = 1.f;
    if (y && p.y_norm_w) {
      float s = 0.f;
      for (int i = c0; i < H; i += step) s += sq4(pending4(p, y, src, i));
      yr = rsqrtf(stream_block_sum(s, red) * inv_dim + p.eps);
    }
    const float* xr = p.x ? p.x + (size_t)src * H : nullptr;
    const T* er = p.x ? nullptr : table + (size_t)p.ids[src] * H;
    const T* er2 = p.table2 ? reinterpret_cast<const T*>(p.table2) + (size_t)pair_row(p, src) * H : nullptr;
    if (er2) carry_token(p, src);
    float s = 0.f;
    for (int i = c0; i < H; i += step) {
      float4 v = xr ? *reinterpret_cast<const float4*>(xr + i) : mul4(load4(er + i), p.embed_scale);
      if (er2) v = add4(v, load4(er2 + i));
      if (y) {
        float4 a = pending4(p, y, src, i);
        if (p.y_norm_w) {
          const float4 w = *reinterpret_cast<const float4*>(p.y_norm_w + i);
          a.x *= yr * w.x; a.y *= yr * w.y; a.z *= yr * w.z; a.w *= yr * w.w;
        }
        v = add4(v, mul4(a, p.y_mult));
      }
      *reinterpret_cast<float4*>(xs + i) = v;
      s += sq4(v);
      if (write) {
        if (p.x_out) *reinterpret_cast<float4*>(p.x_out + (size_t)r * H + i) = v;
        if (p.x_cast) store4(reinterpret_cast<T*>(p.x_cast) + (size_t)r * H + i, v);
      }
    }
    return p.norm_w ? rsqrtf(stream_block_sum(s, red) * inv_dim + p.eps) : 1.f;
  };
  auto normed = [&](int i, float rstd) -> float4 {
    const float4 v = *reinterpret_cast<const float4*>(xs + i), w = *reinterpret_cast<const float4*>(p.norm_w + i);
    return make_float4(v.x * rstd * w.x, v.y * rstd * w.y, v.z * rstd * w.z, v.w * rstd * w.w);
  };

  const int r0 = blockIdx.x * rows_per_cta, r1 = min(p.n_rows, r0 + rows_per_cta);
  for (int r = r0; r < r1; ++r) {
    float* state = nullptr;
    bool state_here = false;
    if (p.shift) {
      const int seq = p.rows.seq_of_row ? p.rows.seq_of_row[r] : r;
      const int q0 = p.rows.q_start ? p.rows.q_start[seq] : r;
      if (r == q0) {
        // first row of its sequence in this launch: the carried row is read here and replaced here, by the CTA that
        // read it (the sequence's last row is normalised a second time for that)
        const int n = p.rows.q_len ? p.rows.q_len[seq] : 1;
        state = p.shift_state + (size_t)(p.rows.slot ? p.rows.slot[seq] : seq) * H;
        const bool fresh = p.rows.pos[r] == 0;
        for (int i = c0; i < H; i += step)
          *reinterpret_cast<float4*>(hp + i) = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(state + i);
        if (n > 1) {
          const float rl = load_row(r + n - 1, false);
          for (int i = c0; i < H; i += step) *reinterpret_cast<float4*>(state + i) = normed(i, rl);
        } else {
          state_here = true;
        }
      } else if (r == r0) {
        const float rl = load_row(r - 1, false);
        for (int i = c0; i < H; i += step) *reinterpret_cast<float4*>(hp + i) = normed(i, rl);
      }
    }
    const float rstd = load_row(r, true);
    if (!p.norm_w) continue;
    T* out = reinterpret_cast<T*>(p.out) + (size_t)r * H;
    for (int i = c0; i < H; i += step) {
      float4 h = normed(i, rstd);
      if (p.shift) {
        const float4 b = *reinterpret_cast<const float4*>(hp + i), mu = *reinterpret_cast<const float4*>(p.shift + i);
        *reinterpret_cast<float4*>(hp + i) = h;
        if (state_here) *reinterpret_cast<float4*>(state + i) = h;
        h.x += (b.x - h.x) * mu.x; h.y += (b.y - h.y) * mu.y; h.z += (b.z - h.z) * mu.z; h.w += (b.w - h.w) * mu.w;
      }
      store4(out + i, h);
    }
  }
}

// The same for rows that fit the registers of a CTA (VPT quads per thread): every operand of a row is requested before the
// first reduction, so a decode step pays one memory round trip, and the next row's operands are requested while the current
// one is reduced.
template <typename T, int VPT>
__global__ void __launch_bounds__(VPT == 4 ? 512 : 1024) stream_norm_reg_kernel(const RfStreamNorm p, int rows_per_cta) {
  pdl_launch_dependents();
  __shared__ float red[2][32];
  const int H = p.H, nthr = blockDim.x, nw = nthr >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float inv_dim = 1.f / (float)p.dim;
  const T* table = reinterpret_cast<const T*>(p.table);
  const T* y = reinterpret_cast<const T*>(p.y);
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  auto col = [&](int k) { return (threadIdx.x + k * nthr) * 4; };
  // weights do not depend on the previous kernel
  float4 nwt[VPT], mu[VPT], yw[VPT];
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const bool in = col(k) < H;
    nwt[k] = p.norm_w && in ? *reinterpret_cast<const float4*>(p.norm_w + col(k)) : zero;
    mu[k] = p.shift && in ? *reinterpret_cast<const float4*>(p.shift + col(k)) : zero;
    yw[k] = p.y_norm_w && in ? *reinterpret_cast<const float4*>(p.y_norm_w + col(k)) : zero;
  }
  pdl_wait();
  int flip = 0;
  auto block_sum = [&](float v) -> float {       // one barrier: consecutive sums use different rows of `red`
    v = warp_sum(v);
    if (lane == 0) red[flip][warp] = v;
    __syncthreads();
    const float t = warp_sum(lane < nw ? red[flip][lane] : 0.f);
    flip ^= 1;
    return t;
  };
  float4 v[VPT], a[VPT];
  auto load = [&](int r) {
    const int src = p.row_idx ? p.row_idx[r] : r;
    const T* second = p.table2 ? reinterpret_cast<const T*>(p.table2) + (size_t)pair_row(p, src) * H : nullptr;
    if (second) carry_token(p, src);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const bool in = col(k) < H;
      v[k] = !in ? zero : p.x ? *reinterpret_cast<const float4*>(p.x + (size_t)src * H + col(k)) : mul4(load4(table + (size_t)p.ids[src] * H + col(k)), p.embed_scale);
      if (second && in) v[k] = add4(v[k], load4(second + col(k)));
      a[k] = y && in ? pending4(p, y, src, col(k)) : zero;
    }
  };
  // v <- v + pending output; returns 1 / rms when the row is normalised
  auto finish_row = [&]() -> float {
    float yr = 1.f;
    if (p.y_norm_w) {
      float s = 0.f;
#pragma unroll
      for (int k = 0; k < VPT; ++k) s += sq4(a[k]);
      yr = rsqrtf(block_sum(s) * inv_dim + p.eps);
    }
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      if (p.y_norm_w) {
        a[k].x *= yr * yw[k].x; a[k].y *= yr * yw[k].y; a[k].z *= yr * yw[k].z; a[k].w *= yr * yw[k].w;
      }
      v[k] = add4(v[k], mul4(a[k], p.y_mult));
      s += sq4(v[k]);
    }
    return p.norm_w ? rsqrtf(block_sum(s) * inv_dim + p.eps) : 1.f;
  };
  auto normed = [&](int k, float r) { return make_float4(v[k].x * r * nwt[k].x, v[k].y * r * nwt[k].y, v[k].z * r * nwt[k].z, v[k].w * r * nwt[k].w); };

  float4 hp[VPT];
  const int r0 = blockIdx.x * rows_per_cta, r1 = min(p.n_rows, r0 + rows_per_cta);
  for (int r = r0; r < r1; ++r) {
    float* state = nullptr;
    bool state_here = false, fresh = false;
    if (p.shift) {
      const int seq = p.rows.seq_of_row ? p.rows.seq_of_row[r] : r;
      const int q0 = p.rows.q_start ? p.rows.q_start[seq] : r;
      if (r == q0) {
        const int n = p.rows.q_len ? p.rows.q_len[seq] : 1;
        state = p.shift_state + (size_t)(p.rows.slot ? p.rows.slot[seq] : seq) * H;
        fresh = p.rows.pos[r] == 0;
#pragma unroll
        for (int k = 0; k < VPT; ++k) hp[k] = col(k) < H ? *reinterpret_cast<const float4*>(state + col(k)) : zero;
        if (n > 1) {                             // the carried row is replaced by the last row's, normalised here a second time
          load(r + n - 1);
          const float rl = finish_row();
#pragma unroll
          for (int k = 0; k < VPT; ++k)
            if (col(k) < H) *reinterpret_cast<float4*>(state + col(k)) = normed(k, rl);
        } else {
          state_here = true;
        }
      } else if (r == r0) {
        load(r - 1);
        const float rl = finish_row();
#pragma unroll
        for (int k = 0; k < VPT; ++k) hp[k] = normed(k, rl);
      }
    }
    load(r);
    const float rstd = finish_row();
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int c = col(k);
      if (c >= H) continue;
      if (p.x_out) *reinterpret_cast<float4*>(p.x_out + (size_t)r * H + c) = v[k];
      if (p.x_cast) store4(reinterpret_cast<T*>(p.x_cast) + (size_t)r * H + c, v[k]);
      if (!p.norm_w) continue;
      float4 h = normed(k, rstd);
      if (p.shift) {
        const float4 b = fresh ? zero : hp[k], m = mu[k];
        hp[k] = h;
        if (state_here) *reinterpret_cast<float4*>(state + c) = h;
        h.x += (b.x - h.x) * m.x; h.y += (b.y - h.y) * m.y; h.z += (b.z - h.z) * m.z; h.w += (b.w - h.w) * m.w;
      }
      store4(reinterpret_cast<T*>(p.out) + (size_t)r * H + c, h);
    }
  }
}

// Input convolution of eight columns of a decode row: h <- h + conv(h), carried rows read and moved up by one.
template <typename T>
__device__ __forceinline__ void input_conv8(const RfStreamNorm& p, int r, int col, float (&h)[8]) {
  const int past = p.conv_taps - 1;
  T* state = reinterpret_cast<T*>(p.conv_state) + (size_t)(p.rows.slot ? p.rows.slot[r] : r) * past * p.H + col;
  const bool fresh = p.rows.pos[r] == 0;
  float w[8], f[8], s[8];
  load8(p.conv_w + (size_t)past * p.H + col, w);
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    h[j] = Num<T>::to_f(Num<T>::from_f(h[j]));     // rows enter the convolution as they are carried
    s[j] = w[j] * h[j];
  }
#pragma unroll 4
  for (int k = 0; k < past; ++k) {
    load8(p.conv_w + (size_t)k * p.H + col, w);
    if (fresh) {
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = 0.f;
    } else {
      load8(state + (size_t)k * p.H, f);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) s[j] += w[j] * f[j];
    if (k > 0) store8(state + (size_t)(k - 1) * p.H, f);
  }
  if (past > 0) store8(state + (size_t)(past - 1) * p.H, h);
#pragma unroll
  for (int j = 0; j < 8; ++j) h[j] += s[j];
}

// The stream step of 16-bit activations without a token shift: one CTA per row, a thread holds NC groups of eight columns, so that
// every operand moves in 16-byte pieces; of several picked rows four are in flight at a time.
template <typename T, int NC, bool CONV>
__global__ void __launch_bounds__(512) stream_out_kernel(const RfStreamNorm p) {
  pdl_launch_dependents();
  __shared__ float red[2][16];
  const int H = p.H, nthr = blockDim.x, nw = nthr >> 5, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float inv_dim = 1.f / (float)p.dim;
  auto col = [&](int k) { return (threadIdx.x + k * nthr) * 8; };
  float w[NC][8];                                              // the first norm's weights: they do not depend on the previous kernel
  const float* first_w = p.y_norm_w ? p.y_norm_w : p.norm_w;
#pragma unroll
  for (int k = 0; k < NC; ++k)
    if (first_w && col(k) < H) load8(first_w + col(k), w[k]);
  pdl_wait();
  const int r = blockIdx.x, src = p.row_idx ? p.row_idx[r] : r;
  const T* y = reinterpret_cast<const T*>(p.y);
  const T* second = p.table2 ? reinterpret_cast<const T*>(p.table2) + (size_t)pair_row(p, src) * H : nullptr;
  if (second) carry_token(p, src);
  float v[NC][8], a[NC][8];
#pragma unroll
  for (int k = 0; k < NC; ++k) {
#pragma unroll
    for (int j = 0; j < 8; ++j) v[k][j] = a[k][j] = 0.f;
    if (col(k) >= H) continue;
    if (p.x) load8(p.x + (size_t)src * H + col(k), v[k]);
    else {
      load8(reinterpret_cast<const T*>(p.table) + (size_t)p.ids[src] * H + col(k), v[k]);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] *= p.embed_scale;
      if (second) {
        float f[8];
        load8(second + col(k), f);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[k][j] += f[j];
      }
    }
  }
  const int picks = !y ? 0 : p.y_picks > 0 ? p.y_picks : 1;
  for (int j0 = 0; j0 < picks; j0 += 4) {
    int row[4];
    uint4 raw[4][NC];
#pragma unroll
    for (int i = 0; i < 4; ++i) row[i] = j0 + i >= picks ? -1 : (p.y_picks > 0 ? p.y_slots[(size_t)src * picks + j0 + i] : src);
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int k = 0; k < NC; ++k) {
        raw[i][k] = make_uint4(0u, 0u, 0u, 0u);                // zero bits are zero in both formats
        if (row[i] >= 0 && col(k) < H) raw[i][k] = *reinterpret_cast<const uint4*>(y + (size_t)row[i] * H + col(k));
      }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int k = 0; k < NC; ++k) {
        const typename Num<T>::T2* t = reinterpret_cast<const typename Num<T>::T2*>(&raw[i][k]);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 f = Num<T>::to_f2(t[j]);
          a[k][2 * j] += f.x;
          a[k][2 * j + 1] += f.y;
        }
      }
  }
  if (p.y_self_w) {
    const float sw = p.y_self_w[src];
#pragma unroll
    for (int k = 0; k < NC; ++k) {
      if (col(k) >= H) continue;
      float f[8];
      load8(reinterpret_cast<const T*>(p.y_self) + (size_t)src * H + col(k), f);
#pragma unroll
      for (int j = 0; j < 8; ++j) a[k][j] += sw * f[j];
    }
  }
  auto block_sum = [&](float s, int flip) -> float {
    s = warp_sum(s);
    if (lane == 0) red[flip][warp] = s;
    __syncthreads();
    return warp_sum(lane < nw ? red[flip][lane] : 0.f);
  };
  float s = 0.f, yr = p.y_mult;
  if (p.y_norm_w) {
#pragma unroll
    for (int k = 0; k < NC; ++k)
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        s += a[k][j] * a[k][j];
        a[k][j] *= w[k][j];
      }
    yr *= rsqrtf(block_sum(s, 0) * inv_dim + p.eps);
  }
  s = 0.f;
#pragma unroll
  for (int k = 0; k < NC; ++k) {
    if (col(k) >= H) continue;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      v[k][j] += a[k][j] * yr;
      s += v[k][j] * v[k][j];
    }
    if (p.x_out) store8(p.x_out + (size_t)r * H + col(k), v[k]);
    if (p.x_cast) store8(reinterpret_cast<T*>(p.x_cast) + (size_t)r * H + col(k), v[k]);
  }
  if (!p.norm_w) return;
  const float xr = rsqrtf(block_sum(s, 1) * inv_dim + p.eps);
#pragma unroll
  for (int k = 0; k < NC; ++k) {
    if (col(k) >= H) continue;
    float n8[8];
    if (p.y_norm_w) load8(p.norm_w + col(k), w[k]);
#pragma unroll
    for (int j = 0; j < 8; ++j) n8[j] = w[k][j] * v[k][j] * xr;
    if constexpr (CONV) input_conv8<T>(p, r, col(k), n8);
    store8(reinterpret_cast<T*>(p.out) + (size_t)r * H + col(k), n8);
  }
}

template <typename T>
__global__ void token_gate_kernel(T* __restrict__ g, int64_t ldg, const T* __restrict__ table, int64_t ldt,
                                  const int32_t* __restrict__ ids, int col0, int rows, int cols) {
  pdl_prologue();
  const int per = cols / 8;
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (int64_t)rows * per) return;
  const int r = (int)(i / per), c = (int)(i % per) * 8;
  float a[8], b[8];
  load8(g + (size_t)r * ldg + c, a);
  load8(table + (size_t)ids[r] * ldt + col0 + c, b);
#pragma unroll
  for (int j = 0; j < 8; ++j) a[j] *= b[j];
  store8(g + (size_t)r * ldg + c, a);
}

// ------------------------------------------------------------------ fp32 GEMM ----
constexpr int kFBM = 64, kFBN = 64, kFBK = 16;

__device__ __forceinline__ float act_f32(int act, float v, float u, ActArgs a) {
  switch (act) {
    case kActSiluMul: return v / (1.f + expf(-v)) * u;
    case kActClippedGlu: v = fminf(v, a.limit); return v / (1.f + expf(-a.alpha * v)) * (fminf(fmaxf(u, -a.limit), a.limit) + 1.f);
    case kActSoftCap: return a.limit * tanhf(v / a.limit);
    case kActRelu2: return relu2_f(v);
    case kActSilu: return v / (1.f + expf(-v));
    case kActGeluTanh: return 0.5f * v * (1.f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
    case kActGeluErf: return 0.5f * v * (1.f + erff(v * 0.7071067811865476f));
    default: return v;
  }
}

// DUAL: a second block of weight rows, dual_offset rows below the first, feeds the activation's second operand.
template <bool DUAL>
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ x, int64_t ldx, const float* __restrict__ w,
                                                       int64_t ldw, float* __restrict__ out, int64_t ldo, int M, int N,
                                                       int K, int act, int dual_offset, const float* __restrict__ row_scale, ActArgs args) {
  pdl_prologue();
  constexpr int D = DUAL ? 2 : 1;
  __shared__ __align__(16) float sx[kFBK][kFBM + 4], sw[D][kFBK][kFBN + 4];
  const int n0 = blockIdx.x * kFBN, m0 = blockIdx.y * kFBM, tid = threadIdx.x;
  const int tx = tid % 16, ty = tid / 16, lr = tid / 4, lk = (tid % 4) * 4;
  float acc[D][4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kFBK) {
    const bool kin = k0 + lk < K;            // K is a multiple of 4
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    if (kin && m0 + lr < M) a = *reinterpret_cast<const float4*>(x + (size_t)(m0 + lr) * ldx + k0 + lk);
    sx[lk][lr] = a.x; sx[lk + 1][lr] = a.y; sx[lk + 2][lr] = a.z; sx[lk + 3][lr] = a.w;
#pragma unroll
    for (int d = 0; d < D; ++d) {
      float4 b = make_float4(0.f, 0.f, 0.f, 0.f);
      if (kin && n0 + lr < N) b = *reinterpret_cast<const float4*>(w + (size_t)(n0 + lr + d * dual_offset) * ldw + k0 + lk);
      sw[d][lk][lr] = b.x; sw[d][lk + 1][lr] = b.y; sw[d][lk + 2][lr] = b.z; sw[d][lk + 3][lr] = b.w;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kFBK; ++k) {
      const float4 av = *reinterpret_cast<const float4*>(&sx[k][ty * 4]);
      const float am[4] = {av.x, av.y, av.z, av.w};
#pragma unroll
      for (int d = 0; d < D; ++d) {
        const float4 bv = *reinterpret_cast<const float4*>(&sw[d][k][tx * 4]);
        const float bn[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[d][i][j] = fmaf(am[i], bn[j], acc[d][i][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m >= M || n >= N) continue;
      const float rs = row_scale ? row_scale[m] : 1.f;
      out[(size_t)m * ldo + n] = act_f32(act, acc[0][i][j] * rs, acc[D - 1][i][j] * rs, args);
    }
}

}  // namespace rf

using namespace rf;

#define RF_DISPATCH3(dtype, ...)                                        \
  if ((dtype) == kF16) { using T = __half; __VA_ARGS__; }               \
  else if ((dtype) == kBF16) { using T = __nv_bfloat16; __VA_ARGS__; }  \
  else { using T = float; __VA_ARGS__; }

extern "C" int rf_stream_norm(const RfStreamNorm* args, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_REQUIRE(args != nullptr, "stream_norm: null arguments");
  RfStreamNorm filled = *args;
  if (filled.embed_scale == 0.f) filled.embed_scale = 1.f;
  if (filled.y_mult == 0.f) filled.y_mult = 1.f;
  const RfStreamNorm* a = &filled;
  RF_REQUIRE(a->y_picks <= 0 || (a->y && a->y_slots), "stream_norm: picked rows need y and y_slots");
  RF_REQUIRE(a && a->H > 0 && a->H % 8 == 0 && a->dim > 0 && a->dim <= a->H, "stream_norm: row length");
  RF_REQUIRE(a->x || (a->table && a->ids), "stream_norm: no input");
  RF_REQUIRE(!a->norm_w || a->out, "stream_norm: no output");
  RF_REQUIRE(a->dtype >= 0 && a->dtype <= 2, "stream_norm: dtype %d", a->dtype);
  if (a->shift) RF_REQUIRE(a->norm_w && a->shift_state && a->rows.pos && !a->row_idx && a->x_out != a->x,
                           "stream_norm: the token shift needs a norm, its state, positions, all rows and separate streams");
  if (a->table2) RF_REQUIRE(!a->x && !a->shift && !a->row_idx && a->rows.pos && a->last_token && a->buckets > 0 && a->mul_prev >= 0 && a->mul_cur >= 0,
                            "stream_norm: token pairs need the embedding rows of all rows, positions, the carried tokens and no token shift");
  RF_REQUIRE(!a->y_self_w || (a->y_self && a->y_picks > 0), "stream_norm: the identity part belongs to picked rows");
  if (a->conv_w) RF_REQUIRE(a->conv_taps >= 1 && (a->conv_taps == 1 || a->conv_state) && a->norm_w && a->rows.pos && !a->rows.q_start && !a->shift &&
                                !a->row_idx && a->dtype != kF32 && a->H / 8 <= 1024, "stream_norm: the input convolution takes decode rows in 16 bits");
  if (a->n_rows == 0) return RF_OK;
  // halo of one row per CTA with the shift: walk several rows per CTA once that still fills the GPU
  const int rpc = (a->shift && a->rows.q_start) ? std::max(1, std::min(8, a->n_rows / (2 * sm_count()))) : 1;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int groups = a->H / 8;
  if (!a->shift && a->dtype != kF32 && groups <= 1024) {
    // decode rows: one group of columns per thread; many rows: two, so that several rows share an SM
    const int nc = groups > 512 || (groups > 256 && a->n_rows > 4 * sm_count()) ? 2 : 1;
    const dim3 block(std::max(32, round_up(ceil_div(groups, nc), 32)));
#define RF_SO(T, NC, CV) RF_CUDA_CHECK(::rf::launch_k(stream_out_kernel<T, NC, CV>, dim3(a->n_rows), block, 0, s, 1, *a))
#define RF_SO_C(T, NC) if (a->conv_w) { RF_SO(T, NC, true); } else { RF_SO(T, NC, false); }
#define RF_SO_T(T) if (nc == 1) { RF_SO_C(T, 1) } else { RF_SO_C(T, 2) }
    if (a->dtype == kF16) { RF_SO_T(__half) } else { RF_SO_T(__nv_bfloat16) }
#undef RF_SO_T
#undef RF_SO_C
#undef RF_SO
    ::rf::count_launch();
    return RF_OK;
  }
  const int quads = a->H / 4;
  if (quads <= 2048) {
    // decode rows: as many threads as there are quads (one round trip); many rows: smaller CTAs, several per SM
    const int vpt = a->n_rows > 4 * sm_count() ? (quads > 512 ? 4 : quads > 256 ? 2 : 1) : (quads > 1024 ? 2 : 1);
    const int threads = std::max(32, round_up(ceil_div(quads, vpt), 32));
    const dim3 grid(ceil_div(a->n_rows, rpc));
#define RF_SN(V) RF_DISPATCH3(a->dtype, RF_CUDA_CHECK(::rf::launch_k(stream_norm_reg_kernel<T, V>, grid, dim3(threads), 0, s, 1, *a, rpc)))
    if (vpt == 1) { RF_SN(1); } else if (vpt == 2) { RF_SN(2); } else { RF_SN(4); }
#undef RF_SN
    ::rf::count_launch();
    return RF_OK;
  }
  const int threads = 512;
  const size_t smem = ((size_t)a->H * (a->shift ? 2 : 1) + 32) * sizeof(float);
  RF_REQUIRE(smem <= 200 * 1024, "stream_norm: rows of %d values do not fit in shared memory", a->H);
  RF_DISPATCH3(a->dtype, {
    RF_ALLOW_SMEM_PER_DEVICE(stream_norm_kernel<T>, 200 * 1024);
    RF_CUDA_CHECK(::rf::launch_k(stream_norm_kernel<T>, dim3(ceil_div(a->n_rows, rpc)), dim3(threads), smem, s, 1, *a, rpc));
  });
  ::rf::count_launch();
  return RF_OK;
}

extern "C" int rf_token_gate(void* g, int64_t ldg, const void* table, int64_t ld_table, const int32_t* ids, int32_t col0,
                             int32_t rows, int32_t cols, int32_t dtype, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_REQUIRE(g && table && ids && cols % 8 == 0 && ldg % 8 == 0 && ld_table % 8 == 0 && col0 % 8 == 0, "token_gate arguments");
  if (rows == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int64_t n = (int64_t)rows * (cols / 8);
  RF_DISPATCH3(dtype, RF_CUDA_CHECK(::rf::launch_k(token_gate_kernel<T>, dim3((unsigned)((n + 127) / 128)), dim3(128), 0, s, 1,
                                                   (T*)g, ldg, (const T*)table, ld_table, ids, col0, rows, cols)));
  ::rf::count_launch();
  return RF_OK;
}

extern "C" int rf_gemm_f32(const RfGemm* g, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_REQUIRE(g && g->x && g->w && g->out && g->M >= 0 && g->N > 0 && g->K > 0, "gemm_f32 arguments");
  RF_REQUIRE(g->K % 4 == 0 && g->ldx % 4 == 0 && g->ldw % 4 == 0, "gemm_f32: K and the pitches must be multiples of 4");
  RF_REQUIRE(!g->residual && !g->bias && !g->scale && !g->w_packed && g->ar_world <= 1, "gemm_f32 has a row-scale and activation epilogue only");
  RF_REQUIRE(act_is_dual(g->act) == (g->dual_offset > 0) && g->act != kActGeluTanhMul, "dual_offset and an activation of two operands go together");
  if (g->act == kActClippedGlu || g->act == kActSoftCap) RF_REQUIRE(g->act_limit > 0.f, "this activation needs a positive limit");
  if (g->M == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid(ceil_div(g->N, kFBN), ceil_div(g->M, kFBM));
  const ActArgs args = {g->act_limit, g->act_alpha};
#define RF_F32(DUAL)                                                                                                                 \
  RF_CUDA_CHECK(::rf::launch_k(gemm_f32_kernel<DUAL>, grid, dim3(256), 0, s, 1, (const float*)g->x, g->ldx, (const float*)g->w, g->ldw, \
                               (float*)g->out, g->ldo, g->M, g->N, g->K, g->act, g->dual_offset, g->row_scale, args))
  if (g->dual_offset > 0) RF_F32(true);
  else RF_F32(false);
#undef RF_F32
  ::rf::count_launch();
  return RF_OK;
}
