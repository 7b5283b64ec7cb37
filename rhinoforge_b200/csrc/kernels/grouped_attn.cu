// Grouped-head attention of the mixed-layer decoders: what happens between the input projection and the attention (causal
// convolution, norms, rotation, value mixing, insertion into the K/V pages; one launch), and a plain attention kernel for models served in
// 32 bits and for head sizes that the tensor-core kernels do not take.
#include "../common/dtype.cuh"
#include "../common/host_util.h"
#include "../common/ptx.cuh"
#include "../rf_api.h"

namespace rf {

// A head of hd values is held by GL lanes, NC chunks of eight consecutive values each (hd <= 8 * GL * NC).  The items of a row are
// its query heads, key heads and value heads.
struct HeadItem {
  int row, item, head;
  bool is_q, is_v, live;
  __device__ __forceinline__ HeadItem(const RfQkvInsert& p, int row_, int item_, bool live_)
      : row(row_), item(item_), is_q(item_ < p.heads), is_v(item_ >= p.heads + p.kv_heads), live(live_) {
    head = is_q ? item : (is_v ? item - p.heads - p.kv_heads : item - p.heads);
  }
  template <typename T>
  __device__ __forceinline__ T* source(const RfQkvInsert& p) const {
    return reinterpret_cast<T*>(p.qkv) + (size_t)row * p.ld + (is_q ? 0 : (is_v ? p.v_off : p.k_off)) + (size_t)head * p.hd;
  }
};

// 1 / rms of this group's head (all lanes of the warp).
template <int GL, int NC>
__device__ __forceinline__ float head_rstd(const RfQkvInsert& p, const float (&x)[NC][8]) {
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += x[c][j] * x[c][j];
#pragma unroll
  for (int d = GL / 2; d >= 1; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
  return rsqrtf(ss / (float)p.dim + p.eps);
}

// Page-table row of the sequence that owns a row.
__device__ __forceinline__ int slot_of_row(const RfQkvInsert& p, int row) {
  const int seq = p.rows.seq_of_row ? p.rows.seq_of_row[row] : row;
  return p.rows.slot ? p.rows.slot[seq] : seq;
}

// Norm with `rstd`, rotation, value mixing and the store of one head at position pos; all lanes of the warp, buf: the group's scratch.
template <typename T, int GL, int NC>
__device__ __forceinline__ void finish_head(const RfQkvInsert& p, const HeadItem& it, int pos, int slot, float (&x)[NC][8], float rstd, int gl,
                                            float* buf) {
  const int hd = p.hd;
  const float* nw = it.is_v ? nullptr : (it.is_q ? p.q_norm : p.k_norm);
  if (nw) {
    if (p.norm_all) nw += (size_t)it.head * hd;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int o = (gl + c * GL) * 8;
      if (o < hd) {
#pragma unroll
        for (int j = 0; j < 8; ++j) x[c][j] *= rstd * nw[o + j];
      }
    }
  }
  if (it.is_q && p.growth_every > 0) {             // queries grow with their position
    const float f = 1.f + p.growth * logf((float)((pos + 1) / p.growth_every) + 1.f);
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
      for (int j = 0; j < 8; ++j) x[c][j] *= f;
  }
  const int half = p.rot_dims >> 1;                // uniform over the grid
  if (NC == 1 && half > 0 && half % 8 == 0) {
    // whole lanes turn with one another: dimensions of lane l with those of lane l + half / 8
    const int hl = half >> 3, with = gl < hl ? gl + hl : (gl < 2 * hl ? gl - hl : gl), lane = threadIdx.x & 31;
    const bool turns = it.live && !it.is_v && gl < 2 * hl;
    const size_t at = (size_t)pos * half + (gl < hl ? gl : gl - hl) * 8;
    float cs[8], sn[8];
    if (turns) {
      load8(p.cos + at, cs);
      load8(p.sin + at, sn);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float other = __shfl_sync(0xffffffffu, x[0][j], lane - gl + with);
      if (turns) x[0][j] = x[0][j] * cs[j] + (gl < hl ? -other : other) * sn[j];
    }
  } else if (half > 0) {
    __syncwarp();
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int o = (gl + c * GL) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (o + j < p.rot_dims) buf[o + j] = x[c][j];
    }
    __syncwarp();
    if (it.live && !it.is_v) {
      const float* cs = p.cos + (size_t)pos * half;
      const float* sn = p.sin + (size_t)pos * half;
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const int o = (gl + c * GL) * 8;
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const int i = o + j;
          if (i < half) x[c][j] = x[c][j] * cs[i] - buf[i + half] * sn[i];
          else if (i < p.rot_dims) x[c][j] = x[c][j] * cs[i - half] + buf[i - half] * sn[i - half];
        }
      }
    }
  }
  if (!it.live) return;
  if (it.is_v && p.v_role != RF_VMIX_NONE) {
    T* first = reinterpret_cast<T*>(p.v_first) + (size_t)it.row * p.kv_heads * p.vdim + (size_t)it.head * p.vdim;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int o = (gl + c * GL) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        if (o + j >= p.vdim) continue;
        if (p.v_role == RF_VMIX_FIRST) first[o + j] = Num<T>::from_f(x[c][j]);
        else x[c][j] = (1.f - p.v_lambda) * x[c][j] + p.v_lambda * Num<T>::to_f(first[o + j]);
      }
    }
  }
  T* dst;
  if (it.is_q) {
    dst = p.q_out ? reinterpret_cast<T*>(p.q_out) + ((size_t)it.row * p.heads + it.head) * hd : it.source<T>(p);
  } else {
    const int page = p.rows.page_table[(size_t)slot * p.rows.pt_stride + (pos >> 4)];
    dst = reinterpret_cast<T*>(it.is_v ? p.v_pool : p.k_pool) + (((size_t)page * p.kv_heads + it.head) * 16 + (pos & 15)) * hd;
  }
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int o = (gl + c * GL) * 8;
    if (o < hd) store8(dst + o, x[c]);
  }
}

template <typename T, int GL, int NC>
__device__ __forceinline__ void load_head(const T* src, bool live, int hd, int gl, float (&x)[NC][8]) {
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int o = (gl + c * GL) * 8;
    if (live && o < hd) load8(src + o, x[c]);
    else {
#pragma unroll
      for (int j = 0; j < 8; ++j) x[c][j] = 0.f;
    }
  }
}

// Groups are numbered over (row, item).
template <typename T, int GL, int NC>
__global__ void __launch_bounds__(256) qkv_insert_kernel(const RfQkvInsert p) {
  pdl_prologue();
  extern __shared__ __align__(16) float rot_buf[];
  constexpr int HPW = 32 / GL;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gl = lane % GL, sub = lane / GL;
  const int items = p.heads + 2 * p.kv_heads;
  const int64_t idx = ((int64_t)blockIdx.x * (blockDim.x >> 5) + warp) * HPW + sub;
  const bool live = idx < (int64_t)p.n_rows * items;
  const HeadItem it(p, live ? (int)(idx / items) : 0, live ? (int)(idx % items) : 0, live);
  float x[NC][8];
  load_head<T, GL, NC>(it.source<T>(p), live, p.hd, gl, x);
  finish_head<T, GL, NC>(p, it, p.rows.pos[it.row], slot_of_row(p, it.row), x, head_rstd<GL, NC>(p, x), gl,
                         rot_buf + (size_t)(warp * HPW + sub) * p.rot_dims);
}

// One norm over all query heads of a row and one over all key heads: a CTA per row, which is read twice.
template <typename T, int GL, int NC>
__global__ void __launch_bounds__(256) qkv_insert_row_kernel(const RfQkvInsert p) {
  pdl_prologue();
  extern __shared__ __align__(16) float rot_buf[];
  __shared__ float red[2][8];
  constexpr int HPW = 32 / GL;
  const int warp = threadIdx.x >> 5, nw = blockDim.x >> 5, lane = threadIdx.x & 31, gl = lane % GL, sub = lane / GL;
  const int row = blockIdx.x, items = p.heads + 2 * p.kv_heads, groups = nw * HPW, qn = p.heads * p.hd / 8, kn = p.kv_heads * p.hd / 8;
  const T* src = reinterpret_cast<const T*>(p.qkv) + (size_t)row * p.ld;
  const int pos = p.rows.pos[row], slot = slot_of_row(p, row);
  float sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x; i < qn + kn; i += blockDim.x) {
    float f[8], s = 0.f;
    load8(i < qn ? src + i * 8 : src + p.k_off + (i - qn) * 8, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) s += f[j] * f[j];
    if (i < qn) sq += s;
    else sk += s;
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
  __syncthreads();
  sq = sk = 0.f;
  for (int w = 0; w < nw; ++w) { sq += red[0][w]; sk += red[1][w]; }
  const float rq = rsqrtf(sq / (float)(p.heads * p.dim) + p.eps), rk = rsqrtf(sk / (float)(p.kv_heads * p.dim) + p.eps);
  for (int i0 = 0; i0 < items; i0 += groups) {
    const int item = i0 + warp * HPW + sub;
    const bool live = item < items;
    const HeadItem it(p, row, live ? item : 0, live);
    float x[NC][8];
    load_head<T, GL, NC>(it.source<T>(p), live, p.hd, gl, x);
    finish_head<T, GL, NC>(p, it, pos, slot, x, it.is_q ? rq : rk, gl, rot_buf + (size_t)(warp * HPW + sub) * p.rot_dims);
  }
}

// With the convolution: a group walks `tile` neighbouring rows of one sequence for its head, four at a time, the last inputs and the
// next four rows in registers (TAPS = 0: any number of taps, every input read again for each of them).  The group of a sequence's first rows also replaces the
// carried inputs; later tiles find theirs among the rows of this launch.
template <typename T, int GL, int NC, int TAPS>
__global__ void __launch_bounds__(128) qkv_conv_insert_kernel(const RfQkvInsert p, int tile) {
  pdl_prologue();
  extern __shared__ __align__(16) float rot_buf[];
  constexpr int HPW = 32 / GL;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gl = lane % GL, sub = lane / GL;
  const int items = p.heads + 2 * p.kv_heads, hd = p.hd, seq = blockIdx.z, past = (TAPS > 0 ? TAPS : p.taps) - 1;
  const int q0 = p.rows.q_start ? p.rows.q_start[seq] : seq, n = p.rows.q_len ? p.rows.q_len[seq] : 1;
  const int t0 = blockIdx.y * tile, t1 = min(n, t0 + tile);
  if (t0 >= n) return;
  const int item = (blockIdx.x * (blockDim.x >> 5) + warp) * HPW + sub;
  const bool live = item < items;
  const int pos0 = p.rows.pos[q0], slot = p.rows.slot ? p.rows.slot[seq] : seq;       // positions of a portion follow one another
  const size_t channels = (size_t)items * hd, at = (size_t)(live ? item : 0) * hd;
  T* state = reinterpret_cast<T*>(p.conv_state) + (size_t)slot * past * channels + at;
  const T* src = reinterpret_cast<const T*>(p.qkv) + (size_t)q0 * p.ld + at;
  const float* w = p.conv_w + at;
  float* buf = rot_buf + (size_t)(warp * HPW + sub) * p.rot_dims;
  // input at place i of this launch's rows; negative places are carried ones
  auto input_at = [&](int i) -> const T* {
    return i >= 0 ? src + (size_t)i * p.ld : (pos0 > 0 ? state + (size_t)(past + i) * channels : nullptr);
  };
  auto input = [&](int i, float (&f)[NC][8]) {
    const T* q = input_at(i);
    load_head<T, GL, NC>(q, live && q != nullptr, hd, gl, f);
  };
  auto finish = [&](int t, float (&x)[NC][8]) {
    const HeadItem it(p, q0 + t, live ? item : 0, live);
    finish_head<T, GL, NC>(p, it, pos0 + t, slot, x, head_rstd<GL, NC>(p, x), gl, buf);
  };
  if constexpr (TAPS > 0 && NC == 1) {
    constexpr int R = 4;
    const bool mine = live && gl * 8 < hd;
    Vec8<T> old[TAPS - 1], cur[R], nxt[R];
    float wt[TAPS][1][8];
    auto fetch = [&](int i, bool in) -> Vec8<T> {
      const float zero[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      Vec8<T> v;
      const T* q = in && mine ? input_at(i) : nullptr;
      if (q) v = *reinterpret_cast<const Vec8<T>*>(q + gl * 8);
      else store8(reinterpret_cast<T*>(&v), zero);
      return v;
    };
#pragma unroll
    for (int r = 0; r < R; ++r) nxt[r] = fetch(t0 + r, t0 + r < t1);
#pragma unroll
    for (int k = 0; k < TAPS - 1; ++k) old[k] = fetch(t0 - (TAPS - 1) + k, true);
#pragma unroll
    for (int k = 0; k < TAPS; ++k) load_head<float, GL, 1>(w + k * channels, live, hd, gl, wt[k]);
    for (int t = t0; t < t1; t += R) {
#pragma unroll
      for (int r = 0; r < R; ++r) {
        cur[r] = nxt[r];
        nxt[r] = fetch(t + R + r, t + R + r < t1);
      }
#pragma unroll
      for (int r = 0; r < R; ++r) {
        if (t + r >= t1) break;
        float x[1][8];
#pragma unroll
        for (int j = 0; j < 8; ++j) x[0][j] = 0.f;
#pragma unroll
        for (int k = 0; k < TAPS; ++k) {
          const int i = r - (TAPS - 1) + k;
          const Vec8<T> v = i < 0 ? old[i < 0 ? TAPS - 1 + i : 0] : cur[i < 0 ? 0 : i];
          float f[8];
          load8(reinterpret_cast<const T*>(&v), f);
#pragma unroll
          for (int j = 0; j < 8; ++j) x[0][j] += wt[k][0][j] * f[j];
        }
        finish(t + r, x);
      }
      static_assert(TAPS - 1 <= R, "the last inputs lie in the rows just done");
#pragma unroll
      for (int k = 0; k < TAPS - 1; ++k) old[k] = cur[R - (TAPS - 1) + k];
    }
  } else {
    for (int t = t0; t < t1; ++t) {
      float x[NC][8], f[NC][8], v[NC][8];
#pragma unroll
      for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int j = 0; j < 8; ++j) x[c][j] = 0.f;
      for (int k = 0; k <= past; ++k) {
        load_head<float, GL, NC>(w + k * channels, live, hd, gl, f);
        input(t - past + k, v);
#pragma unroll
        for (int c = 0; c < NC; ++c)
#pragma unroll
          for (int j = 0; j < 8; ++j) x[c][j] += f[c][j] * v[c][j];
      }
      finish(t, x);
    }
  }
  if (blockIdx.y == 0 && live)
    for (int i = 0; i < past; ++i) {             // ascending: row i comes from a later row of the old state, or from this launch
      float v[NC][8];
      input(n - past + i, v);
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const int o = (gl + c * GL) * 8;
        if (o < hd) store8(state + (size_t)i * channels + o, v[c]);
      }
    }
}

// One CTA per (row, query head): four warps walk the visible keys, lanes share the head dimension, everything in fp32.
template <typename T>
__global__ void __launch_bounds__(128) attn_rows_kernel(const RfAttn p) {
  pdl_prologue();
  extern __shared__ __align__(16) float ar_sm[];
  const int h = blockIdx.x, row = blockIdx.y, hd = p.hd, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float* q = ar_sm;
  float* acc = ar_sm + hd * (1 + warp);
  float* ml = ar_sm + hd * 5;
  const int seq = p.seq_of_row ? p.seq_of_row[row] : row, pt_row = p.slot ? p.slot[seq] : seq;
  const int pos = p.pos[row], kvh = h / (p.Hq / p.Hkv);
  int lo = p.chunk > 0 ? pos / p.chunk * p.chunk : 0;
  if (p.window > 0) lo = max(lo, pos - p.window + 1);
  const int keep = min(p.keep_first, lo);          // visible positions: [0, keep) and [lo, pos]
  const float fall = p.slopes ? p.slopes[h] : 0.f;
  for (int i = threadIdx.x; i < hd; i += blockDim.x)
    q[i] = Num<T>::to_f(reinterpret_cast<const T*>(p.q)[(size_t)row * p.ldq + (size_t)h * hd + i]);
  for (int i = lane; i < hd; i += 32) acc[i] = 0.f;
  __syncthreads();
  float m = -INFINITY, l = 0.f;
  for (int n = warp; n < keep + pos - lo + 1; n += 4) {
    const int j = n < keep ? n : n - keep + lo;
    const int page = p.page_table[(size_t)pt_row * p.pt_stride + (j >> 4)];
    const size_t at = (((size_t)page * p.Hkv + kvh) * 16 + (j & 15)) * hd;
    const T* k = reinterpret_cast<const T*>(p.k_pool) + at;
    const T* v = reinterpret_cast<const T*>(p.v_pool) + at;
    float s = 0.f;
    for (int i = lane; i < hd; i += 32) s += q[i] * Num<T>::to_f(k[i]);
    const float dist = (float)(pos - j);
    s = warp_sum(s) * p.scale - fall * (p.rates ? logf(1.f + p.rates[h] * dist) : dist);
    const float mn = fmaxf(m, s), keep = expf(m - mn), w = expf(s - mn);
    l = l * keep + w;
    m = mn;
    for (int i = lane; i < hd; i += 32) acc[i] = acc[i] * keep + w * Num<T>::to_f(v[i]);
  }
  if (lane == 0) { ml[warp] = m; ml[4 + warp] = l; }
  __syncthreads();
  float top = -INFINITY;
  for (int w = 0; w < 4; ++w) top = fmaxf(top, ml[w]);
  if (p.sink) top = fmaxf(top, p.sink[h]);
  float den = p.sink ? expf(p.sink[h] - top) : 0.f, f[4];
  for (int w = 0; w < 4; ++w) {
    f[w] = expf(ml[w] - top);
    den += f[w] * ml[4 + w];
  }
  for (int i = threadIdx.x; i < hd; i += blockDim.x) {
    float o = 0.f;
    for (int w = 0; w < 4; ++w) o += f[w] * ar_sm[hd * (1 + w) + i];
    o /= den;
    const size_t col = (size_t)h * hd + i;
    if (p.gate) o *= 1.f / (1.f + expf(-Num<T>::to_f(reinterpret_cast<const T*>(p.gate)[(size_t)row * p.ld_gate + (p.gate_by_head ? h : col)])));
    reinterpret_cast<T*>(p.out)[(size_t)row * p.ldo + col] = Num<T>::from_f(o);
  }
}

template <typename T, int GL, int NC, int TAPS>
static int launch_qkv_conv(const RfQkvInsert* a, cudaStream_t s) {
  const int items = a->heads + 2 * a->kv_heads, hpw = 32 / GL, warps = std::min(4, ceil_div(items, hpw)), per_block = warps * hpw;
  const int tile = std::max(16, a->taps - 1);      // later tiles find their past in the rows of this launch
  const size_t smem = (size_t)per_block * a->rot_dims * sizeof(float);
  RF_ALLOW_SMEM_PER_DEVICE((qkv_conv_insert_kernel<T, GL, NC, TAPS>), 64 * 1024);
  const dim3 grid(ceil_div(items, per_block), ceil_div(a->max_q_len, tile), a->rows.num_seqs);
  RF_CUDA_CHECK(::rf::launch_k(qkv_conv_insert_kernel<T, GL, NC, TAPS>, grid, dim3(warps * 32), smem, s, 1, *a, tile));
  ::rf::count_launch();
  return RF_OK;
}

template <typename T, int GL, int NC>
static int launch_qkv_insert(const RfQkvInsert* a, cudaStream_t s) {
  const int64_t groups = (int64_t)a->n_rows * (a->heads + 2 * a->kv_heads);
  const int warps = groups * GL / 32 < 8 * sm_count() ? 2 : 8, per_block = warps * (32 / GL);
  if (a->taps > 0) {
    if (NC > 1) return launch_qkv_conv<T, GL, NC, 0>(a, s);
    switch (a->taps) {
      case 2: return launch_qkv_conv<T, GL, NC, NC == 1 ? 2 : 0>(a, s);
      case 3: return launch_qkv_conv<T, GL, NC, NC == 1 ? 3 : 0>(a, s);
      case 4: return launch_qkv_conv<T, GL, NC, NC == 1 ? 4 : 0>(a, s);
      default: return launch_qkv_conv<T, GL, NC, 0>(a, s);
    }
  }
  if (a->norm_all) {
    const int threads = 256;
    const size_t smem = (size_t)(threads / GL) * a->rot_dims * sizeof(float);
    RF_ALLOW_SMEM_PER_DEVICE((qkv_insert_row_kernel<T, GL, NC>), 64 * 1024);
    RF_CUDA_CHECK(::rf::launch_k(qkv_insert_row_kernel<T, GL, NC>, dim3(a->n_rows), dim3(threads), smem, s, 1, *a));
    ::rf::count_launch();
    return RF_OK;
  }
  const size_t smem = (size_t)per_block * a->rot_dims * sizeof(float);
  RF_ALLOW_SMEM_PER_DEVICE((qkv_insert_kernel<T, GL, NC>), 64 * 1024);
  RF_CUDA_CHECK(::rf::launch_k(qkv_insert_kernel<T, GL, NC>, dim3((unsigned)((groups + per_block - 1) / per_block)), dim3(warps * 32),
                               smem, s, 1, *a));
  ::rf::count_launch();
  return RF_OK;
}

template <typename T>
static int dispatch_qkv_insert(const RfQkvInsert* a, cudaStream_t s) {
  const int chunks = a->hd / 8;
  if (chunks <= 2) return launch_qkv_insert<T, 2, 1>(a, s);
  if (chunks <= 4) return launch_qkv_insert<T, 4, 1>(a, s);
  if (chunks <= 8) return launch_qkv_insert<T, 8, 1>(a, s);
  if (chunks <= 16) return launch_qkv_insert<T, 16, 1>(a, s);
  if (chunks <= 32) return launch_qkv_insert<T, 32, 1>(a, s);
  return launch_qkv_insert<T, 32, 4>(a, s);
}

}  // namespace rf

using namespace rf;

extern "C" int rf_qkv_insert(const RfQkvInsert* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_REQUIRE(a && a->qkv && a->k_pool && a->v_pool && a->rows.pos && a->rows.page_table, "qkv_insert: missing buffers");
  RF_REQUIRE(a->hd > 0 && a->hd % 8 == 0 && a->hd <= 1024 && a->dim > 0 && a->dim <= a->hd && a->vdim > 0 && a->vdim <= a->hd,
             "qkv_insert: head sizes %d / %d in %d", a->dim, a->vdim, a->hd);
  RF_REQUIRE(a->ld % 8 == 0 && a->k_off % 8 == 0 && a->v_off % 8 == 0 && a->heads > 0 && a->kv_heads > 0, "qkv_insert: row layout");
  RF_REQUIRE(a->rot_dims >= 0 && a->rot_dims % 2 == 0 && a->rot_dims <= a->dim && (a->rot_dims == 0 || (a->cos && a->sin)),
             "qkv_insert: rotation of %d dimensions", a->rot_dims);
  RF_REQUIRE(a->v_role == RF_VMIX_NONE || a->v_first, "qkv_insert: value mixing needs the first values");
  RF_REQUIRE(a->dtype >= 0 && a->dtype <= 2, "qkv_insert: dtype %d", a->dtype);
  RF_REQUIRE(a->growth_every >= 0, "qkv_insert: growth of the queries");
  if (a->taps > 0) {
    RF_REQUIRE(a->conv_w && a->q_out && a->q_out != a->qkv && (a->taps == 1 || a->conv_state) && !a->norm_all,
               "qkv_insert: the convolution needs weights, its state and an output for the queries, and per-head norms");
    RF_REQUIRE(a->k_off == a->heads * a->hd && a->v_off == (a->heads + a->kv_heads) * a->hd, "qkv_insert: queries, keys and values are neighbours");
    RF_REQUIRE(a->max_q_len >= 1 && a->rows.num_seqs <= 65535 && (int64_t)a->max_q_len <= 16ll * 65535, "qkv_insert: %d sequences of up to %d rows",
               a->rows.num_seqs, a->max_q_len);
    if (a->rows.num_seqs == 0) return RF_OK;
  }
  if (a->n_rows == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (a->dtype == kF16) return dispatch_qkv_insert<__half>(a, s);
  if (a->dtype == kBF16) return dispatch_qkv_insert<__nv_bfloat16>(a, s);
  return dispatch_qkv_insert<float>(a, s);
}

extern "C" int rf_attn_rows(const RfAttn* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_REQUIRE(a && a->q && a->out && a->k_pool && a->v_pool && a->page_table && a->pos, "attn_rows: missing buffers");
  RF_REQUIRE(a->hd > 0 && a->hd <= 2048 && a->Hkv > 0 && a->Hq % a->Hkv == 0, "attn_rows: heads");
  RF_REQUIRE(a->keep_first >= 0 && !a->mask && !a->seg_q && a->dtype >= 0 && a->dtype <= 2, "attn_rows: options");
  RF_REQUIRE(!a->rates || a->slopes, "attn_rows: the rates of a logarithmic fall need its slopes");
  RF_REQUIRE(a->num_seqs <= 65535, "attn_rows: %d rows in one launch", a->num_seqs);
  if (a->num_seqs == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const size_t smem = ((size_t)a->hd * 5 + 8) * sizeof(float);
  const dim3 grid(a->Hq, a->num_seqs);
  if (a->dtype == kF16) RF_CUDA_CHECK(::rf::launch_k(attn_rows_kernel<__half>, grid, dim3(128), smem, s, 1, *a));
  else if (a->dtype == kBF16) RF_CUDA_CHECK(::rf::launch_k(attn_rows_kernel<__nv_bfloat16>, grid, dim3(128), smem, s, 1, *a));
  else RF_CUDA_CHECK(::rf::launch_k(attn_rows_kernel<float>, grid, dim3(128), smem, s, 1, *a));
  ::rf::count_launch();
  return RF_OK;
}
