// Grouped-head attention of the mixed-layer decoders: what happens between the input projection and the attention (per-head
// norms, rotation, value mixing, insertion into the K/V pages; one launch), and a plain attention kernel for models served in
// 32 bits and for head sizes that the tensor-core kernels do not take.
#include "../common/dtype.cuh"
#include "../common/host_util.h"
#include "../common/ptx.cuh"
#include "../rf_api.h"

namespace rf {

// A head of hd values is held by GL lanes, NC chunks of eight consecutive values each (hd <= 8 * GL * NC).  Groups are numbered
// over (row, item), items of a row being its query heads, key heads and value heads.
template <typename T, int GL, int NC>
__global__ void __launch_bounds__(256) qkv_insert_kernel(const RfQkvInsert p) {
  pdl_prologue();
  extern __shared__ __align__(16) float rot_buf[];
  constexpr int HPW = 32 / GL;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gl = lane % GL, sub = lane / GL;
  const int items = p.heads + 2 * p.kv_heads;
  const int64_t idx = ((int64_t)blockIdx.x * (blockDim.x >> 5) + warp) * HPW + sub;
  const bool live = idx < (int64_t)p.n_rows * items;
  const int row = live ? (int)(idx / items) : 0, item = live ? (int)(idx % items) : 0;
  const bool is_q = item < p.heads, is_v = item >= p.heads + p.kv_heads;
  const int head = is_q ? item : (is_v ? item - p.heads - p.kv_heads : item - p.heads);
  const int hd = p.hd;
  T* src = reinterpret_cast<T*>(p.qkv) + (size_t)row * p.ld + (is_q ? 0 : (is_v ? p.v_off : p.k_off)) + (size_t)head * hd;
  const int pos = p.rows.pos[row];
  float x[NC][8];
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int o = (gl + c * GL) * 8;
    if (live && o < hd) load8(src + o, x[c]);
    else {
#pragma unroll
      for (int j = 0; j < 8; ++j) x[c][j] = 0.f;
    }
  }
  const float* nw = is_v ? nullptr : (is_q ? p.q_norm : p.k_norm);
  float ss = 0.f;
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += x[c][j] * x[c][j];
#pragma unroll
  for (int d = GL / 2; d >= 1; d >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, d);
  if (nw) {
    const float rstd = rsqrtf(ss / (float)p.dim + p.eps);
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int o = (gl + c * GL) * 8;
      if (o < hd) {
#pragma unroll
        for (int j = 0; j < 8; ++j) x[c][j] *= rstd * nw[o + j];
      }
    }
  }
  if (p.rot_dims > 0) {                            // uniform over the grid
    float* buf = rot_buf + (size_t)(warp * HPW + sub) * p.rot_dims;
    const int half = p.rot_dims >> 1;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int o = (gl + c * GL) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (o + j < p.rot_dims) buf[o + j] = x[c][j];
    }
    __syncwarp();
    if (live && !is_v) {
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
  if (!live) return;
  if (is_v && p.v_role != RF_VMIX_NONE) {
    T* first = reinterpret_cast<T*>(p.v_first) + (size_t)row * p.kv_heads * p.vdim + (size_t)head * p.vdim;
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
  T* dst = src;
  if (!is_q) {
    const int seq = p.rows.seq_of_row ? p.rows.seq_of_row[row] : row;
    const int slot = p.rows.slot ? p.rows.slot[seq] : seq;
    const int page = p.rows.page_table[(size_t)slot * p.rows.pt_stride + (pos >> 4)];
    dst = reinterpret_cast<T*>(is_v ? p.v_pool : p.k_pool) + (((size_t)page * p.kv_heads + head) * 16 + (pos & 15)) * hd;
  }
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int o = (gl + c * GL) * 8;
    if (o < hd) store8(dst + o, x[c]);
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
  const int lo = p.chunk > 0 ? pos / p.chunk * p.chunk : 0;
  for (int i = threadIdx.x; i < hd; i += blockDim.x)
    q[i] = Num<T>::to_f(reinterpret_cast<const T*>(p.q)[(size_t)row * p.ldq + (size_t)h * hd + i]);
  for (int i = lane; i < hd; i += 32) acc[i] = 0.f;
  __syncthreads();
  float m = -INFINITY, l = 0.f;
  for (int j = lo + warp; j <= pos; j += 4) {
    const int page = p.page_table[(size_t)pt_row * p.pt_stride + (j >> 4)];
    const size_t at = (((size_t)page * p.Hkv + kvh) * 16 + (j & 15)) * hd;
    const T* k = reinterpret_cast<const T*>(p.k_pool) + at;
    const T* v = reinterpret_cast<const T*>(p.v_pool) + at;
    float s = 0.f;
    for (int i = lane; i < hd; i += 32) s += q[i] * Num<T>::to_f(k[i]);
    s = warp_sum(s) * p.scale;
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
    if (p.gate) o *= 1.f / (1.f + expf(-Num<T>::to_f(reinterpret_cast<const T*>(p.gate)[(size_t)row * p.ld_gate + col])));
    reinterpret_cast<T*>(p.out)[(size_t)row * p.ldo + col] = Num<T>::from_f(o);
  }
}

template <typename T, int GL, int NC>
static int launch_qkv_insert(const RfQkvInsert* a, cudaStream_t s) {
  const int64_t groups = (int64_t)a->n_rows * (a->heads + 2 * a->kv_heads);
  const int warps = groups * GL / 32 < 8 * sm_count() ? 2 : 8, per_block = warps * (32 / GL);
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
  RF_REQUIRE(a->window <= 0 && !a->mask && !a->seg_q && a->dtype >= 0 && a->dtype <= 2, "attn_rows: options");
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
