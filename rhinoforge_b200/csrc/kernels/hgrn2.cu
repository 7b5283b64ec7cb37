// HGRN2 linear attention: the forget gate of a channel also decides how much of the value is written,
//   S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T,   o_t = S_t^T q_t,
// with an fp32 state per (slot, head), q = silu(.), f = lower + (1 - lower) sigmoid(. + bias), and an RMSNorm per head on o.
//   * rf_hgrn2_recurrent: token by token (decode steps, short portions, everything in fp32),
//   * rf_hgrn2_chunked: block by block on the tensor cores (prefill-sized portions).
#include "../common/dtype.cuh"
#include "../common/host_util.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"
#include "../rf_api.h"

namespace rf {

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.f / (1.f + expf(-x)); }

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
    for (int r = 0; r < RPT; ++r) st[r] = (on && !fresh && row0 + r < p.dim) ? S[(size_t)(row0 + r) * p.vdim + j] : 0.f;
  }
  const float nw = (p.norm_w && on) ? p.norm_w[j] : 1.f;
  for (int t = 0; t < n; ++t) {
    const int buf = t & 1;
    const T* xr = x + (size_t)(q0 + t) * p.ldx;
    for (int i = threadIdx.x; i < p.dim; i += blockDim.x) {
      const int ch = head * p.dim + i;
      const float qv = Num<T>::to_f(xr[ch]);
      sq[buf * p.dim + i] = qv * sigmoid_f32(qv);
      const float lo = p.lower[ch];
      sf[buf * p.dim + i] = lo + (1.f - lo) * sigmoid_f32(Num<T>::to_f(xr[p.f_off + ch]) + p.f_bias[ch]);
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
      for (int w = 0; w < (int)((blockDim.x + 31) / 32); ++w) tot += ws[w];
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
        if (row0 + r < p.dim) S[(size_t)(row0 + r) * p.vdim + j] = st[r];
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
  if (a->dtype == kF32) return launch_recurrent<float>(a, s);
  if (a->dtype == kF16) return launch_recurrent<__half>(a, s);
  return launch_recurrent<__nv_bfloat16>(a, s);
}

extern "C" int rf_hgrn2_chunked_supported(int dim, int vdim, int dtype) {
  (void)dim; (void)vdim; (void)dtype;
  return 0;
}

extern "C" int rf_hgrn2_chunked(const RfHgrn2* a, rf_stream_t stream) { return rf_hgrn2_recurrent(a, stream); }
