// Gated delta rule of the mixed-layer decoders, for any head sizes.  Per head, with unit vectors q (times dim^-1/2) and k:
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q,
//   g = exp(-rate * softplus(a + dt_bias)), beta = sigmoid(b),   out = o / rms(o) * norm_w * silu(gate)
//   * rf_delta_recurrent: token by token (decode steps, short portions, everything in 32 bits); in decode steps the short
//     convolution of queries, keys and values runs inside it,
//   * rf_delta_chunked: 64 tokens at a time on the tensor cores (prefill-sized portions).
// The state is fp32, and so is all that enters the recurrence behind the convolutions.
#include "../common/dtype.cuh"
#include "../common/host_util.h"
#include "../common/ptx.cuh"
#include "../rf_api.h"

namespace rf {

__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float sigmoid_f(float v) { return 1.f / (1.f + expf(-v)); }

constexpr int kDrCols = 8;            // a warp covers 8 quads of state columns ...
constexpr int kDrRows = 4;            // ... times 4 groups of state rows

// One CTA per (head, sequence).  Warps lie side by side over blocks of 32 state columns (`col_blocks`) and over row blocks; a
// thread holds RPT rows of four columns in registers, rows interleaved over the row groups.
template <typename T, int RPT, bool CONV>
__global__ void __launch_bounds__(512) delta_recurrent_kernel(const RfDelta p, int col_blocks, int row_blocks) {
  pdl_prologue();
  extern __shared__ __align__(16) float dsm[];
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int D = p.dim, V = p.vdim, per = p.heads / p.kv_heads, hk = h / per;
  float* sq = dsm;                      // [D] q, [D] k, [V] v of the current token
  float* sk = sq + D;
  float* sv = sk + D;
  float* red = sv + V;                  // [2][row_blocks][V] partial sums over the state rows
  float* part = red + 2 * row_blocks * V;   // [16] sums of squares by warp
  const int cb = warp % col_blocks, rb = warp / col_blocks, col = cb * 32 + (lane % kDrCols) * 4, rg = rb * kDrRows + lane / kDrCols;
  const int groups = row_blocks * kDrRows;
  const bool live = col < V;            // V is a multiple of 8
  const int q0 = p.rows.q_start ? p.rows.q_start[seq] : seq, n = p.rows.q_len ? p.rows.q_len[seq] : 1;
  const int slot = p.rows.slot ? p.rows.slot[seq] : seq, pos0 = p.rows.pos[q0];
  float* S = p.state + ((size_t)slot * p.heads + h) * D * V;
  const int ko = p.kv_heads * D, vo = 2 * ko;
  float4 st[RPT];
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int row = rg + r * groups;
    st[r] = live && pos0 > 0 && row < D ? *reinterpret_cast<const float4*>(S + (size_t)row * V + col) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const float rate = p.rate[h], dt_bias = p.dt_bias[h], q_scale = rsqrtf((float)p.dim_true);
  for (int t = 0; t < n; ++t) {
    const size_t row = (size_t)(q0 + t);
    const T* x = reinterpret_cast<const T*>(p.x) + row * p.ldx;
    for (int i = tid; i < 2 * D + V; i += blockDim.x) {
      const int c = i < D ? hk * D + i : i < 2 * D ? ko + hk * D + i - D : vo + h * V + i - 2 * D;
      float f = Num<T>::to_f(x[c]);
      if constexpr (CONV) {
        // ring of the last `taps` inputs: rows of positions pos - taps + 1 .. pos - 1 are read, the one of pos is written; heads that
        // share a query / key head write the same value
        const int taps = p.taps, channels = vo + p.heads * V;
        T* ring = reinterpret_cast<T*>(p.conv_state) + (size_t)slot * taps * channels + c;
        float s = f * p.conv_w[(size_t)(taps - 1) * channels + c];
        for (int k = 1; k < taps; ++k)
          if (pos0 - k >= 0) s += Num<T>::to_f(ring[(size_t)((pos0 - k) % taps) * channels]) * p.conv_w[(size_t)(taps - 1 - k) * channels + c];
        ring[(size_t)(pos0 % taps) * channels] = x[c];
        f = s * sigmoid_f(s);
      }
      dsm[i] = f;
    }
    const float beta = sigmoid_f(Num<T>::to_f(reinterpret_cast<const T*>(p.b)[row * p.ld_ba + h]));
    const float decay = expf(-rate * softplus_f(Num<T>::to_f(reinterpret_cast<const T*>(p.a)[row * p.ld_ba + h]) + dt_bias));
    __syncthreads();
    float q2 = 0.f, k2 = 0.f;                       // every warp for itself
    for (int i = lane; i < D; i += 32) {
      q2 += sq[i] * sq[i];
      k2 += sk[i] * sk[i];
    }
    const float qn = rsqrtf(warp_sum(q2) + 1e-6f) * q_scale, kn = rsqrtf(warp_sum(k2) + 1e-6f);
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      const int i = rg + r * groups;
      const float k = i < D ? sk[i] * kn : 0.f;
      st[r].x *= decay; st[r].y *= decay; st[r].z *= decay; st[r].w *= decay;
      acc.x += st[r].x * k; acc.y += st[r].y * k; acc.z += st[r].z * k; acc.w += st[r].w * k;
    }
    auto over_groups = [&](float4 v) {
#pragma unroll
      for (int o = kDrCols; o < 32; o <<= 1) {
        v.x += __shfl_xor_sync(0xffffffffu, v.x, o);
        v.y += __shfl_xor_sync(0xffffffffu, v.y, o);
        v.z += __shfl_xor_sync(0xffffffffu, v.z, o);
        v.w += __shfl_xor_sync(0xffffffffu, v.w, o);
      }
      return v;
    };
    acc = over_groups(acc);
    if (live && lane < kDrCols) *reinterpret_cast<float4*>(red + rb * V + col) = acc;
    __syncthreads();
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
    if (live) {
      float4 m = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int b = 0; b < row_blocks; ++b) {
        const float4 v = *reinterpret_cast<const float4*>(red + b * V + col);
        m.x += v.x; m.y += v.y; m.z += v.z; m.w += v.w;
      }
      const float4 v = *reinterpret_cast<const float4*>(sv + col);
      u = make_float4((v.x - m.x) * beta, (v.y - m.y) * beta, (v.z - m.z) * beta, (v.w - m.w) * beta);
    }
    acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      const int i = rg + r * groups;
      const float k = i < D ? sk[i] * kn : 0.f, q = i < D ? sq[i] * qn : 0.f;
      st[r].x += k * u.x; st[r].y += k * u.y; st[r].z += k * u.z; st[r].w += k * u.w;
      acc.x += st[r].x * q; acc.y += st[r].y * q; acc.z += st[r].z * q; acc.w += st[r].w * q;
    }
    acc = over_groups(acc);
    float* ro = red + row_blocks * V;
    if (live && lane < kDrCols) *reinterpret_cast<float4*>(ro + rb * V + col) = acc;
    __syncthreads();
    // norm over the head's values and the output gate: all threads walk the columns
    float ss = 0.f;
    for (int c = tid; c < V; c += blockDim.x) {
      float o = 0.f;
      for (int b = 0; b < row_blocks; ++b) o += ro[b * V + c];
      ro[c] = o;                                    // a column belongs to one thread
      ss += o * o;
    }
    ss = warp_sum(ss);
    if (lane == 0) part[warp] = ss;
    __syncthreads();
    ss = 0.f;
    for (int w = 0; w < (int)(blockDim.x >> 5); ++w) ss += part[w];
    const float rstd = rsqrtf(ss / (float)p.vdim_true + p.eps);
    for (int c = tid; c < V; c += blockDim.x) {
      const float z = Num<T>::to_f(reinterpret_cast<const T*>(p.gate)[row * p.ldg + (size_t)h * V + c]);
      reinterpret_cast<T*>(p.out)[row * p.ldo + (size_t)h * V + c] = Num<T>::from_f(ro[c] * rstd * p.norm_w[c] * (z * sigmoid_f(z)));
    }
  }
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int row = rg + r * groups;
    if (live && row < D) *reinterpret_cast<float4*>(S + (size_t)row * V + col) = st[r];
  }
}

template <typename T, int RPT>
static int launch_delta_recurrent(const RfDelta* a, int col_blocks, int row_blocks, cudaStream_t s) {
  const size_t smem = ((size_t)2 * a->dim + a->vdim + 2 * row_blocks * a->vdim + 16) * sizeof(float);
  const dim3 grid(a->heads, a->rows.num_seqs), block(32 * col_blocks * row_blocks);
  if (a->conv_w) RF_CUDA_CHECK(::rf::launch_k(delta_recurrent_kernel<T, RPT, true>, grid, block, smem, s, 1, *a, col_blocks, row_blocks));
  else RF_CUDA_CHECK(::rf::launch_k(delta_recurrent_kernel<T, RPT, false>, grid, block, smem, s, 1, *a, col_blocks, row_blocks));
  ::rf::count_launch();
  return RF_OK;
}

template <typename T>
static int dispatch_delta_recurrent(const RfDelta* a, cudaStream_t s) {
  const int cb = ceil_div(a->vdim, 32), rb = std::max(1, std::min(16 / cb, ceil_div(a->dim, 4 * kDrRows))), rpt = ceil_div(a->dim, rb * kDrRows);
  if (rpt <= 4) return launch_delta_recurrent<T, 4>(a, cb, rb, s);
  if (rpt <= 8) return launch_delta_recurrent<T, 8>(a, cb, rb, s);
  if (rpt <= 16) return launch_delta_recurrent<T, 16>(a, cb, rb, s);
  if (rpt <= 32) return launch_delta_recurrent<T, 32>(a, cb, rb, s);
  return launch_delta_recurrent<T, 64>(a, cb, rb, s);
}

}  // namespace rf

using namespace rf;

static int check_delta(const RfDelta* a) {
  RF_REQUIRE(a && a->x && a->b && a->a && a->gate && a->rate && a->dt_bias && a->norm_w && a->state && a->out && a->rows.pos, "delta: missing buffers");
  RF_REQUIRE(a->kv_heads > 0 && a->heads % a->kv_heads == 0 && a->dim % 8 == 0 && a->vdim % 8 == 0 && a->dim_true > 0 && a->dim_true <= a->dim &&
                 a->dim <= 256 && a->vdim_true > 0 && a->vdim_true <= a->vdim && a->vdim <= 512, "delta: %d / %d heads of %d x %d", a->heads, a->kv_heads, a->dim, a->vdim);
  RF_REQUIRE(a->dtype >= 0 && a->dtype <= 2 && a->rows.num_seqs <= 65535, "delta: dtype %d, %d sequences", a->dtype, a->rows.num_seqs);
  return RF_OK;
}

extern "C" int rf_delta_recurrent(const RfDelta* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  int rc = check_delta(a);
  if (rc) return rc;
  if (a->conv_w) RF_REQUIRE(a->conv_state && a->taps > 0 && !a->rows.q_start, "delta: the convolution runs inside decode steps only");
  if (a->rows.num_seqs == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (a->dtype == kF16) return dispatch_delta_recurrent<__half>(a, s);
  if (a->dtype == kBF16) return dispatch_delta_recurrent<__nv_bfloat16>(a, s);
  return dispatch_delta_recurrent<float>(a, s);
}
