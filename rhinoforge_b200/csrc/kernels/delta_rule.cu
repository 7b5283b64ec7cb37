// Gated delta rule of the mixed-layer decoders, for any head sizes.  Per head, with unit vectors q (times dim^-1/2) and k:
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q,
//   g = exp(-rate * softplus(a + dt_bias)), beta = sigmoid(b),   out = o / rms(o) * norm_w * silu(gate)
//   * rf_delta_recurrent: token by token (decode steps, short portions, everything in 32 bits); in decode steps the short
//     convolution of queries, keys and values runs inside it,
//   * rf_delta_chunked: 64 tokens at a time on the tensor cores (prefill-sized portions).
// The state is fp32, and so is all that enters the recurrence behind the convolutions.
#include "../common/dtype.cuh"
#include "../common/host_util.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"
#include "../rf_api.h"

namespace rf {

__device__ __forceinline__ float softplus_f(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
__device__ __forceinline__ float sigmoid_f(float v) { return 1.f / (1.f + expf(-v)); }

constexpr int kDrCols = 8;            // a warp covers 8 quads of state columns ...
constexpr int kDrRows = 4;            // ... times 4 groups of state rows

// One CTA per (head, sequence).  Warps lie side by side over blocks of 32 state columns (`col_blocks`) and over row blocks; a
// thread holds RPT rows of four columns in registers, rows interleaved over the row groups.
template <typename T, int RPT, bool CONV, int PER_SM>
__global__ void __launch_bounds__(512, PER_SM) delta_recurrent_kernel(const RfDelta p, int col_blocks, int row_blocks) {
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
  const int now = CONV ? pos0 % p.taps : 0;            // ring row of the current token
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
#pragma unroll 3
        for (int k = 1; k < taps; ++k) {
          const int at = now - k + (now < k ? taps : 0);
          if (pos0 >= k) s += Num<T>::to_f(ring[(size_t)at * channels]) * p.conv_w[(size_t)(taps - 1 - k) * channels + c];
        }
        ring[(size_t)now * channels] = x[c];
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
  constexpr int kMany = RPT <= 8 ? 2 : 1;                // decode steps with more heads than SMs: two CTAs overlap their phases
#define RF_DR(CONV, PER_SM) RF_CUDA_CHECK(::rf::launch_k(delta_recurrent_kernel<T, RPT, CONV, PER_SM>, grid, block, smem, s, 1, *a, col_blocks, row_blocks))
  if (!a->conv_w) RF_DR(false, 1);
  else if (a->heads * a->rows.num_seqs > sm_count()) RF_DR(true, kMany);
  else RF_DR(true, 1);
#undef RF_DR
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

// ------------------------------------------------------------------- 64 tokens at a time ----
// With G_i the running sum of the log decays inside a chunk, S0 the incoming state, raw rows q, k (16 bits) and 1 / their norms iq, ik:
//   L_ij = beta_i e^(G_i - G_j) ik_i ik_j (k_i . k_j) for j < i,   P_ij = e^(G_i - G_j) iq_i ik_j (q_i . k_j) for j <= i
//   (I + L) U = beta (v - e^G ik (k S0)),   O = e^G iq (q S0) + P U,   S' = e^G_C S0 + k^T (e^(G_C - G) ik U)
// One CTA owns 32 state columns of one head of one sequence and walks its chunks; the fp32 state stays in registers.  Products run as
// 16-bit mma.sync with fp32 accumulators.  The rows enter them unnormalised, so they are exact; every fp32 operand (S0, P, U) enters as
// a sum of 16-bit terms (three in bf16, two in fp16: 22 bits and more), kept as planes in shared memory.  Every decay that appears is
// e^(G_i - G_j) with j <= i, at most one.  The unit-triangular system is solved in 16-row blocks.  Rows behind a sequence's end are
// zero tokens with beta = 0 and no decay.
constexpr int kDcC = 64, kDcCols = 32, kDcThreads = 256;

template <typename T> struct Terms { static constexpr int n = 3; };
template <> struct Terms<__half> { static constexpr int n = 2; };

template <typename T, int DK> struct DcGeom {
  static constexpr int N = Terms<T>::n, C = kDcC;
  static constexpr int LQ = DK + 8, LV = kDcCols + 8, LF = 40, LL = 68, LP = C + 8, LD = 17;   // row pitches
  static constexpr int raw = 2 * C * LQ + C * LV;                                              // 16-bit values of one chunk: q, k, v
  static constexpr int o_raw = 0;
  static constexpr int o_s = o_raw + 2 * raw * 2;                    // [N][DK][LV] planes of the state
  static constexpr int o_p = o_s + N * DK * LV * 2;                  // [N][C][LP] planes of P
  static constexpr int o_u = o_p + N * C * LP * 2;                   // [N][C][LV] planes of U
  static constexpr int o_w = o_u + N * C * LV * 2;                   // [N][C][LV] planes of e^(G_C - G) ik U
  static constexpr int o_l = o_w + N * C * LV * 2;                   // fp32: L, right-hand sides, U, inverses of the diagonal blocks
  static constexpr int o_v = o_l + C * LL * 4;
  static constexpr int o_f = o_v + C * LF * 4;
  static constexpr int o_d = o_f + C * LF * 4;
  static constexpr int o_g = o_d + 4 * 16 * LD * 4;                  // G, beta, iq, ik, log decays
  static constexpr int total = o_g + 5 * C * 4;
};

__device__ __forceinline__ void dc_cp16(void* dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
// two neighbouring values as N 16-bit terms, one 32-bit word per plane
template <typename T, int N>
__device__ __forceinline__ void store_terms(T* at, int plane, float a, float b) {
#pragma unroll
  for (int i = 0; i < N; ++i) {
    const T ta = Num<T>::from_f(a), tb = Num<T>::from_f(b);
    *reinterpret_cast<uint32_t*>(at + i * plane) = MmaOp<T>::pack(a, b);
    a -= Num<T>::to_f(ta);
    b -= Num<T>::to_f(tb);
  }
}

template <typename T, int DK>
__global__ void __launch_bounds__(kDcThreads, 1) delta_chunked_kernel(const RfDelta p) {
  pdl_prologue();
  using G = DcGeom<T, DK>;
  constexpr int C = kDcC, N = G::N, LQ = G::LQ, LV = G::LV, LF = G::LF, LL = G::LL, LP = G::LP, LD = G::LD;
  constexpr int SR = DK / 16, NCT = DK / 32;           // state row tiles; 8-column tiles of a warp's state
  extern __shared__ __align__(16) uint8_t csm[];
  T* raw = reinterpret_cast<T*>(csm + G::o_raw);
  T* sS = reinterpret_cast<T*>(csm + G::o_s);
  T* sP = reinterpret_cast<T*>(csm + G::o_p);
  T* sU = reinterpret_cast<T*>(csm + G::o_u);
  T* sW = reinterpret_cast<T*>(csm + G::o_w);
  float* sL = reinterpret_cast<float*>(csm + G::o_l);
  float* sV = reinterpret_cast<float*>(csm + G::o_v);
  float* sF = reinterpret_cast<float*>(csm + G::o_f);
  float* sD = reinterpret_cast<float*>(csm + G::o_d);
  float* sG = reinterpret_cast<float*>(csm + G::o_g);
  float* sBeta = sG + C;
  float* sIq = sBeta + C;
  float* sIk = sIq + C;
  float* sLg = sIk + C;

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int seq = blockIdx.z, h = blockIdx.y, j0 = blockIdx.x * kDcCols, hk = h / (p.heads / p.kv_heads);
  const int q0 = p.rows.q_start ? p.rows.q_start[seq] : seq, n = p.rows.q_len ? p.rows.q_len[seq] : 1;
  const int slot = p.rows.slot ? p.rows.slot[seq] : seq;
  const bool fresh = p.rows.pos[q0] == 0;
  const int V = p.vdim, ko = p.kv_heads * DK, qc = hk * DK, kc = ko + hk * DK, vc = 2 * ko + h * V + j0;
  float* S = p.state + ((size_t)slot * p.heads + h) * DK * V + j0;
  const T* x = reinterpret_cast<const T*>(p.x);
  const float rate = p.rate[h], dt_bias = p.dt_bias[h], q_scale = rsqrtf((float)p.dim_true);

  // this warp's state: rows sr .. sr + 15, columns sc .. sc + 8 * NCT - 1, as accumulator fragments
  const int sr = (warp % SR) * 16, sc = (warp / SR) * NCT * 8;
  float st[NCT][4];
#pragma unroll
  for (int a = 0; a < NCT; ++a)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int row = sr + g + half * 8, col = sc + a * 8 + t4 * 2;
      const float2 v = fresh ? make_float2(0.f, 0.f) : *reinterpret_cast<const float2*>(S + (size_t)row * V + col);
      st[a][half * 2] = v.x;
      st[a][half * 2 + 1] = v.y;
    }
  auto publish_state = [&]() {
#pragma unroll
    for (int a = 0; a < NCT; ++a)
#pragma unroll
      for (int half = 0; half < 2; ++half)
        store_terms<T, N>(sS + (sr + g + half * 8) * LV + sc + a * 8 + t4 * 2, DK * LV, st[a][half * 2], st[a][half * 2 + 1]);
  };
  publish_state();

  float nb = 0.f, na = 0.f;                            // gate inputs of row `tid` of the chunk in flight
  auto prefetch = [&](int c0, int buf) {
    if (c0 < n) {
      T* dst = raw + buf * G::raw;
      constexpr int per = DK / 8;                      // 16-byte pieces of a q or k row
#pragma unroll
      for (int k = 0; k < C * 2 * per / kDcThreads; ++k) {
        const int idx = tid + kDcThreads * k, i = idx / (2 * per), part = idx % (2 * per), piece = part % per;
        const bool key = part >= per, valid = c0 + i < n;
        dc_cp16(dst + (key ? C * LQ : 0) + i * LQ + piece * 8, x + (size_t)(q0 + (valid ? c0 + i : 0)) * p.ldx + (key ? kc : qc) + piece * 8, valid);
      }
      const int i = tid >> 2, part = tid & 3;
      const bool valid = c0 + i < n;
      dc_cp16(dst + 2 * C * LQ + i * LV + part * 8, x + (size_t)(q0 + (valid ? c0 + i : 0)) * p.ldx + vc + part * 8, valid);
      if (tid < C && c0 + tid < n) {
        const size_t row = (size_t)(q0 + c0 + tid) * p.ld_ba + h;
        nb = Num<T>::to_f(reinterpret_cast<const T*>(p.b)[row]);
        na = Num<T>::to_f(reinterpret_cast<const T*>(p.a)[row]);
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  prefetch(0, 0);

  for (int c0 = 0, buf = 0; c0 < n; c0 += C, buf ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                   // this chunk's rows, the state planes; the other raw buffer is free
    const T* rQ = raw + buf * G::raw;
    const T* rK = rQ + C * LQ;
    const T* rV = rK + C * LQ;
    if (tid < C) {
      float beta = 0.f, lg = 0.f;
      if (c0 + tid < n) {
        beta = sigmoid_f(nb);
        lg = -rate * softplus_f(na + dt_bias);
      }
      sBeta[tid] = beta;
      sLg[tid] = lg;
    }
    prefetch(c0 + C, buf ^ 1);
    // 1 / norms: half a warp per row of q or k
#pragma unroll
    for (int rr = 0; rr < C * 2 / 16; ++rr) {
      const int item = warp * (C * 2 / 8) + rr * 2 + (lane >> 4), i = item >> 1, l16 = lane & 15;
      const bool key = item & 1;
      float ss = 0.f;
      if (l16 * 8 < DK) {
        float f[8];
        load8((key ? rK : rQ) + i * LQ + l16 * 8, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
      }
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (l16 == 0) (key ? sIk : sIq)[i] = rsqrtf(ss + 1e-6f) * (key ? 1.f : q_scale);
    }
    __syncthreads();
    if (warp == 0) {                                   // inclusive running sum of the log decays
      const float x0 = sLg[2 * lane], x1 = sLg[2 * lane + 1];
      float run = x0 + x1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += y;
      }
      sG[2 * lane] = run - x1;
      sG[2 * lane + 1] = run;
    }
    // ---- raw products: k k^T and q k^T on and below the diagonal, k S0 and q S0
    const int gr = warp >> 1, cnt = gr + 1, nt0 = (warp & 1) * cnt;     // row tile gr has 2 (gr + 1) column tiles
    float accL[4][4] = {}, accP[4][4] = {};
#pragma unroll
    for (int ks = 0; ks < DK / 32; ++ks) {
      uint32_t aK[2][4], aQ[2][4];
#pragma unroll
      for (int hk2 = 0; hk2 < 2; ++hk2) {
        const int at = (gr * 16 + (lane & 15)) * LQ + ks * 32 + hk2 * 16 + (lane >> 4) * 8;
        ldsm_x4(smem_u32(rK + at), aK[hk2][0], aK[hk2][1], aK[hk2][2], aK[hk2][3]);
        ldsm_x4(smem_u32(rQ + at), aQ[hk2][0], aQ[hk2][1], aQ[hk2][2], aQ[hk2][3]);
      }
#pragma unroll
      for (int ti = 0; ti < 4; ++ti)
        if (ti < cnt) {
          uint32_t b[4];                               // eight keys, two k16 steps
          ldsm_x4(smem_u32(rK + ((nt0 + ti) * 8 + (lane & 7)) * LQ + ks * 32 + (lane >> 3) * 8), b[0], b[1], b[2], b[3]);
#pragma unroll
          for (int hk2 = 0; hk2 < 2; ++hk2) {
            MmaOp<T>::mma(accL[ti], aK[hk2], b[hk2 * 2], b[hk2 * 2 + 1]);
            MmaOp<T>::mma(accP[ti], aQ[hk2], b[hk2 * 2], b[hk2 * 2 + 1]);
          }
        }
    }
    const int rt = warp & 3, nh = warp >> 2;           // row tile and column half of k S0, q S0 and O
    float accR[2][4] = {}, accO[2][4] = {};
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks) {
      uint32_t aK[4], aQ[4];
      const int at = (rt * 16 + (lane & 15)) * LQ + ks * 16 + (lane >> 4) * 8;
      ldsm_x4(smem_u32(rK + at), aK[0], aK[1], aK[2], aK[3]);
      ldsm_x4(smem_u32(rQ + at), aQ[0], aQ[1], aQ[2], aQ[3]);
#pragma unroll
      for (int i = N - 1; i >= 0; --i) {               // the small terms first
        uint32_t b[4];
        ldsm_x4_t(smem_u32(sS + i * DK * LV + (ks * 16 + (lane & 15)) * LV + nh * 16 + (lane >> 4) * 8), b[0], b[1], b[2], b[3]);
#pragma unroll
        for (int a = 0; a < 2; ++a) {
          MmaOp<T>::mma(accR[a], aK, b[a * 2], b[a * 2 + 1]);
          MmaOp<T>::mma(accO[a], aQ, b[a * 2], b[a * 2 + 1]);
        }
      }
    }
    __syncthreads();                                   // G is there; the state planes are read
    // ---- L, P, right-hand sides
#pragma unroll
    for (int ti = 0; ti < 4; ++ti)
      if (ti < cnt) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = gr * 16 + g + half * 8, j = (nt0 + ti) * 8 + t4 * 2;
          const float gi = sG[i], bi = sBeta[i] * sIk[i], qi = sIq[i];
          const float2 gj = *reinterpret_cast<const float2*>(sG + j), kj = *reinterpret_cast<const float2*>(sIk + j);
          const float d0 = j <= i ? __expf(gi - gj.x) * kj.x : 0.f, d1 = j + 1 <= i ? __expf(gi - gj.y) * kj.y : 0.f;
          *reinterpret_cast<float2*>(sL + i * LL + j) = make_float2(j < i ? bi * d0 * accL[ti][half * 2] : 0.f, j + 1 < i ? bi * d1 * accL[ti][half * 2 + 1] : 0.f);
          store_terms<T, N>(sP + i * LP + j, C * LP, qi * d0 * accP[ti][half * 2], qi * d1 * accP[ti][half * 2 + 1]);
        }
      }
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = rt * 16 + g + half * 8, j = (nh * 2 + a) * 8 + t4 * 2;
        const float eg = __expf(sG[i]), kr = eg * sIk[i], qr = eg * sIq[i], beta = sBeta[i];
        const float2 v = Num<T>::to_f2(*reinterpret_cast<const typename Num<T>::T2*>(rV + i * LV + j));
        *reinterpret_cast<float2*>(sV + i * LF + j) = make_float2(beta * (v.x - kr * accR[a][half * 2]), beta * (v.y - kr * accR[a][half * 2 + 1]));
        accO[a][half * 2] *= qr;
        accO[a][half * 2 + 1] *= qr;
      }
    __syncthreads();
    // ---- inverses of the four 16 x 16 diagonal blocks of I + L (warps 0..3, one column per lane)
    if (warp < 4 && lane < 16) {
      float y[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float acc = i == lane ? 1.f : 0.f;
#pragma unroll
        for (int j = 0; j < i; ++j) acc -= sL[(warp * 16 + i) * LL + warp * 16 + j] * y[j];
        y[i] = acc;
        sD[(warp * 16 + i) * LD + lane] = acc;
      }
    }
    // ---- U by block forward substitution; finished rows leave as planes, plain and weighted for the state update
    {
      const int r = tid >> 4, cc = (tid & 15) * 2;
      const float gl = sG[C - 1];
      for (int b = 0; b < 4; ++b) {
        const int i = b * 16 + r;
        float2 a = *reinterpret_cast<const float2*>(sV + i * LF + cc);
#pragma unroll 8
        for (int j = 0; j < b * 16; ++j) {
          const float l = sL[i * LL + j];
          const float2 u = *reinterpret_cast<const float2*>(sF + j * LF + cc);
          a.x -= l * u.x;
          a.y -= l * u.y;
        }
        *reinterpret_cast<float2*>(sV + i * LF + cc) = a;          // a row of block b is touched by its owners only until the barrier
        __syncthreads();
        float2 u = make_float2(0.f, 0.f);
#pragma unroll
        for (int r2 = 0; r2 < 16; ++r2)
          if (r2 <= r) {
            const float d = sD[i * LD + r2];
            const float2 v = *reinterpret_cast<const float2*>(sV + (b * 16 + r2) * LF + cc);
            u.x += d * v.x;
            u.y += d * v.y;
          }
        *reinterpret_cast<float2*>(sF + i * LF + cc) = u;
        store_terms<T, N>(sU + i * LV + cc, C * LV, u.x, u.y);
        const float w = __expf(gl - sG[i]) * sIk[i];
        store_terms<T, N>(sW + i * LV + cc, C * LV, w * u.x, w * u.y);
        __syncthreads();
      }
    }
    // ---- O += P U
    for (int ks = 0; ks <= rt; ++ks) {
      uint32_t a[N][4];
#pragma unroll
      for (int i = 0; i < N; ++i)
        ldsm_x4(smem_u32(sP + i * C * LP + (rt * 16 + (lane & 15)) * LP + ks * 16 + (lane >> 4) * 8), a[i][0], a[i][1], a[i][2], a[i][3]);
#pragma unroll
      for (int i = N - 1; i >= 0; --i) {
        uint32_t b[4];
        ldsm_x4_t(smem_u32(sU + i * C * LV + (ks * 16 + (lane & 15)) * LV + nh * 16 + (lane >> 4) * 8), b[0], b[1], b[2], b[3]);
#pragma unroll
        for (int k = N - 1 - i; k >= 0; --k)           // products of terms whose places add up to less than N
#pragma unroll
          for (int c = 0; c < 2; ++c) MmaOp<T>::mma(accO[c], a[k], b[c * 2], b[c * 2 + 1]);
      }
    }
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = rt * 16 + g + half * 8, j = (nh * 2 + a) * 8 + t4 * 2;
        if (c0 + i < n)
          *reinterpret_cast<uint32_t*>(reinterpret_cast<T*>(p.out) + (size_t)(q0 + c0 + i) * p.ldo + (size_t)h * V + j0 + j) = MmaOp<T>::pack(accO[a][half * 2], accO[a][half * 2 + 1]);
      }
    // ---- S' = e^G_C S0 + k^T W
    {
      const float egl = __expf(sG[C - 1]);
#pragma unroll
      for (int a = 0; a < NCT; ++a)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[a][e] *= egl;
#pragma unroll
      for (int ks = 0; ks < C / 16; ++ks) {
        uint32_t aT[4];
        ldsm_x4_t(smem_u32(rK + (ks * 16 + (lane >> 4) * 8 + (lane & 7)) * LQ + sr + ((lane >> 3) & 1) * 8), aT[0], aT[1], aT[2], aT[3]);
#pragma unroll
        for (int i = N - 1; i >= 0; --i)
#pragma unroll
          for (int c = 0; c < NCT; c += 2) {
            uint32_t b[4];
            ldsm_x4_t(smem_u32(sW + i * C * LV + (ks * 16 + (lane & 15)) * LV + sc + c * 8 + (lane >> 4) * 8), b[0], b[1], b[2], b[3]);
            MmaOp<T>::mma(st[c], aT, b[0], b[1]);
            MmaOp<T>::mma(st[c + 1], aT, b[2], b[3]);
          }
      }
      publish_state();
    }
  }
#pragma unroll
  for (int a = 0; a < NCT; ++a)
#pragma unroll
    for (int half = 0; half < 2; ++half)
      *reinterpret_cast<float2*>(S + (size_t)(sr + g + half * 8) * V + sc + a * 8 + t4 * 2) = make_float2(st[a][half * 2], st[a][half * 2 + 1]);
}

// What the chunked form leaves out: out <- out / rms(out) * norm_w * silu(gate) per head, in place; a warp per (row, head).
template <typename T>
__global__ void __launch_bounds__(256) delta_out_kernel(const RfDelta p, int row0, int rows) {
  pdl_prologue();
  const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, V = p.vdim;
  if (item >= rows * p.heads) return;
  const size_t row = (size_t)(row0 + item / p.heads);
  const int h = item % p.heads;
  T* o = reinterpret_cast<T*>(p.out) + row * p.ldo + (size_t)h * V;
  const T* z = reinterpret_cast<const T*>(p.gate) + row * p.ldg + (size_t)h * V;
  float v[2][8], ss = 0.f;                             // up to 512 values
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int c = (lane + 32 * k) * 8;
    if (c < V) load8(o + c, v[k]);
    else {
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] = 0.f;
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += v[k][j] * v[k][j];
  }
  const float rstd = rsqrtf(warp_sum(ss) / (float)p.vdim_true + p.eps);
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int c = (lane + 32 * k) * 8;
    if (c >= V) continue;
    float zf[8], w[8];
    load8(z + c, zf);
    load8(p.norm_w + c, w);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[k][j] *= rstd * w[j] * silu_f(zf[j]);
    store8(o + c, v[k]);
  }
}

template <typename T, int DK>
static int launch_delta_chunked(const RfDelta* a, int row0, int rows, cudaStream_t s) {
  constexpr int smem = DcGeom<T, DK>::total;
  RF_ALLOW_SMEM_PER_DEVICE((delta_chunked_kernel<T, DK>), smem);
  RF_CUDA_CHECK(::rf::launch_k(delta_chunked_kernel<T, DK>, dim3(a->vdim / kDcCols, a->heads, a->rows.num_seqs), dim3(kDcThreads), smem, s, 1, *a));
  ::rf::count_launch();
  RF_CUDA_CHECK(::rf::launch_k(delta_out_kernel<T>, dim3((unsigned)(((int64_t)rows * a->heads + 7) / 8)), dim3(256), 0, s, 1, *a, row0, rows));
  ::rf::count_launch();
  return RF_OK;
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

extern "C" int rf_delta_chunked_supported(int dim, int vdim, int dtype) {
  return dtype != kF32 && (dim == 64 || dim == 128) && vdim > 0 && vdim % kDcCols == 0 && vdim <= 512;
}

extern "C" int rf_delta_chunked(const RfDelta* a, int row0, int rows, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  int rc = check_delta(a);
  if (rc) return rc;
  RF_REQUIRE(rf_delta_chunked_supported(a->dim, a->vdim, a->dtype) && !a->conv_w, "delta: the chunked form takes heads of 64 / 128 by multiples of 32 in 16 bits");
  RF_REQUIRE(a->ldx % 8 == 0 && a->ldo % 8 == 0 && a->ldg % 8 == 0 && row0 >= 0 && rows >= 0, "delta: pitches");
  if (a->rows.num_seqs == 0 || rows == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (a->dtype == kF16) return a->dim == 64 ? launch_delta_chunked<__half, 64>(a, row0, rows, s) : launch_delta_chunked<__half, 128>(a, row0, rows, s);
  return a->dim == 64 ? launch_delta_chunked<__nv_bfloat16, 64>(a, row0, rows, s) : launch_delta_chunked<__nv_bfloat16, 128>(a, row0, rows, s);
}
