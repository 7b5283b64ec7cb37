// Latent attention: one small normalised row per token is cached, and every head's keys and values are linear maps of it.
//   * rf_latent_insert / rf_latent_gather: the paged latent cache (16-token pages),
//   * rf_head_linear: the per-head maps into and out of the latent space,
//   * rf_latent_attn: attention with the maps folded into the queries and the output (decode steps, short portions, and
//     everything in fp32); prefill-sized portions expand keys and values and run on the tcgen05 attention instead.
#include "../common/dtype.cuh"
#include "../common/host_util.h"
#include "../common/mma.cuh"
#include "../common/ptx.cuh"
#include "../rf_api.h"

namespace rf {

__device__ __forceinline__ int row_seq(const RfRows& r, int row) { return r.seq_of_row ? r.seq_of_row[row] : row; }
__device__ __forceinline__ int seq_slot(const RfRows& r, int seq) { return r.slot ? r.slot[seq] : seq; }

// --------------------------------------------------------------- cache rows ----
// 1 / rms of n values of a row, eight per lane and step (all lanes of the warp); dim: what the mean runs over.
template <typename T>
__device__ __forceinline__ float row_rstd(const T* x, int n, int dim, float eps, int lane) {
  float s = 0.f;
  for (int i = lane * 8; i < n; i += 256) {
    float f[8];
    load8(x + i, f);
#pragma unroll
    for (int j = 0; j < 8; ++j) s += f[j] * f[j];
  }
  return rsqrtf(warp_sum(s) / (float)dim + eps);
}
template <typename T>
__device__ __forceinline__ void scale_row(const T* x, T* y, const float* w, int n, float rstd, int lane) {
  for (int i = lane * 8; i < n; i += 256) {
    float f[8], g[8];
    load8(x + i, f);
    load8(w + i, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) f[j] *= rstd * g[j];
    store8(y + i, f);
  }
}
// Eight neighbouring values, from dimension c on, of `dims` rotated ones at one position.
template <typename T>
__device__ __forceinline__ void rotate8(const T* x, T* y, const float* cos, const float* sin, int pos, int c, int dims) {
  float f[8];
  load8(x + c, f);
  const size_t at = (size_t)pos * (dims >> 1) + (c >> 1);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if (c + 2 * i < dims) {
      const float co = cos[at + i], si = sin[at + i], u = f[2 * i], v = f[2 * i + 1];
      f[2 * i] = u * co - v * si;
      f[2 * i + 1] = v * co + u * si;
    } else {
      f[2 * i] = f[2 * i + 1] = 0.f;
    }
  }
  store8(y + c, f);
}
template <typename T>
__device__ __forceinline__ void head_rotate_item(const RfHeadRotate& p, int64_t i) {
  const int per = p.dims_pad / 8, c = (int)(i % per) * 8;
  const int64_t rh = i / per;
  if (rh >= (int64_t)p.rows * p.heads) return;
  const int row = (int)(rh / p.heads), h = (int)(rh % p.heads);
  rotate8(reinterpret_cast<const T*>(p.x) + (size_t)row * p.ldx + (size_t)h * p.xs, reinterpret_cast<T*>(p.y) + (size_t)row * p.ldy + (size_t)h * p.ys,
          p.cos, p.sin, p.pos[row], c, p.dims);
}

// One warp normalises one row's latent and stores it at its position, together with the rotated part.
template <typename T>
__device__ __forceinline__ void latent_insert_row(const RfLatentInsert& p, int row, int lane) {
  const T* xr = reinterpret_cast<const T*>(p.x) + (size_t)row * p.ldx;
  const int pos = p.rows.pos[row];
  const int page = p.rows.page_table[(size_t)seq_slot(p.rows, row_seq(p.rows, row)) * p.rows.pt_stride + (pos >> 4)];
  T* dst = reinterpret_cast<T*>(p.pool) + ((size_t)page * 16 + (pos & 15)) * (p.rank + p.rot_pad);
  for (int c = lane * 8; c < p.rot_pad; c += 256) rotate8(xr + p.rank, dst + p.rank, p.cos, p.sin, pos, c, p.rot);
  scale_row(xr, dst, p.norm_w, p.rank, row_rstd(xr, p.rank, p.rank_true, p.eps, lane), lane);
}

// A warp per row and part: the cached row (with x), the query latent (with q).
template <typename T>
__global__ void latent_insert_kernel(const RfLatentInsert p) {
  pdl_prologue();
  const int item = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31, parts = (p.x ? 1 : 0) + (p.q ? 1 : 0);
  const int row = item / parts;
  if (row >= p.n_rows) return;
  if (p.x && item % parts == 0) {
    latent_insert_row<T>(p, row, lane);
  } else {
    T* q = reinterpret_cast<T*>(p.q) + (size_t)row * p.ldq;
    scale_row(q, q, p.q_norm, p.q_rank, row_rstd(q, p.q_rank, p.q_rank_true, p.eps, lane), lane);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) head_rotate_kernel(const RfHeadRotate p) {
  pdl_prologue();
  head_rotate_item<T>(p, (int64_t)blockIdx.x * blockDim.x + threadIdx.x);
}

template <typename T>
__global__ void latent_gather_kernel(const T* __restrict__ pool, T* __restrict__ out, const RfRows rows,
                                     const int32_t* __restrict__ kv_start, const int32_t* __restrict__ kv_len, int rank) {
  pdl_prologue();
  const int seq = blockIdx.y, n = kv_len[seq], base = kv_start[seq];
  const int first = rows.pos[rows.q_start[seq]] + rows.q_len[seq] - n;       // position of the first copied row
  const int32_t* pt = rows.page_table + (size_t)seq_slot(rows, seq) * rows.pt_stride;
  const int per = rank / 8;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < (int64_t)n * per; i += (int64_t)gridDim.x * blockDim.x) {
    const int j = (int)(i / per), c = (int)(i % per) * 8, pos = first + j;
    *reinterpret_cast<Vec8<T>*>(out + (size_t)(base + j) * rank + c) =
        *reinterpret_cast<const Vec8<T>*>(pool + ((size_t)pt[pos >> 4] * 16 + (pos & 15)) * rank + c);
  }
}

// ----------------------------------------------------------- per-head linear ----
constexpr int kHlRows = 16, kHlN = 64, kHlK = 32;

template <typename T>
__global__ void __launch_bounds__(128) head_linear_kernel(const RfHeadLinear p) {
  pdl_prologue();
  __shared__ float sx[kHlRows][kHlK + 1], sw[kHlN][kHlK + 1];
  const int h = blockIdx.y, n0 = blockIdx.x * kHlN, r0 = blockIdx.z * kHlRows, tid = threadIdx.x;
  const T* x = reinterpret_cast<const T*>(p.x) + (size_t)h * p.xs;
  const T* w = reinterpret_cast<const T*>(p.w) + (size_t)h * p.n * p.k;
  const int n = tid % kHlN, rg = tid / kHlN;      // rows rg, rg + 2, ...
  float acc[kHlRows / 2] = {};
  for (int k0 = 0; k0 < p.k; k0 += kHlK) {
    for (int i = tid; i < kHlRows * kHlK; i += 128) {
      const int r = i / kHlK, k = i % kHlK;
      sx[r][k] = (r0 + r < p.rows && k0 + k < p.k) ? Num<T>::to_f(x[(size_t)(r0 + r) * p.ldx + k0 + k]) : 0.f;
    }
    for (int i = tid; i < kHlN * kHlK; i += 128) {
      const int r = i / kHlK, k = i % kHlK;
      sw[r][k] = (n0 + r < p.n && k0 + k < p.k) ? Num<T>::to_f(w[(size_t)(n0 + r) * p.k + k0 + k]) : 0.f;
    }
    __syncthreads();
    for (int k = 0; k < kHlK; ++k) {
      const float b = sw[n][k];
#pragma unroll
      for (int i = 0; i < kHlRows / 2; ++i) acc[i] = fmaf(sx[rg + 2 * i][k], b, acc[i]);
    }
    __syncthreads();
  }
  if (n0 + n < p.n) {
#pragma unroll
    for (int i = 0; i < kHlRows / 2; ++i) {
      const int r = r0 + rg + 2 * i;
      if (r < p.rows) reinterpret_cast<T*>(p.y)[(size_t)r * p.ldy + (size_t)h * p.ys + n0 + n] = Num<T>::from_f(acc[i]);
    }
  }
}

__device__ __forceinline__ void la_cp16(uint32_t dst, const void* src, bool valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}
__device__ __forceinline__ void la_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void la_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// 16-bit form on the tensor cores: 64 rows x (NT * 32) outputs of one head per CTA, warps side by side along the outputs, a
// ring of 64-wide k blocks.  The weights of the first blocks are fetched ahead of the dependency wait.
constexpr int kHmRows = 64, kHmK = 64, kHmLd = kHmK + 8, kHmStages = 4;

template <typename T, int NT>
__global__ void __launch_bounds__(128) head_linear_mma_kernel(const RfHeadLinear p, const RfLatentInsert ins, const RfHeadRotate turn, int row_tiles) {
  pdl_launch_dependents();
  if ((int)blockIdx.z >= row_tiles) {    // the grid's last planes insert latent rows, one per warp, then rotate, eight values per thread
    pdl_wait();
    const int block = (((int)blockIdx.z - row_tiles) * gridDim.y + blockIdx.y) * gridDim.x + blockIdx.x, ins_blocks = (ins.n_rows + 3) / 4;
    const int row = block * 4 + (threadIdx.x >> 5);
    if (row < ins.n_rows) latent_insert_row<T>(ins, row, threadIdx.x & 31);
    if (block >= ins_blocks && turn.rows > 0) head_rotate_item<T>(turn, (int64_t)(block - ins_blocks) * 128 + threadIdx.x);
    return;
  }
  constexpr int BN = NT * 32;
  extern __shared__ __align__(16) uint8_t hsm[];
  constexpr uint32_t kXBytes = kHmRows * kHmLd * 2, kStage = kXBytes + BN * kHmLd * 2;
  const uint32_t ring = smem_u32(hsm);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, n0 = blockIdx.x * BN, r0 = blockIdx.z * kHmRows;
  const T* x = reinterpret_cast<const T*>(p.x) + (size_t)h * p.xs;
  const T* w = reinterpret_cast<const T*>(p.w) + (size_t)h * p.n * p.k;
  const int nblk = (p.k + kHmK - 1) / kHmK, mt = min(4, (p.rows - r0 + 15) / 16);
  auto load_w = [&](int b) {
    const uint32_t dst = ring + (uint32_t)(b % kHmStages) * kStage + kXBytes;
    for (int i = tid; i < BN * 8; i += 128) {
      const int r = i >> 3, c = (i & 7) * 8, k = b * kHmK + c;
      const bool ok = n0 + r < p.n && k < p.k;
      la_cp16(dst + (uint32_t)(r * kHmLd + c) * 2, ok ? w + (size_t)(n0 + r) * p.k + k : w, ok);
    }
  };
  auto load_x = [&](int b) {
    const uint32_t dst = ring + (uint32_t)(b % kHmStages) * kStage;
    for (int i = tid; i < mt * 16 * 8; i += 128) {
      const int r = i >> 3, c = (i & 7) * 8, k = b * kHmK + c;
      const bool ok = r0 + r < p.rows && k < p.k;
      la_cp16(dst + (uint32_t)(r * kHmLd + c) * 2, ok ? x + (size_t)(r0 + r) * p.ldx + k : x, ok);
    }
  };
  for (int b = 0; b < kHmStages - 1; ++b)
    if (b < nblk) load_w(b);
  pdl_wait();
  for (int b = 0; b < kHmStages - 1; ++b) {
    if (b < nblk) load_x(b);
    la_commit();
  }
  float acc[4][NT][4] = {};
  for (int b = 0; b < nblk; ++b) {
    la_wait<kHmStages - 2>();
    __syncthreads();
    if (b + kHmStages - 1 < nblk) {
      load_w(b + kHmStages - 1);
      load_x(b + kHmStages - 1);
    }
    la_commit();
    const uint32_t sx = ring + (uint32_t)(b % kHmStages) * kStage, sw = sx + kXBytes;
#pragma unroll
    for (int ks = 0; ks < kHmK / 32; ++ks) {
      uint32_t bf[NT][4];
#pragma unroll
      for (int t = 0; t < NT; ++t)       // eight outputs, two k16 steps
        ldsm_x4(sw + (uint32_t)((warp * NT * 8 + t * 8 + (lane & 7)) * kHmLd + ks * 32 + (lane >> 3) * 8) * 2, bf[t][0], bf[t][1], bf[t][2], bf[t][3]);
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        if (m < mt) {
#pragma unroll
          for (int hk = 0; hk < 2; ++hk) {
            uint32_t a[4];
            ldsm_x4(sx + (uint32_t)((m * 16 + (lane & 15)) * kHmLd + ks * 32 + hk * 16 + (lane >> 4) * 8) * 2, a[0], a[1], a[2], a[3]);
#pragma unroll
            for (int t = 0; t < NT; ++t) MmaOp<T>::mma(acc[m][t], a, bf[t][hk * 2], bf[t][hk * 2 + 1]);
          }
        }
      }
    }
  }
  T* y = reinterpret_cast<T*>(p.y) + (size_t)h * p.ys;
  const int g = lane >> 2, q = lane & 3;
#pragma unroll
  for (int m = 0; m < 4; ++m)
#pragma unroll
    for (int t = 0; t < NT; ++t)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int r = r0 + m * 16 + g + half * 8, n = n0 + warp * NT * 8 + t * 8 + q * 2;
        if (m < mt && r < p.rows && n < p.n)
          *reinterpret_cast<uint32_t*>(y + (size_t)r * p.ldy + n) = MmaOp<T>::pack(acc[m][t][half * 2], acc[m][t][half * 2 + 1]);
      }
}

template <typename T>
static int launch_head_linear_mma(const RfHeadLinear* a, const RfLatentInsert* c, const RfHeadRotate* t, cudaStream_t s) {
  const int rt = ceil_div(a->rows, kHmRows);
  const RfLatentInsert ins = c ? *c : RfLatentInsert{};
  const RfHeadRotate turn = t ? *t : RfHeadRotate{};
  const int extra = ceil_div(ins.n_rows, 4) + (int)(((int64_t)turn.rows * turn.heads * (turn.dims_pad / 8) + 127) / 128);
#define RF_HM(NT)                                                                                                            \
  do {                                                                                                                       \
    constexpr size_t smem = (size_t)kHmStages * (kHmRows + NT * 32) * kHmLd * 2;                                              \
    const int gx = ceil_div(a->n, NT * 32);                                                                                  \
    const dim3 grid(gx, a->heads, rt + ceil_div(extra, gx * a->heads));                                                        \
    RF_ALLOW_SMEM_PER_DEVICE((head_linear_mma_kernel<T, NT>), smem);                                                         \
    RF_CUDA_CHECK(::rf::launch_k(head_linear_mma_kernel<T, NT>, grid, dim3(128), smem, s, 1, *a, ins, turn, rt)); \
  } while (0)
  if ((long)ceil_div(a->n, 64) * a->heads * rt < sm_count()) RF_HM(1);
  else RF_HM(2);
#undef RF_HM
  ::rf::count_launch();
  return RF_OK;
}

// --------------------------------------------- attention in the latent space ----
// One CTA per (row, head), four warps striding over the keys with an online softmax each, merged at the end.  A lane keeps
// elements lane, lane + 32, .. of the query, the key row and the accumulator.  All products in fp32.
template <typename T, int RPL>
__global__ void __launch_bounds__(128) latent_attn_kernel(const RfLatentAttn p) {
  pdl_prologue();
  extern __shared__ float sm[];           // [4][rank] accumulators, then max and sum of the four warps
  const int row = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, rank = p.rank;
  const T* q = reinterpret_cast<const T*>(p.q) + ((size_t)row * p.heads + h) * rank;
  const T* pool = reinterpret_cast<const T*>(p.pool);
  const int pos = p.rows.pos[row];
  const int32_t* pt = p.rows.page_table + (size_t)seq_slot(p.rows, row_seq(p.rows, row)) * p.rows.pt_stride;
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  float qv[RPL], acc[RPL], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int i = 0; i < RPL; ++i) {
    qv[i] = lane + 32 * i < rank ? Num<T>::to_f(q[lane + 32 * i]) * p.scale : 0.f;
    acc[i] = 0.f;
  }
  for (int j = lo + warp; j <= pos; j += 4) {
    const T* c = pool + ((size_t)pt[j >> 4] * 16 + (j & 15)) * rank;
    float cv[RPL], s = 0.f;
#pragma unroll
    for (int i = 0; i < RPL; ++i) {
      cv[i] = lane + 32 * i < rank ? Num<T>::to_f(c[lane + 32 * i]) : 0.f;
      s = fmaf(qv[i], cv[i], s);
    }
    s = warp_sum(s);
    const float mn = fmaxf(m, s), corr = expf(m - mn), w = expf(s - mn);
    m = mn;
    l = l * corr + w;
#pragma unroll
    for (int i = 0; i < RPL; ++i) acc[i] = acc[i] * corr + w * cv[i];
  }
  const int vrank = p.vrank > 0 ? p.vrank : rank;
  float* sml = sm + 4 * rank;
#pragma unroll
  for (int i = 0; i < RPL; ++i)
    if (lane + 32 * i < rank) sm[warp * rank + lane + 32 * i] = acc[i];
  if (lane == 0) { sml[warp] = m; sml[4 + warp] = l; }
  __syncthreads();
  float mm = -INFINITY;
  for (int w = 0; w < 4; ++w) mm = fmaxf(mm, sml[w]);
  float f[4], tot = 0.f;
  for (int w = 0; w < 4; ++w) {
    f[w] = sml[w] == -INFINITY ? 0.f : expf(sml[w] - mm);
    tot += f[w] * sml[4 + w];
  }
  T* o = reinterpret_cast<T*>(p.o) + ((size_t)row * p.heads + h) * vrank;
  for (int i = threadIdx.x; i < vrank; i += 128) {
    float v = 0.f;
    for (int w = 0; w < 4; ++w) v += f[w] * sm[w * rank + i];
    o[i] = Num<T>::from_f(v / tot);
  }
}

// 16-bit form on the tensor cores.  One CTA (W warps) takes MT * 16 heads of one row and a range of its keys, 64 keys per
// step.  Scores: a warp holds its share (2 / W) of the latent columns of all queries in registers for the whole launch and scores
// half of the keys; the shares are summed by the softmax, which runs row-wise over shared memory.  Output: every warp
// accumulates NT * 64 / W latent columns.  The cached rows are keys and values both, so a key block is read once.  The
// probabilities enter the second product as a 16-bit pair (value + remainder), so they keep about 16 mantissa bits.
constexpr int kLaKeys = 64;

struct LatentSplit {
  float* o;      // [rows, heads, splits, rank] partial outputs, unnormalised
  float* ml;     // [rows, heads, splits, 2] running maximum (log2 domain) and sum
  int splits;
};

template <int NT, int MT> struct LaGeom {
  static constexpr int W = NT >= 2 ? 16 : 8, KG = W / 2;            // warps; shares of the latent columns
  static constexpr int steps = NT * 4, KS = (steps + KG - 1) / KG;  // k16 steps of all columns, of the largest share
  static constexpr int out = NT * 64 > 512 ? 512 : NT * 64, NTW = (out / 8 + W - 1) / W;   // value columns at most, output tiles per warp
  static constexpr int M = 16 * MT, LD = NT * 64 + 8, LDS = kLaKeys + 4, LDP = kLaKeys + 8;
  static constexpr int c = 0;                                       // [2][64][LD] key blocks (the queries pass through here first)
  static constexpr int s = c + 2 * kLaKeys * LD * 2;                // [KG][M][LDS] partial scores
  static constexpr int p = s + KG * M * LDS * 4;                     // [2][M][LDP] probabilities: value, remainder
  static constexpr int m = p + 2 * M * LDP * 2;                     // running maximum, sum, rescale of this step
  static constexpr int total = m + 3 * M * 4;
};

template <typename T, int NT, int MT>
__global__ void __launch_bounds__(32 * LaGeom<NT, MT>::W, 1) latent_attn_mma_kernel(const RfLatentAttn p, const LatentSplit sp) {
  pdl_prologue();
  using L = LaGeom<NT, MT>;
  constexpr int M = L::M, ld = L::LD, LDS = L::LDS, LDP = L::LDP, RP = NT * 64;
  constexpr int W = L::W, KG = L::KG, kThreads = 32 * W, KS = L::KS, NTW = L::NTW;
  extern __shared__ __align__(16) uint8_t lsm[];
  const int rank = p.rank, vrank = p.vrank > 0 ? p.vrank : rank;
  T* sC = reinterpret_cast<T*>(lsm + L::c);
  float* sS = reinterpret_cast<float*>(lsm + L::s);
  T* sP = reinterpret_cast<T*>(lsm + L::p);
  float* sM = reinterpret_cast<float*>(lsm + L::m);
  float* sL = sM + M;
  float* sA = sL + M;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, q4 = lane & 3;
  const int split = blockIdx.x, h0 = blockIdx.y * M, row = blockIdx.z;
  const int pos = p.rows.pos[row];
  const int32_t* pt = p.rows.page_table + (size_t)seq_slot(p.rows, row_seq(p.rows, row)) * p.rows.pt_stride;
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int blocks = (pos - lo) / kLaKeys + 1, per = (blocks + sp.splits - 1) / sp.splits;
  const int b0 = split * per, b1 = min(blocks, b0 + per);
  const T* pool = reinterpret_cast<const T*>(p.pool);
  const T* q = reinterpret_cast<const T*>(p.q) + ((size_t)row * p.heads + h0) * rank;
  const int heads_here = min(M, p.heads - h0);
  const int kq = warp >> 1, key0 = (warp & 1) * 32;        // this warp's column share and key half for the scores
  const int k0 = kq * L::steps / KG, kn = (kq + 1) * L::steps / KG - k0;
  constexpr bool kEven = L::steps % KG == 0;

  for (int i = tid; i < M * (RP / 8); i += kThreads) {
    const int r = i / (RP / 8), c = (i % (RP / 8)) * 8;
    const bool ok = r < heads_here && c < rank;
    la_cp16(smem_u32(sC + r * ld + c), ok ? q + (size_t)r * rank + c : q, ok);
  }
  la_commit();
  if (tid < M) { sM[tid] = -INFINITY; sL[tid] = 0.f; }
  la_wait<0>();
  __syncthreads();
  uint32_t qf[MT][KS][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int k = 0; k < KS; ++k)
      if (kEven || k < kn) ldsm_x4(smem_u32(sC + (m * 16 + (lane & 15)) * ld + (k0 + k) * 16 + (lane >> 4) * 8), qf[m][k][0], qf[m][k][1], qf[m][k][2], qf[m][k][3]);
  __syncthreads();
  auto load_keys = [&](int b) {
    constexpr int TPR = kThreads / kLaKeys;                // threads per key row
    const int r = tid / TPR, j = lo + b * kLaKeys + r;
    const bool in = j <= pos;
    const T* src = in ? pool + ((size_t)pt[j >> 4] * 16 + (j & 15)) * rank : pool;
    T* dst = sC + ((b & 1) * kLaKeys + r) * ld;
#pragma unroll
    for (int i = 0; i < RP / (8 * TPR); ++i) {
      const int c = (tid % TPR + i * TPR) * 8;
      la_cp16(smem_u32(dst + c), in && c < rank ? src + c : pool, in && c < rank);
    }
  };
  if (b0 < b1) load_keys(b0);
  la_commit();
  float acc[MT][NTW][4] = {};
  const float scale_log2 = p.scale * 1.4426950408889634f;

  for (int b = b0; b < b1; ++b) {
    if (b + 1 < b1) load_keys(b + 1);
    la_commit();
    la_wait<1>();
    __syncthreads();
    const T* kc = sC + (b & 1) * kLaKeys * ld;
    {
      float s[MT][4][4] = {};
#pragma unroll
      for (int k = 0; k < KS; ++k)
#pragma unroll
        for (int np = 0; np < 2; ++np) {                   // sixteen keys, one k16 step
          if (!kEven && k >= kn) continue;
          uint32_t bf[4];
          ldsm_x4(smem_u32(kc + (key0 + np * 16 + (lane >> 4) * 8 + (lane & 7)) * ld + (k0 + k) * 16 + ((lane >> 3) & 1) * 8), bf[0], bf[1], bf[2], bf[3]);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            MmaOp<T>::mma(s[m][np * 2], qf[m][k], bf[0], bf[1]);
            MmaOp<T>::mma(s[m][np * 2 + 1], qf[m][k], bf[2], bf[3]);
          }
        }
      float* dst = sS + kq * M * LDS;
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
          for (int half = 0; half < 2; ++half)
            *reinterpret_cast<float2*>(dst + (m * 16 + g + half * 8) * LDS + key0 + n * 8 + q4 * 2) = make_float2(s[m][n][half * 2], s[m][n][half * 2 + 1]);
    }
    __syncthreads();
    // softmax step of M / W rows per warp, all of them in flight (every block holds at least one visible key)
    {
      constexpr int NR = M / W;
      const int r0 = warp * NR, j = lo + b * kLaKeys + lane * 2;
      float2 v[NR];
      float old[NR], mx[NR], sum[NR];
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        v[i] = make_float2(0.f, 0.f);
        old[i] = sM[r0 + i];
#pragma unroll
        for (int k = 0; k < KG; ++k) {
          const float2 t = *reinterpret_cast<const float2*>(sS + (k * M + r0 + i) * LDS + lane * 2);
          v[i].x += t.x; v[i].y += t.y;
        }
        v[i].x = j <= pos ? v[i].x * scale_log2 : -INFINITY;
        v[i].y = j + 1 <= pos ? v[i].y * scale_log2 : -INFINITY;
        mx[i] = fmaxf(v[i].x, v[i].y);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int i = 0; i < NR; ++i) mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], o));
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        mx[i] = fmaxf(mx[i], old[i]);
        v[i].x = exp2f(v[i].x - mx[i]);
        v[i].y = exp2f(v[i].y - mx[i]);
        sum[i] = v[i].x + v[i].y;
        const T a0 = Num<T>::from_f(v[i].x), a1 = Num<T>::from_f(v[i].y);
        *reinterpret_cast<uint32_t*>(sP + (r0 + i) * LDP + lane * 2) = MmaOp<T>::pack(v[i].x, v[i].y);
        *reinterpret_cast<uint32_t*>(sP + (M + r0 + i) * LDP + lane * 2) = MmaOp<T>::pack(v[i].x - Num<T>::to_f(a0), v[i].y - Num<T>::to_f(a1));
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int i = 0; i < NR; ++i) sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], o);
      __syncwarp();
#pragma unroll
      for (int i = 0; i < NR; ++i)
        if (lane == i) {
          const float corr = exp2f(old[i] - mx[i]);
          sA[r0 + i] = corr;
          sL[r0 + i] = sL[r0 + i] * corr + sum[i];
          sM[r0 + i] = mx[i];
        }
    }
    __syncthreads();
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float c0 = sA[m * 16 + g], c1 = sA[m * 16 + g + 8];
#pragma unroll
      for (int t = 0; t < NTW; ++t) {
        acc[m][t][0] *= c0; acc[m][t][1] *= c0; acc[m][t][2] *= c1; acc[m][t][3] *= c1;
      }
    }
#pragma unroll
    for (int kk = 0; kk < kLaKeys; kk += 32) {
      uint32_t a[MT][2][2][4];                             // [m][value / remainder][k16 step]
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int hl = 0; hl < 2; ++hl)
#pragma unroll
          for (int hk = 0; hk < 2; ++hk)
            ldsm_x4(smem_u32(sP + (hl * M + m * 16 + (lane & 15)) * LDP + kk + hk * 16 + (lane >> 4) * 8), a[m][hl][hk][0], a[m][hl][hk][1],
                    a[m][hl][hk][2], a[m][hl][hk][3]);
#pragma unroll
      for (int t = 0; t < NTW; ++t) {
        const int c = (warp + t * W) * 8;
        if (c < vrank) {
          uint32_t bf[4];                                  // eight columns, 32 keys
          ldsm_x4_t(smem_u32(kc + (kk + lane) * ld + c), bf[0], bf[1], bf[2], bf[3]);
#pragma unroll
          for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int hl = 0; hl < 2; ++hl) {
              MmaOp<T>::mma(acc[m][t], a[m][hl][0], bf[0], bf[1]);
              MmaOp<T>::mma(acc[m][t], a[m][hl][1], bf[2], bf[3]);
            }
        }
      }
    }
    __syncthreads();                                       // the key buffer and the score tile are free again
  }
  __syncthreads();                                         // also for a range without blocks
  // ---- results
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = m * 16 + g + half * 8;
      if (r >= heads_here) continue;
      const size_t hr = (size_t)row * p.heads + h0 + r;
      const float inv = sp.splits == 1 ? 1.f / sL[r] : 1.f;
#pragma unroll
      for (int t = 0; t < NTW; ++t) {
        const int c = (warp + t * W) * 8 + q4 * 2;
        if (c >= vrank) continue;
        const float v0 = acc[m][t][half * 2] * inv, v1 = acc[m][t][half * 2 + 1] * inv;
        if (sp.splits == 1) *reinterpret_cast<uint32_t*>(reinterpret_cast<T*>(p.o) + hr * vrank + c) = MmaOp<T>::pack(v0, v1);
        else *reinterpret_cast<float2*>(sp.o + (hr * sp.splits + split) * vrank + c) = make_float2(v0, v1);
      }
      if (sp.splits > 1 && warp == 0 && q4 == 0) {
        sp.ml[(hr * sp.splits + split) * 2] = sM[r];
        sp.ml[(hr * sp.splits + split) * 2 + 1] = sL[r];
      }
    }
}

template <typename T>
__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentSplit sp, T* __restrict__ o, int rank) {
  pdl_prologue();
  const size_t hr = blockIdx.x;
  __shared__ float sw[64];                                 // weight of every split
  if (threadIdx.x < 32) {
    const float* ml = sp.ml + hr * sp.splits * 2;
    float m = -INFINITY, l = 0.f;
    for (int s = threadIdx.x; s < sp.splits; s += 32) m = fmaxf(m, ml[s * 2]);
    m = warp_max(m);
    for (int s = threadIdx.x; s < sp.splits; s += 32) {
      const float w = exp2f(ml[s * 2] - m);                // a split without keys: maximum -inf, weight 0
      sw[s] = w;
      l += w * ml[s * 2 + 1];
    }
    l = warp_sum(l);
    for (int s = threadIdx.x; s < sp.splits; s += 32) sw[s] /= l;
  }
  __syncthreads();
  for (int c = threadIdx.x * 4; c < rank; c += blockDim.x * 4) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < sp.splits; ++s) {
      const float4 t = *reinterpret_cast<const float4*>(sp.o + (hr * sp.splits + s) * rank + c);
      const float w = sw[s];
      v.x += w * t.x; v.y += w * t.y; v.z += w * t.z; v.w += w * t.w;
    }
    uint2 u;
    u.x = MmaOp<T>::pack(v.x, v.y);
    u.y = MmaOp<T>::pack(v.z, v.w);
    *reinterpret_cast<uint2*>(o + hr * rank + c) = u;
  }
}

// Split the keys of a row until about one CTA per SM exists.
static int la_splits(int rows, int heads, int max_kv) {
  const int mt = heads <= 16 ? 1 : 2, ctas = rows * ceil_div(heads, 16 * mt), blocks = ceil_div(std::max(max_kv, 1), kLaKeys);
  return std::max(1, std::min(std::min(sm_count() / std::max(ctas, 1), blocks), 64));
}

}  // namespace rf

using namespace rf;

#define RF_DISPATCH3(dtype, ...)                                        \
  if ((dtype) == kF16) { using T = __half; __VA_ARGS__; }               \
  else if ((dtype) == kBF16) { using T = __nv_bfloat16; __VA_ARGS__; }  \
  else { using T = float; __VA_ARGS__; }

static int check_rows(const RfRows* r) {
  RF_REQUIRE(r && r->pos && r->page_table && r->pt_stride > 0, "latent attention: positions and page table");
  return RF_OK;
}

static int check_insert(const RfLatentInsert* c) {
  RF_REQUIRE(c && (c->x || c->q), "latent_insert: neither latents nor query latents");
  if (c->x) {
    RF_REQUIRE(c->norm_w && c->pool && c->rank > 0 && c->rank % 16 == 0 && c->rank_true > 0 && c->rank_true <= c->rank && c->ldx % 8 == 0, "latent_insert arguments");
    RF_REQUIRE(c->rot >= 0 && c->rot % 2 == 0 && c->rot_pad >= c->rot && c->rot_pad % 16 == 0 && (c->rot_pad == 0 || (c->rot > 0 && c->cos && c->sin)),
               "latent_insert: rotated part of %d values", c->rot);
  }
  if (c->q) RF_REQUIRE(c->q_norm && c->q_rank > 0 && c->q_rank % 8 == 0 && c->ldq % 8 == 0 && c->q_rank_true > 0 && c->q_rank_true <= c->q_rank, "latent_insert: query latents");
  return check_rows(&c->rows);
}

extern "C" int rf_latent_insert(const RfLatentInsert* c, int32_t dtype, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  int rc = check_insert(c);
  if (rc) return rc;
  if (c->n_rows == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int items = c->n_rows * ((c->x ? 1 : 0) + (c->q ? 1 : 0));
  RF_DISPATCH3(dtype, RF_CUDA_CHECK(::rf::launch_k(latent_insert_kernel<T>, dim3(ceil_div(items, 4)), dim3(128), 0, s, 1, *c)));
  ::rf::count_launch();
  return RF_OK;
}

static int check_rotate(const RfHeadRotate* a) {
  RF_REQUIRE(a && a->x && a->y && a->pos && a->cos && a->sin && a->heads > 0 && a->dims > 0 && a->dims % 2 == 0 && a->dims_pad >= a->dims && a->dims_pad % 8 == 0,
             "head_rotate arguments");
  RF_REQUIRE(a->ldx % 8 == 0 && a->xs % 8 == 0 && a->ldy % 8 == 0 && a->ys % 8 == 0, "head_rotate: pitches must be multiples of 8");
  return RF_OK;
}

extern "C" int rf_head_rotate(const RfHeadRotate* a, int32_t dtype, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  int rc = check_rotate(a);
  if (rc) return rc;
  if (a->rows == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int64_t items = (int64_t)a->rows * a->heads * (a->dims_pad / 8);
  RF_DISPATCH3(dtype, RF_CUDA_CHECK(::rf::launch_k(head_rotate_kernel<T>, dim3((unsigned)((items + 255) / 256)), dim3(256), 0, s, 1, *a)));
  ::rf::count_launch();
  return RF_OK;
}

extern "C" int rf_latent_gather(const void* pool, void* out, const RfRows* rows, const int32_t* kv_start, const int32_t* kv_len,
                                int32_t rank, int32_t max_len, int32_t dtype, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_REQUIRE(pool && out && kv_start && kv_len && rank > 0 && rank % 16 == 0 && max_len > 0, "latent_gather arguments");
  int rc = check_rows(rows);
  if (rc) return rc;
  RF_REQUIRE(rows->q_start && rows->q_len && rows->num_seqs > 0, "latent_gather works on portions");
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int blocks = (int)std::min<int64_t>(ceil_div(max_len, 1) * (int64_t)(rank / 8) / 1024 + 1, 512);
  RF_DISPATCH3(dtype, RF_CUDA_CHECK(::rf::launch_k(latent_gather_kernel<T>, dim3(blocks, rows->num_seqs), dim3(256), 0, s, 1,
                                                   (const T*)pool, (T*)out, *rows, kv_start, kv_len, rank)));
  ::rf::count_launch();
  return RF_OK;
}

static int check_head_linear(const RfHeadLinear* a) {
  RF_REQUIRE(a && a->x && a->y && a->w && a->heads > 0 && a->n > 0 && a->k > 0, "head_linear arguments");
  RF_REQUIRE(a->n % 8 == 0 && a->k % 8 == 0 && a->xs % 8 == 0 && a->ys % 8 == 0 && a->ldx % 8 == 0 && a->ldy % 8 == 0,
             "head_linear: sizes and pitches must be multiples of 8");
  return RF_OK;
}

extern "C" int rf_head_linear(const RfHeadLinear* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  int rc = check_head_linear(a);
  if (rc) return rc;
  if (a->rows == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (a->dtype == kF16) return launch_head_linear_mma<__half>(a, nullptr, nullptr, s);
  if (a->dtype == kBF16) return launch_head_linear_mma<__nv_bfloat16>(a, nullptr, nullptr, s);
  RF_DISPATCH3(a->dtype, RF_CUDA_CHECK(::rf::launch_k(head_linear_kernel<T>, dim3(ceil_div(a->n, kHlN), a->heads, ceil_div(a->rows, kHlRows)),
                                                      dim3(128), 0, s, 1, *a)));
  ::rf::count_launch();
  return RF_OK;
}

extern "C" int rf_latent_absorb(const RfHeadLinear* q, const RfLatentInsert* c, const RfHeadRotate* t, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_REQUIRE(q != nullptr, "latent_absorb: no queries");
  int rc = c ? check_insert(c) : RF_OK;
  if (!rc && t) rc = check_rotate(t);
  if (rc) return rc;
  RF_REQUIRE(!c || (c->x && !c->q), "latent_absorb inserts cached rows only");
  if (q->dtype == kF32 || q->rows == 0) {
    if (c) rc = rf_latent_insert(c, q->dtype, stream);
    if (!rc && t) rc = rf_head_rotate(t, q->dtype, stream);
    return rc ? rc : rf_head_linear(q, stream);
  }
  rc = check_head_linear(q);
  if (rc) return rc;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return q->dtype == kF16 ? launch_head_linear_mma<__half>(q, c, t, s) : launch_head_linear_mma<__nv_bfloat16>(q, c, t, s);
}

// Room for the largest split of any launch of at most `rows` rows.
extern "C" uint64_t rf_latent_attn_scratch_bytes(int rows, int heads, int rank, int max_kv) {
  uint64_t most = 0;
  const int ht = ceil_div(std::max(heads, 1), heads <= 16 ? 16 : 32);
  for (int r = 1; r <= rows && r * ht <= sm_count(); ++r) {
    const int sp = la_splits(r, heads, max_kv);
    if (sp > 1) most = std::max<uint64_t>(most, (uint64_t)r * heads * sp * (rank + 2) * sizeof(float));
  }
  return most;
}

template <typename T>
static int launch_latent_attn_mma(const RfLatentAttn* a, cudaStream_t s) {
  LatentSplit sp = {};
  sp.splits = la_splits(a->n_rows, a->heads, a->max_kv);
  const int vrank = a->vrank > 0 ? a->vrank : a->rank;
  const uint64_t slots = (uint64_t)a->n_rows * a->heads * sp.splits;
  if (sp.splits > 1 && (!a->ws || a->ws_bytes < slots * (a->rank + 2) * sizeof(float))) sp.splits = 1;
  sp.o = a->ws;
  sp.ml = a->ws ? a->ws + slots * a->rank : nullptr;
  const int mt = a->heads <= 16 ? 1 : 2;
  const dim3 grid(sp.splits, ceil_div(a->heads, 16 * mt), a->n_rows);
#define RF_LM(NT, MT)                                                                                             \
  do {                                                                                                            \
    constexpr int smem = LaGeom<NT, MT>::total;                                                                   \
    RF_ALLOW_SMEM_PER_DEVICE((latent_attn_mma_kernel<T, NT, MT>), smem);                                          \
    RF_CUDA_CHECK(::rf::launch_k(latent_attn_mma_kernel<T, NT, MT>, grid, dim3(32 * LaGeom<NT, MT>::W), smem, s, 1, *a, sp)); \
  } while (0)
#define RF_LN(NT)             \
  do {                        \
    if (mt == 1) RF_LM(NT, 1); \
    else RF_LM(NT, 2);         \
  } while (0)
  if (a->rank <= 64) RF_LN(1);
  else if (a->rank <= 128) RF_LN(2);
  else if (a->rank <= 192) RF_LN(3);
  else if (a->rank <= 256) RF_LN(4);
  else if (a->rank <= 320) RF_LN(5);
  else if (a->rank <= 512) RF_LN(8);
  else RF_LN(9);
#undef RF_LN
#undef RF_LM
  ::rf::count_launch();
  if (sp.splits > 1) {
    RF_CUDA_CHECK(::rf::launch_k(latent_combine_kernel<T>, dim3(a->n_rows * a->heads), dim3(std::min(128, round_up(vrank / 4, 32))), 0, s, 1,
                                 sp, (T*)a->o, vrank));
    ::rf::count_launch();
  }
  return RF_OK;
}

template <typename T>
static int launch_latent_attn(const RfLatentAttn* a, cudaStream_t s) {
  const size_t smem = ((size_t)4 * a->rank + 8) * sizeof(float);
  const int per_lane = ceil_div(a->rank, 32);
#define RF_LA(N)                                                                                                  \
  if (per_lane <= N) {                                                                                            \
    RF_CUDA_CHECK(::rf::launch_k(latent_attn_kernel<T, N>, dim3(a->n_rows, a->heads), dim3(128), smem, s, 1, *a)); \
    ::rf::count_launch();                                                                                         \
    return RF_OK;                                                                                                 \
  }
  RF_LA(2) RF_LA(4) RF_LA(8) RF_LA(16) RF_LA(32) RF_LA(64)
#undef RF_LA
  return fail(RF_ERR_UNSUPPORTED, "latent attention: rank %d is larger than 2048", a->rank);
}

extern "C" int rf_latent_attn(const RfLatentAttn* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_REQUIRE(a && a->q && a->o && a->pool && a->heads > 0 && a->rank > 0 && a->rank % 16 == 0, "latent_attn arguments");
  int rc = check_rows(&a->rows);
  if (rc) return rc;
  if (a->n_rows == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  RF_REQUIRE(a->vrank >= 0 && a->vrank % 16 == 0 && a->vrank <= a->rank, "latent_attn: %d value columns of %d", a->vrank, a->rank);
  const bool mma = a->rank <= 576 && (a->vrank > 0 ? a->vrank : a->rank) <= 512;
  if (mma && a->dtype == kF16) return launch_latent_attn_mma<__half>(a, s);
  if (mma && a->dtype == kBF16) return launch_latent_attn_mma<__nv_bfloat16>(a, s);
  RF_DISPATCH3(a->dtype, return launch_latent_attn<T>(a, s));
}
