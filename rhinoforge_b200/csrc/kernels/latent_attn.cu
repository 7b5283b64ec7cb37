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
template <typename T>
__global__ void latent_insert_kernel(const T* __restrict__ x, int64_t ldx, const float* __restrict__ w, T* __restrict__ pool,
                                     const RfRows rows, int n_rows, int rank, int rank_true, float eps) {
  pdl_prologue();
  const int row = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5), lane = threadIdx.x & 31;   // one warp per row
  if (row >= n_rows) return;
  const T* xr = x + (size_t)row * ldx;
  float s = 0.f;
  for (int i = lane; i < rank; i += 32) {
    const float v = Num<T>::to_f(xr[i]);
    s += v * v;
  }
  const float rstd = rsqrtf(warp_sum(s) / (float)rank_true + eps);
  const int pos = rows.pos[row];
  const int page = rows.page_table[(size_t)seq_slot(rows, row_seq(rows, row)) * rows.pt_stride + (pos >> 4)];
  T* dst = pool + ((size_t)page * 16 + (pos & 15)) * rank;
  for (int i = lane; i < rank; i += 32) dst[i] = Num<T>::from_f(Num<T>::to_f(xr[i]) * rstd * w[i]);
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
  T* o = reinterpret_cast<T*>(p.o) + ((size_t)row * p.heads + h) * rank;
  for (int i = threadIdx.x; i < rank; i += 128) {
    float v = 0.f;
    for (int w = 0; w < 4; ++w) v += f[w] * sm[w * rank + i];
    o[i] = Num<T>::from_f(v / tot);
  }
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

extern "C" int rf_latent_insert(const void* x, int64_t ldx, const float* norm_w, void* pool, const RfRows* rows, int32_t n_rows,
                                int32_t rank, int32_t rank_true, float eps, int32_t dtype, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_REQUIRE(x && norm_w && pool && rank > 0 && rank % 16 == 0 && rank_true > 0 && rank_true <= rank, "latent_insert arguments");
  int rc = check_rows(rows);
  if (rc) return rc;
  if (n_rows == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  RF_DISPATCH3(dtype, RF_CUDA_CHECK(::rf::launch_k(latent_insert_kernel<T>, dim3(ceil_div(n_rows, 4)), dim3(128), 0, s, 1,
                                                   (const T*)x, ldx, norm_w, (T*)pool, *rows, n_rows, rank, rank_true, eps)));
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

extern "C" int rf_head_linear(const RfHeadLinear* a, rf_stream_t stream) {
  RF_SKIP_IF_REPLAYING();
  RF_REQUIRE(a && a->x && a->y && a->w && a->heads > 0 && a->n > 0 && a->k > 0, "head_linear arguments");
  RF_REQUIRE(a->n % 8 == 0 && a->k % 8 == 0 && a->xs % 8 == 0 && a->ys % 8 == 0 && a->ldx % 8 == 0 && a->ldy % 8 == 0,
             "head_linear: sizes and pitches must be multiples of 8");
  if (a->rows == 0) return RF_OK;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  RF_DISPATCH3(a->dtype, RF_CUDA_CHECK(::rf::launch_k(head_linear_kernel<T>, dim3(ceil_div(a->n, kHlN), a->heads, ceil_div(a->rows, kHlRows)),
                                                      dim3(128), 0, s, 1, *a)));
  ::rf::count_launch();
  return RF_OK;
}

extern "C" uint64_t rf_latent_attn_scratch_bytes(int rows, int heads, int rank, int max_kv) {
  (void)rows; (void)heads; (void)rank; (void)max_kv;
  return 0;
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
  RF_DISPATCH3(a->dtype, return launch_latent_attn<T>(a, s));
}
