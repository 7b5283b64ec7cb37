// Kernel-side argument block shared by the attention kernels (attention.cu: mma.sync prefill and
// split-KV decode; attention_tc.cu: tcgen05 prefill).
#pragma once
#include <stdint.h>

namespace rf {

struct AttnParams {
  const void* q; int64_t ldq;
  void* out; int64_t ldo;
  const int32_t* page_table; int32_t pt_stride;
  int32_t paged;
  int32_t num_seqs, Hq, Hkv, G;
  const int32_t* q_start; const int32_t* q_len; const int32_t* kv_start; const int32_t* kv_len;
  int32_t max_q_len;
  int32_t causal, window;
  const uint8_t* mask; int64_t mask_ld, mask_seq_stride;
  const int32_t* seg_q; const int32_t* seg_k;
  float scale_log2;
  float* ws_o; float* ws_lse;
  int32_t splits, pages_per_split, stages;
  int32_t kv_stream;      // decode: K/V pages are read with the L2 evict-first policy
  int32_t* status;
  const int32_t* slot;    // page-table row of a sequence
  int32_t chunk;
  const float* sink;      // natural-log units
  const void* gate; int64_t ld_gate;
  int32_t gate_by_head, keep_first;
  const float* slopes;    // natural-log units per token of distance, or per unit of ln(1 + rate * distance)
  const float* rates;
  const int32_t* seq_of_row; const int32_t* pos;
  int32_t g_tiles;        // decode: CTAs that share one K/V head (16 query heads each)
};

constexpr float kLog2e = 1.4426950408889634f;
// log2(1 + rate * distance); distances in front of a row (masked by the caller) may give anything
__device__ __forceinline__ float log2_distance(float rate, float distance) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(fmaf(rate, distance, 1.f)));
  return y;
}
__device__ __forceinline__ float sigmoid_fast(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }


}  // namespace rf
