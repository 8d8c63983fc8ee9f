// Arguments shared by the forms of attention whose heads' weights are mixed after the softmax.
#pragma once
#include "attention.cuh"

namespace ts {

struct TalkArgs {
  const void* q;             // [T, num_heads, head_dim]
  void* out;                 // [T, num_heads, v_head_dim]
  const void* k_cache;       // [pages, num_kv_heads, page_size, head_dim]
  const void* v_cache;       // [pages, num_kv_heads, page_size, v_head_dim]
  const int* block_tables; int table_width;
  const int* cu_q;           // [B + 1]
  const int* ctx_lens;       // [B]
  int num_heads, num_kv_heads, head_dim, v_head_dim, page_size, page_shift;
  float scale;
  int window;                // 0 = every earlier position
  float softcap;             // 0 = none
  const float* talk;         // [num_heads, num_heads] or null
  const float* sinks;        // [num_heads] or null
  int num_splits;
  float* part_ml;            // [T, num_heads, num_splits, 2]
  float* part_out;           // [T, num_splits, num_heads * v_head_dim]
};

// Row index (in units of one head's elements) of position `kpos` of a request for kv head `kvh`.
__device__ __forceinline__ size_t talk_row(const int* table, int kpos, int kvh, const TalkArgs& a) {
  int page, off;
  if (a.page_shift >= 0) {
    page = table[kpos >> a.page_shift];
    off = kpos & (a.page_size - 1);
  } else {
    const int idx = kpos / a.page_size;
    page = table[idx];
    off = kpos - idx * a.page_size;
  }
  return ((size_t)page * a.num_kv_heads + kvh) * a.page_size + off;
}

}  // namespace ts
