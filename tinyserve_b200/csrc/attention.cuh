// Arguments shared by the paged attention kernels.
#pragma once
#include "common.cuh"

namespace ts {

struct AttnArgs {
  const void* q;           // [T, num_heads, head_dim]
  void* out;               // [T, num_heads, head_dim]
  const void* k_cache;     // [pages, num_kv_heads, page_size, head_dim]
  const void* v_cache;
  const int* block_tables; // [B, table_width]
  const int* cu_q;         // [B + 1] first flat row of each request's new tokens
  const int* ctx_lens;     // [B] tokens of each request, the new ones included
  const int* seq_ids;      // requests this launch handles
  int num_seqs;            // how many of them
  int table_width;
  int num_heads, num_kv_heads, head_dim, page_size;
  int page_shift;          // log2(page_size) if it is a power of two, else -1
  float scale_log2;        // softmax scale times log2(e)
  int window;              // 0 = every earlier position; w = the last w positions
  // split-K decode
  int num_splits;
  float* part_acc;         // [num_seqs, num_heads, num_splits, head_dim]
  float* part_ml;          // [num_seqs, num_heads, num_splits, 2]  (max, sum)
  // Optional extras (kernels that do not know them leave them at their defaults).
  const float* sinks = nullptr;  // [num_heads] a logit per head that joins the softmax's denominator without a value
  int v_head_dim = 0;            // size of a value head when it differs from head_dim (0: the same)
  int keep_first = 0;            // with a window: positions below this stay visible to every later query
  int chunk = 0;                 // c > 0 (without a window): a query sees its own run of c positions, counted from position 0
  // 2: every query head and every cached key row holds two maps side by side (head_dim / 2 elements each) over the same
  // values. `num_heads` counts (head, map) pairs, map innermost; a pair scores with its own half of both rows.
  int maps = 1;
  // Two maps, kernels that finish a head themselves: out = (a1 - *mix_factor a2) / rms(.) * mix_mult per head
  const float* mix_factor = nullptr;
  float mix_mult = 1.f, mix_eps = 0.f;
};

// The row of q (in rows of head_dim elements) that holds a (head, map) pair of a token, and whether column c of it
// (all of an aligned run of 8 columns alike) belongs to that pair.
__device__ __forceinline__ size_t q_row_of(size_t token, int pair, const AttnArgs& a) {
  return a.maps == 2 ? token * (a.num_heads >> 1) + (pair >> 1) : token * a.num_heads + pair;
}
__device__ __forceinline__ bool q_col_lives(int pair, int c, int head_dim, const AttnArgs& a) {
  return a.maps != 2 || (2 * c >= head_dim) == ((pair & 1) != 0);
}

// The first position that a query at position p sees (the kept first positions of a window apart).
__device__ __forceinline__ int first_visible(int p, const AttnArgs& a) {
  if (a.window > 0) return max(0, p - a.window + 1);
  return a.chunk > 0 ? p / a.chunk * a.chunk : 0;
}

// The finished row: num / den, where the denominator also takes 2^(sink - max) when the head has
// a sink logit (given in natural units; the running maximum `mx` is in base-2 units).
__device__ __forceinline__ float finish_row(float num, float den, float mx, const float* sinks, int head) {
  if (!sinks) return num / den;
  const float sl = sinks[head] * 1.4426950408889634f;
  const float top = fmaxf(mx, sl);
  const float c = (mx == -INFINITY) ? 0.f : exp2f(mx - top);
  return num * c / (den * c + exp2f(sl - top));
}

__device__ __forceinline__ size_t kv_offset(int page, int kvh, int off, const AttnArgs& a) {
  return (((size_t)page * a.num_kv_heads + kvh) * a.page_size + off) * a.head_dim;
}

// Row index (in units of one head's elements) of position `kpos` of a request for kv head `kvh`.
__device__ __forceinline__ size_t kv_row_of(const int* table, int kpos, int kvh, const AttnArgs& a) {
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

// Element offset of position `kpos` of a request (block table `table`) for kv head `kvh`.
__device__ __forceinline__ size_t kv_offset_of(const int* table, int kpos, int kvh, const AttnArgs& a) {
  int page, off;
  if (a.page_shift >= 0) {
    page = table[kpos >> a.page_shift];
    off = kpos & (a.page_size - 1);
  } else {
    const int idx = kpos / a.page_size;
    page = table[idx];
    off = kpos - idx * a.page_size;
  }
  return kv_offset(page, kvh, off, a);
}

static inline int page_shift_of(int page_size) {
  if (page_size <= 0 || (page_size & (page_size - 1))) return -1;
  int s = 0;
  while ((1 << s) < page_size) ++s;
  return s;
}

// Merge of the key ranges of one request for `ng` heads starting at `head0`, by a whole CTA:
// out = sum_s w_s acc_s / sum_s w_s l_s with w_s = 2^(m_s - max_s m_s). The (max, sum) pairs are
// staged in shared memory first (`ml` holds ng * S * 2 floats), so that the loop over the ranges
// issues independent loads.
template <typename T>
__device__ __forceinline__ void merge_splits(const AttnArgs& a, int si, int qrow, int head0, int ng, float* ml) {
  const int S = a.num_splits, D = a.head_dim;
  for (int idx = threadIdx.x; idx < ng * S * 2; idx += blockDim.x) {
    const int r = idx / (S * 2), rest = idx - r * (S * 2);
    ml[idx] = __ldcg(&a.part_ml[((size_t)si * a.num_heads + head0 + r) * S * 2 + rest]);
  }
  __syncthreads();
  for (int idx = threadIdx.x; idx < ng * D; idx += blockDim.x) {
    const int r = idx / D, d = idx - r * D;
    const float* mlr = ml + (size_t)r * S * 2;
    float mm = -INFINITY;
    for (int sp = 0; sp < S; ++sp) mm = fmaxf(mm, mlr[sp * 2]);
    const float* acc = a.part_acc + ((size_t)si * a.num_heads + head0 + r) * S * D + d;
    float num = 0.f, den = 0.f;
    int sp = 0;
    for (; sp + 4 <= S; sp += 4) {
      float v[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) v[u] = __ldcg(acc + (size_t)(sp + u) * D);
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float ms = mlr[(sp + u) * 2];
        const float c = (ms == -INFINITY) ? 0.f : exp2f(ms - mm);
        num += v[u] * c;
        den += mlr[(sp + u) * 2 + 1] * c;
      }
    }
    for (; sp < S; ++sp) {
      const float ms = mlr[sp * 2];
      const float c = (ms == -INFINITY) ? 0.f : exp2f(ms - mm);
      num += __ldcg(acc + (size_t)sp * D) * c;
      den += mlr[sp * 2 + 1] * c;
    }
    ((T*)a.out)[((size_t)qrow * a.num_heads + head0 + r) * D + d] = from_float<T>(finish_row(num, den, mm, a.sinks, head0 + r));
  }
}

constexpr int ATTN_MAX_SPLITS = 32;

}  // namespace ts
