// Paged attention whose heads' weights are mixed before they meet the values ("talking heads"):
//
//   s_h(i, j) = scale * q_h(i) . k_{kv(h)}(j), optionally capped: cap * tanh(s / cap)
//   p_h(i, .) = softmax over the visible j (causal, optionally the last `window` positions), optionally with a
//               sink logit per head in the denominator
//   w_h(i, j) = sum_g T[h, g] p_g(i, j)
//   o_h(i)    = sum_j w_h(i, j) v_{kv(h)}(j)
//
// A weight of one head reaches every head, so the softmax of all heads must be finished (maximum and sum) before
// the first value is weighted: the keys are visited twice, first for every head's maximum and sum, then again for the
// normalised weights, their mixing and the product with the values. Because the weights of the second visit
// are already normalised, partial outputs over ranges of the keys simply add up.
//
// This file holds the form on CUDA cores, for float and bf16, any head count and head size, and single tokens whose
// keys are cut into ranges. A CTA owns all heads of a few queries of one request. Everything is 32-bit.
#define TS_PDL_CLASS PDL_ATTENTION
#include "talking_attention.cuh"

namespace ts {

constexpr int TK_THREADS = 256, TK_KEYS = 32;
constexpr int PHASE_BOTH = 0, PHASE_STATS = 1, PHASE_VALUES = 2;

template <typename T>
__global__ void __launch_bounds__(TK_THREADS) talking_attention_kernel(TalkArgs a, int QT, int phase) {
  extern __shared__ float sm[];
  const int H = a.num_heads, G = a.num_kv_heads, per = H / G, D = a.head_dim, DV = a.v_head_dim;
  const int tile_w = (D + 1 > DV ? D + 1 : DV);
  float* Qs = sm;                                   // [QT][H][D], times scale
  float* Ss = Qs + (size_t)QT * H * D;              // [QT][H][KEYS] scores, then weights
  float* Ws = Ss + (size_t)QT * H * TK_KEYS;        // [QT][H][KEYS] mixed weights
  float* tile = Ws + (size_t)QT * H * TK_KEYS;      // [KEYS][tile_w] keys (stride D + 1) or values (stride DV)
  float* Os = tile + (size_t)TK_KEYS * tile_w;      // [QT][H][DV]
  float* Ms = Os + (size_t)QT * H * DV;             // [QT][H] maximum
  float* Ls = Ms + (size_t)QT * H;                  // [QT][H] sum, then its inverse
  float* Ts = Ls + (size_t)QT * H;                  // [H][H]
  pdl_trigger();
  pdl_wait();
  const int seq = blockIdx.y;
  const int row0 = a.cu_q[seq], n = a.cu_q[seq + 1] - row0;
  const int q0 = blockIdx.x * QT;
  if (q0 >= n) return;
  const int ctx = a.ctx_lens[seq];
  const int first_pos = ctx - n + q0;               // position of the tile's first query
  const int nq = min(QT, n - q0);
  const int last_pos = first_pos + nq - 1;
  const int lo = a.window > 0 ? max(0, first_pos - a.window + 1) : 0;
  // this CTA's range of the keys (whole tiles, so that ranges never share one)
  const int tiles = (last_pos + 1 - lo + TK_KEYS - 1) / TK_KEYS;
  const int tiles_each = (tiles + a.num_splits - 1) / a.num_splits;
  const int k_begin = lo + blockIdx.z * tiles_each * TK_KEYS;
  const int k_end = min(last_pos + 1, k_begin + tiles_each * TK_KEYS);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int* table = a.block_tables + (size_t)seq * a.table_width;
  const T* q = (const T*)a.q;
  const T* kc = (const T*)a.k_cache;
  const T* vc = (const T*)a.v_cache;

  for (int idx = tid; idx < nq * H * D; idx += TK_THREADS) Qs[idx] = to_float(q[(size_t)(row0 + q0) * H * D + idx]) * a.scale;
  for (int idx = tid; idx < nq * H * DV; idx += TK_THREADS) Os[idx] = 0.f;
  for (int idx = tid; idx < H * H; idx += TK_THREADS) Ts[idx] = a.talk ? a.talk[idx] : (idx / H == idx % H ? 1.f : 0.f);
  for (int idx = tid; idx < nq * H; idx += TK_THREADS) {
    float m = -INFINITY, l = 0.f;
    if (phase == PHASE_VALUES) {                    // the ranges' maxima and sums were left by the launch before
      const float* ml = a.part_ml + ((size_t)(row0 + q0) * H + idx) * a.num_splits * 2;
      for (int s = 0; s < a.num_splits; ++s) m = fmaxf(m, ml[2 * s]);
      for (int s = 0; s < a.num_splits; ++s)
        if (ml[2 * s] != -INFINITY) l += ml[2 * s + 1] * expf(ml[2 * s] - m);
    }
    Ms[idx] = m;
    Ls[idx] = l;
  }
  __syncthreads();

  // scores of all heads for the keys k0 .. k0 + KEYS - 1 into Ss (minus infinity where a query does not see the key)
  auto scores = [&](int k0) {
    for (int g = 0; g < G; ++g) {
      __syncthreads();
      for (int idx = tid; idx < TK_KEYS * D; idx += TK_THREADS) {
        const int kk = idx / D, c = idx - kk * D, kpos = k0 + kk;
        tile[kk * (D + 1) + c] = kpos < k_end ? to_float(kc[talk_row(table, kpos, g, a) * D + c]) : 0.f;
      }
      __syncthreads();
      for (int idx = tid; idx < nq * per * TK_KEYS; idx += TK_THREADS) {
        const int kk = idx & (TK_KEYS - 1), rest = idx / TK_KEYS;
        const int r = rest / per, h = g * per + (rest - r * per);
        const int kpos = k0 + kk, qpos = first_pos + r;
        const bool seen = kpos < k_end && kpos <= qpos && (a.window <= 0 || kpos > qpos - a.window);
        float s = -INFINITY;
        if (seen) {
          const float* qr = Qs + ((size_t)r * H + h) * D;
          const float* kr = tile + kk * (D + 1);
          s = 0.f;
          for (int c = 0; c < D; ++c) s = fmaf(qr[c], kr[c], s);
          if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
        }
        Ss[((size_t)r * H + h) * TK_KEYS + kk] = s;
      }
    }
    __syncthreads();
  };

  if (phase != PHASE_VALUES) {
    for (int k0 = k_begin; k0 < k_end; k0 += TK_KEYS) {
      scores(k0);
      for (int rh = warp; rh < nq * H; rh += TK_THREADS / 32) {
        const float s = Ss[(size_t)rh * TK_KEYS + lane];
        const float m_old = Ms[rh], m = fmaxf(m_old, warp_max(s));
        const float sum = warp_sum(s == -INFINITY ? 0.f : expf(s - m));
        __syncwarp();
        if (lane == 0) {
          Ls[rh] = (m_old == -INFINITY ? 0.f : Ls[rh] * expf(m_old - m)) + sum;
          Ms[rh] = m;
        }
      }
    }
    __syncthreads();
  }
  if (phase == PHASE_STATS) {
    for (int idx = tid; idx < nq * H; idx += TK_THREADS) {
      float* ml = a.part_ml + (((size_t)(row0 + q0) * H + idx) * a.num_splits + blockIdx.z) * 2;
      ml[0] = Ms[idx];
      ml[1] = Ls[idx];
    }
    return;
  }
  for (int idx = tid; idx < nq * H; idx += TK_THREADS) {
    float m = Ms[idx], l = Ls[idx];
    if (a.sinks) {
      const float sink = a.sinks[idx % H], top = fmaxf(m, sink);
      l = (m == -INFINITY ? 0.f : l * expf(m - top)) + expf(sink - top);
      m = top;
    }
    Ms[idx] = m;
    Ls[idx] = 1.f / l;
  }
  for (int k0 = k_begin; k0 < k_end; k0 += TK_KEYS) {
    scores(k0);
    for (int idx = tid; idx < nq * H * TK_KEYS; idx += TK_THREADS) {
      const float s = Ss[idx];
      const int rh = idx / TK_KEYS;
      Ss[idx] = s == -INFINITY ? 0.f : expf(s - Ms[rh]) * Ls[rh];
    }
    __syncthreads();
    for (int idx = tid; idx < nq * H * TK_KEYS; idx += TK_THREADS) {
      const int kk = idx & (TK_KEYS - 1), rh = idx / TK_KEYS, r = rh / H, h = rh - r * H;
      const float* pr = Ss + (size_t)r * H * TK_KEYS + kk;
      const float* tr = Ts + h * H;
      float w = 0.f;
      for (int g = 0; g < H; ++g) w = fmaf(tr[g], pr[g * TK_KEYS], w);
      Ws[idx] = w;
    }
    for (int g = 0; g < G; ++g) {
      __syncthreads();
      for (int idx = tid; idx < TK_KEYS * DV; idx += TK_THREADS) {
        const int kk = idx / DV, c = idx - kk * DV, kpos = k0 + kk;
        tile[idx] = kpos < k_end ? to_float(vc[talk_row(table, kpos, g, a) * DV + c]) : 0.f;
      }
      __syncthreads();
      for (int idx = tid; idx < nq * per * DV; idx += TK_THREADS) {
        const int c = idx % DV, rest = idx / DV, r = rest / per, h = g * per + (rest - r * per);
        const float* wr = Ws + ((size_t)r * H + h) * TK_KEYS;
        float o = 0.f;
        for (int kk = 0; kk < TK_KEYS; ++kk) o = fmaf(wr[kk], tile[kk * DV + c], o);
        Os[((size_t)r * H + h) * DV + c] += o;
      }
    }
  }
  __syncthreads();
  if (a.num_splits == 1) {
    T* out = (T*)a.out + (size_t)(row0 + q0) * H * DV;
    for (int idx = tid; idx < nq * H * DV; idx += TK_THREADS) out[idx] = from_float<T>(Os[idx]);
  } else {
    // part_out [T][splits][H * DV]
    for (int idx = tid; idx < nq * H * DV; idx += TK_THREADS) {
      const int r = idx / (H * DV), c = idx - r * (H * DV);
      a.part_out[((size_t)(row0 + q0 + r) * a.num_splits + blockIdx.z) * H * DV + c] = Os[idx];
    }
  }
}

// The ranges' outputs of every token added up in order.
template <typename T>
__global__ void talking_combine_kernel(const float* part, T* out, int splits, int width, size_t total) {
  pdl_trigger();
  pdl_wait();
  for (size_t idx = (size_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (size_t)gridDim.x * blockDim.x) {
    const size_t t = idx / width, c = idx - t * width;
    float o = 0.f;
    for (int s = 0; s < splits; ++s) o += part[(t * splits + s) * width + c];
    out[idx] = from_float<T>(o);
  }
}

static size_t talk_smem(const TalkArgs& a, int QT) {
  const size_t H = a.num_heads, D = a.head_dim, DV = a.v_head_dim;
  return sizeof(float) * (QT * H * D + 2 * QT * H * TK_KEYS + TK_KEYS * (D + 1 > DV ? D + 1 : DV) + QT * H * DV + 2 * QT * H + H * H);
}

template <typename T>
static int launch_talking(const TalkArgs& a, int num_seqs, int max_query_len, int num_tokens, cudaStream_t stream) {
  constexpr size_t LIMIT = 227 * 1024;
  int QT = max_query_len >= 4 ? 4 : max_query_len;
  while (QT > 1 && talk_smem(a, QT) > LIMIT) --QT;
  const size_t smem = talk_smem(a, QT);
  if (smem > LIMIT) return TS_ERR_UNSUPPORTED;
  auto kern = talking_attention_kernel<T>;
  static size_t allowed = 0;
  if (smem > 48 * 1024 && smem > allowed) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    allowed = smem;
  }
  const dim3 grid((max_query_len + QT - 1) / QT, num_seqs, a.num_splits);
  if (a.num_splits == 1) return launch(kern, grid, TK_THREADS, smem, stream, a, QT, PHASE_BOTH);
  if (int e = launch(kern, grid, TK_THREADS, smem, stream, a, QT, PHASE_STATS)) return e;
  if (int e = launch(kern, grid, TK_THREADS, smem, stream, a, QT, PHASE_VALUES)) return e;
  const int width = a.num_heads * a.v_head_dim;
  const size_t total = (size_t)num_tokens * width;
  size_t blocks = (total + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  return launch(talking_combine_kernel<T>, (unsigned)blocks, 256, 0, stream, (const float*)a.part_out, (T*)a.out, a.num_splits, width, total);
}

}  // namespace ts

using namespace ts;

// q [T, heads, d], out [T, heads, dv]; talk [heads, heads] float (null: no mixing); sinks [heads] float or null; softcap
// 0 = none; window 0 = every earlier position. num_splits > 1 cuts the keys of every query into ranges: part_ml
// [T, heads, splits, 2] and part_out [T, splits, heads * dv] are scratch.
extern "C" int ts_talking_attention(const void* q, void* out, const void* k_cache, const void* v_cache, const int* block_tables,
                                    int table_width, const int* cu_q, const int* ctx_lens, int num_seqs, int max_query_len,
                                    int num_tokens, int heads, int kv_heads, int d, int dv, int page_size, float scale,
                                    int window, float softcap, const float* talk, const float* sinks, int num_splits,
                                    float* part_ml, float* part_out, int dtype, cudaStream_t stream) {
  if (num_seqs <= 0 || num_tokens <= 0) return 0;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || d <= 0 || dv <= 0 || page_size <= 0 || max_query_len <= 0 || window < 0)
    return TS_ERR_BAD_ARGUMENT;
  if (num_splits < 1 || (num_splits > 1 && (!part_ml || !part_out))) return TS_ERR_BAD_ARGUMENT;
  TalkArgs a;
  a.q = q; a.out = out; a.k_cache = k_cache; a.v_cache = v_cache; a.block_tables = block_tables; a.table_width = table_width;
  a.cu_q = cu_q; a.ctx_lens = ctx_lens; a.num_heads = heads; a.num_kv_heads = kv_heads; a.head_dim = d; a.v_head_dim = dv;
  a.page_size = page_size; a.page_shift = page_shift_of(page_size); a.scale = scale; a.window = window; a.softcap = softcap;
  a.talk = talk; a.sinks = sinks; a.num_splits = num_splits; a.part_ml = part_ml; a.part_out = part_out;
  if (dtype == TS_DTYPE_F32) return launch_talking<float>(a, num_seqs, max_query_len, num_tokens, stream);
  if (dtype == TS_DTYPE_BF16) return launch_talking<bf16>(a, num_seqs, max_query_len, num_tokens, stream);
  return TS_ERR_BAD_ARGUMENT;
}
