// Queries, keys and values on their way to attention for mixers that do more than norm and rotate: an optional
// short causal convolution over time on every channel of q, k and v, a rotation of the first `rotary_dim` elements
// of every query and key head (neighbouring pairs or i with i + rotary_dim / 2), an optional division of the
// rotated head by its root mean square (no weight). Queries go to q_out [T, heads, d], keys to
// k_cache [pages, kv_heads, page_size, d], values to v_cache [pages, kv_heads, page_size, dv] at the token's
// slot. q, k and v are the first columns, in that order, of one projection's rows. From the convolution's first
// product to the division everything is 32-bit, rounded once.
//
// Convolution: y_t = sum_j taps[j] * u_(t - K + 1 + j); inputs before this step's first token of a request come
// from its state row [(K - 1), channels] (32-bit, zero at the request's start), which afterwards holds the
// request's last K - 1 inputs: written by the same kernel in a step of single tokens, where a channel's inputs
// have one reader, and by a kernel behind it otherwise.
#define TS_PDL_CLASS PDL_ELEMENTWISE
#include "common.cuh"

namespace ts {

struct RotateArgs {
  const void* proj; int stride;           // [T, >= channels] rows `stride` apart
  const void* taps;                       // [K, channels] (tap by tap), or null: no convolution
  int num_taps;
  float* state; int state_stride;         // [slots, (K - 1) * channels]
  const int* cu_q; const int* state_slots;
  int num_seqs;
  const float* cos_tab; const float* sin_tab;
  int rotary_dim, interleaved, unit_norm;
  float eps;
  const int* slots;
  void* k_cache; void* v_cache;
  int page_size, num_tokens, heads, kv_heads, d, dv;
  void* q_out;
  int single;                             // every request brings one token: the state is moved on here
  int lanes;                              // lanes per head (vector form)
};

// The request of token t: the last b with cu_q[b] <= t.
__device__ __forceinline__ int request_of(const int* cu_q, int num_seqs, int t) {
  int lo = 0, hi = num_seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_q[mid] <= t) lo = mid; else hi = mid - 1;
  }
  return lo;
}

// A group of `lanes` lanes per (token, head), a lane VEC neighbouring elements in one 16-byte access.
template <typename T>
__global__ void __launch_bounds__(256) qkv_rotate_kernel(RotateArgs a) {
  constexpr int VEC = Vec<T>::N;
  pdl_trigger();
  pdl_wait();
  const int jobs = a.heads + 2 * a.kv_heads;
  long long group = ((long long)blockIdx.x * blockDim.x + threadIdx.x) / a.lanes;
  const int sub = threadIdx.x & (a.lanes - 1);
  const bool live = group < (long long)a.num_tokens * jobs;     // lanes behind the last head stay for the shuffles
  if (!live) group = 0;
  const int t = (int)(group / jobs), job = (int)(group - (long long)t * jobs);
  const bool is_v = job >= a.heads + a.kv_heads;
  const int width = is_v ? a.dv : a.d;
  const int e0 = sub * VEC;
  const bool on = live && e0 < width;
  const int qk_cols = (a.heads + a.kv_heads) * a.d, channels = qk_cols + a.kv_heads * a.dv;
  const int col = is_v ? qk_cols + (job - a.heads - a.kv_heads) * a.dv + e0 : job * a.d + e0;
  const T* proj = (const T*)a.proj;
  float x[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) x[e] = 0.f;
  if (on) {
    const T* cur = proj + (size_t)t * a.stride + col;
    if (a.taps) {
      const T* taps = (const T*)a.taps;
      const int K = a.num_taps;
      const int b = request_of(a.cu_q, a.num_seqs, t);
      const int start = a.cu_q[b];
      float* st = K > 1 ? a.state + (size_t)a.state_slots[b] * a.state_stride + col : nullptr;
      float last[VEC];
      for (int j = 0; j < K; ++j) {
        const int src = t - K + 1 + j;
        float u[VEC], w[VEC];
        if (src >= start) {
          Vec<T> v;
          v.load(proj + (size_t)src * a.stride + col);
          v.unpack(u);
        } else {
          const float* row = st + (size_t)(K - 1 + src - start) * channels;
#pragma unroll
          for (int e = 0; e < VEC; e += 4) Quad<float>::load(row + e, u + e);
        }
        Vec<T> wv;
        wv.load(taps + (size_t)j * channels + col);
        wv.unpack(w);
#pragma unroll
        for (int e = 0; e < VEC; ++e) { x[e] = fmaf(w[e], u[e], x[e]); last[e] = u[e]; }
      }
      if (a.single && K > 1) {
        // this lane is the only reader of these channels' inputs: row i takes row i + 1, the last one the current input
        for (int i = 0; i < K - 2; ++i) {
          float u[VEC];
#pragma unroll
          for (int e = 0; e < VEC; e += 4) Quad<float>::load(st + (size_t)(i + 1) * channels + e, u + e);
#pragma unroll
          for (int e = 0; e < VEC; e += 4) Quad<float>::store(st + (size_t)i * channels + e, u + e);
        }
#pragma unroll
        for (int e = 0; e < VEC; e += 4) Quad<float>::store(st + (size_t)(K - 2) * channels + e, last + e);
      }
    } else {
      Vec<T> v;
      v.load(cur);
      v.unpack(x);
    }
  }
  constexpr unsigned mask = 0xffffffffu;
  __syncwarp();
  if (a.rotary_dim) {
    const int half = a.rotary_dim >> 1;
    const float* cs = a.cos_tab + (size_t)t * half;
    const float* sn = a.sin_tab + (size_t)t * half;
    if (a.interleaved) {
      if (!is_v && on) {
#pragma unroll
        for (int e = 0; e < VEC; e += 2) {
          if (e0 + e < a.rotary_dim) {
            const int p = (e0 + e) >> 1;
            const float c = cs[p], s = sn[p], u = x[e], v = x[e + 1];
            x[e] = u * c - v * s;
            x[e + 1] = v * c + u * s;
          }
        }
      }
    } else {
      // half is a multiple of VEC here: the partners of a lane's elements are all in one other lane
      const int hl = half / VEC;
      const int partner = (threadIdx.x & 31 & ~(a.lanes - 1)) | (sub < hl ? sub + hl : sub < 2 * hl ? sub - hl : sub);
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const float o = __shfl_sync(mask, x[e], partner);
        if (!is_v && e0 + e < a.rotary_dim) {
          const int p = e0 + e < half ? e0 + e : e0 + e - half;
          x[e] = e0 + e < half ? x[e] * cs[p] - o * sn[p] : x[e] * cs[p] + o * sn[p];
        }
      }
    }
  }
  if (a.unit_norm) {
    float ss = 0.f;
#pragma unroll
    for (int e = 0; e < VEC; ++e) ss = fmaf(x[e], x[e], ss);
    for (int o = a.lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(mask, ss, o);
    if (!is_v) {
      const float rstd = rsqrtf(ss / (float)a.d + a.eps);
#pragma unroll
      for (int e = 0; e < VEC; ++e) x[e] *= rstd;
    }
  }
  if (!on) return;
  T* dst;
  if (job < a.heads) {
    dst = (T*)a.q_out + ((size_t)t * a.heads + job) * a.d;
  } else {
    const int slot = a.slots[t];
    const int page = slot / a.page_size, off = slot - page * a.page_size;
    const int g = is_v ? job - a.heads - a.kv_heads : job - a.heads;
    dst = (T*)(is_v ? a.v_cache : a.k_cache) + (((size_t)page * a.kv_heads + g) * a.page_size + off) * width;
  }
  Vec<T> r;
  r.pack(x);
  r.store(dst + e0);
}

// Any size and alignment: a warp per (token, head), the head in shared memory.
constexpr int QR_WARPS = 4, QR_MAX_DIM = 256;
template <typename T>
__global__ void __launch_bounds__(QR_WARPS * 32) qkv_rotate_any_kernel(RotateArgs a) {
  __shared__ float rows[QR_WARPS][QR_MAX_DIM];
  pdl_trigger();
  pdl_wait();
  const int jobs = a.heads + 2 * a.kv_heads;
  const long long id = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  if (id >= (long long)a.num_tokens * jobs) return;
  float* row = rows[threadIdx.x >> 5];
  const int t = (int)(id / jobs), job = (int)(id - (long long)t * jobs);
  const bool is_v = job >= a.heads + a.kv_heads;
  const int width = is_v ? a.dv : a.d;
  const int qk_cols = (a.heads + a.kv_heads) * a.d, channels = qk_cols + a.kv_heads * a.dv;
  const int col = is_v ? qk_cols + (job - a.heads - a.kv_heads) * a.dv : job * a.d;
  const T* proj = (const T*)a.proj;
  const int K = a.num_taps;
  const int b = a.taps ? request_of(a.cu_q, a.num_seqs, t) : 0;
  const int start = a.taps ? a.cu_q[b] : 0;
  float* st = a.taps && K > 1 ? a.state + (size_t)a.state_slots[b] * a.state_stride + col : nullptr;
  for (int i = lane; i < width; i += 32) {
    float x = 0.f;
    if (a.taps) {
      const T* taps = (const T*)a.taps + col + i;
      float u = 0.f;
      for (int j = 0; j < K; ++j) {
        const int src = t - K + 1 + j;
        u = src >= start ? to_float(proj[(size_t)src * a.stride + col + i]) : st[(size_t)(K - 1 + src - start) * channels + i];
        x = fmaf(to_float(taps[(size_t)j * channels]), u, x);
      }
      if (a.single && K > 1) {
        for (int r = 0; r < K - 2; ++r) st[(size_t)r * channels + i] = st[(size_t)(r + 1) * channels + i];
        st[(size_t)(K - 2) * channels + i] = u;
      }
    } else {
      x = to_float(proj[(size_t)t * a.stride + col + i]);
    }
    row[i] = x;
  }
  __syncwarp();
  const int half = a.rotary_dim >> 1;
  auto value = [&](int i) -> float {           // element i after the rotation
    const float x = row[i];
    if (is_v || i >= a.rotary_dim) return x;
    const bool first = a.interleaved ? (i & 1) == 0 : i < half;
    const int p = a.interleaved ? i >> 1 : first ? i : i - half;
    const float o = row[a.interleaved ? (first ? i + 1 : i - 1) : (first ? i + half : i - half)];
    const float c = a.cos_tab[(size_t)t * half + p], s = a.sin_tab[(size_t)t * half + p];
    return first ? x * c - o * s : x * c + o * s;
  };
  float rstd = 1.f;
  if (a.unit_norm && !is_v) {
    float ss = 0.f;
    for (int i = lane; i < width; i += 32) { const float v = value(i); ss = fmaf(v, v, ss); }
    rstd = rsqrtf(warp_sum(ss) / (float)a.d + a.eps);
  }
  T* dst;
  if (job < a.heads) {
    dst = (T*)a.q_out + ((size_t)t * a.heads + job) * a.d;
  } else {
    const int slot = a.slots[t];
    const int page = slot / a.page_size, off = slot - page * a.page_size;
    const int g = is_v ? job - a.heads - a.kv_heads : job - a.heads;
    dst = (T*)(is_v ? a.v_cache : a.k_cache) + (((size_t)page * a.kv_heads + g) * a.page_size + off) * width;
  }
  for (int i = lane; i < width; i += 32) dst[i] = from_float<T>(value(i) * rstd);
}

// The state after the step: row i of a request becomes its input at position end - (K - 1) + i. Rows are written in
// order, and a row that is read from the state lies behind the one that is written.
template <typename T>
__global__ void conv_inputs_update_kernel(RotateArgs a, int channels) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x, K = a.num_taps;
  const int start = a.cu_q[b], end = a.cu_q[b + 1];
  if (end <= start) return;
  float* st = a.state + (size_t)a.state_slots[b] * a.state_stride;
  const T* proj = (const T*)a.proj;
  for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < channels; c += gridDim.y * blockDim.x)
    for (int i = 0; i < K - 1; ++i) {
      const int src = end - (K - 1) + i;
      st[(size_t)i * channels + c] = src >= start ? to_float(proj[(size_t)src * a.stride + c]) : st[(size_t)(K - 1 + src - start) * channels + c];
    }
}

}  // namespace ts

using namespace ts;

template <typename T>
static int qkv_rotate(RotateArgs a, cudaStream_t stream) {
  constexpr int VEC = Vec<T>::N;
  const int channels = (a.heads + a.kv_heads) * a.d + a.kv_heads * a.dv;
  const int wide = a.d > a.dv ? a.d : a.dv;
  int lanes = 1;
  while (lanes * VEC < wide) lanes <<= 1;
  const bool vec = lanes <= 32 && a.d % VEC == 0 && a.dv % VEC == 0 && a.stride % VEC == 0 &&
      (a.interleaved || a.rotary_dim % (2 * VEC) == 0) && (!a.state || a.state_stride % 4 == 0) &&
      ((((uintptr_t)a.proj) | ((uintptr_t)a.taps) | ((uintptr_t)a.state) | ((uintptr_t)a.q_out) | ((uintptr_t)a.k_cache) | ((uintptr_t)a.v_cache)) & 15) == 0;
  const long long jobs = (long long)a.num_tokens * (a.heads + 2 * a.kv_heads);
  int st;
  if (vec) {
    a.lanes = lanes;
    st = launch(qkv_rotate_kernel<T>, (unsigned)((jobs * lanes + 255) / 256), 256, 0, stream, a);
  } else {
    st = launch(qkv_rotate_any_kernel<T>, (unsigned)((jobs + QR_WARPS - 1) / QR_WARPS), QR_WARPS * 32, 0, stream, a);
  }
  if (st != 0 || !a.taps || a.num_taps == 1 || a.single) return st;
  int by = (channels + 127) / 128;
  if (by > 64) by = 64;
  return launch(conv_inputs_update_kernel<T>, dim3(a.num_seqs, by), 128, 0, stream, a, channels);
}

// proj [T, >= (heads + kv_heads) * d + kv_heads * dv]: q, then k, then v. taps [num_taps, channels] or null (then
// state, cu_q and state_slots are not read). single: every request brings exactly one token.
extern "C" int ts_qkv_rotate(const void* proj, int stride, const void* taps, int num_taps, float* state, int state_stride,
                             const int* cu_q, const int* state_slots, int num_seqs, const float* cos_tab, const float* sin_tab,
                             int rotary_dim, int interleaved, int unit_norm, float eps, const int* slots, void* k_cache,
                             void* v_cache, int page_size, int num_tokens, int heads, int kv_heads, int d, int dv, void* q_out,
                             int single, int dtype, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (d <= 0 || dv <= 0 || d > QR_MAX_DIM || dv > QR_MAX_DIM) return TS_ERR_UNSUPPORTED;
  if (rotary_dim < 0 || rotary_dim > d || (rotary_dim & 1) || (rotary_dim && (!cos_tab || !sin_tab))) return TS_ERR_BAD_ARGUMENT;
  if (!slots || !k_cache || !v_cache || page_size <= 0 || heads <= 0 || kv_heads <= 0) return TS_ERR_BAD_ARGUMENT;
  if (taps && (num_taps < 1 || !cu_q || num_seqs <= 0 || (num_taps > 1 && (!state || !state_slots)))) return TS_ERR_BAD_ARGUMENT;
  RotateArgs a;
  a.proj = proj; a.stride = stride; a.taps = taps; a.num_taps = taps ? num_taps : 0; a.state = taps ? state : nullptr;
  a.state_stride = state_stride; a.cu_q = cu_q; a.state_slots = state_slots; a.num_seqs = num_seqs; a.cos_tab = cos_tab;
  a.sin_tab = sin_tab; a.rotary_dim = rotary_dim; a.interleaved = interleaved; a.unit_norm = unit_norm; a.eps = eps;
  a.slots = slots; a.k_cache = k_cache; a.v_cache = v_cache; a.page_size = page_size; a.num_tokens = num_tokens;
  a.heads = heads; a.kv_heads = kv_heads; a.d = d; a.dv = dv; a.q_out = q_out; a.single = single; a.lanes = 32;
  if (dtype == TS_DTYPE_F32) return qkv_rotate<float>(a, stream);
  if (dtype == TS_DTYPE_BF16) return qkv_rotate<bf16>(a, stream);
  return TS_ERR_BAD_ARGUMENT;
}
