// The scan of a state-space mixer with one decay per head and token (linear_scan.cu, MODE_STATE_SPACE) for long prompt
// portions, as products over chunks of 64 tokens. With dt = softplus(dt_pre + bias_h), a_t = -exp(A_h) dt_t and the running
// sum c_t of a within a chunk that starts from the state S_0:
//
//   y_t = e^(c_t) S_0^T C_t + sum_{s <= t} e^(c_t - c_s) dt_s (C_t . B_s) x_s + D_h x_t
//   S'  = e^(c_end) S_0 + sum_s e^(c_end - c_s) dt_s B_s x_s^T
//
//  * leave kernel   : what every chunk leaves from a zero state (the last sum) and its decay e^(c_end);
//  * combine kernel : walks a request's chunks in order, leaves each one's starting state S_0 in the place of that sum,
//                     and stores the request's slot;
//  * read kernel    : the scores C B^T of a chunk once for all heads of a group that the CTA handles, then per head
//                     the weighted scores times x plus C times S_0.
//
// Everything is 32-bit on CUDA cores (the state and what enters it must be), but as register-tiled products: a thread
// holds 4 x 4 or 8 x 4 sums and spends a 16-byte read of shared memory on eight or eleven multiply-adds, where the
// token-by-token form spends one on four. The running sums are kept in 64-bit: the difference of two of them is what decays a weight, and
// in 32-bit it would lose the digits that a long or fast decaying chunk has accumulated. Every exponent is at most zero.
//
// Chunks are numbered over the whole step, request b's from cu_q[b] / 64 + b on (gaps of at most one), so scratch and
// grid follow the step's tokens, however unequal the requests are; a request of one token costs one chunk of one row.
#define TS_PDL_CLASS PDL_OTHER
#include <cuda_pipeline_primitives.h>

#include "common.cuh"

namespace ts {

constexpr int SC_Q = 64;              // tokens of a chunk
constexpr int SC_V = 64;              // value columns of a CTA
constexpr int SC_LD = SC_Q + 4;       // row of a tile whose fast index is the token (16-byte aligned, spread over the banks)
constexpr int SC_MAX_STATE = 128;

struct ScanChunkArgs {
  const float* c; int c_stride;       // [T, G * N] rows c_stride apart
  const float* b; int b_stride;
  const float* x; int x_stride;       // [T, H * dv]
  const float* dt_pre; int dt_stride; // [T, H]
  const float* dt_bias; const float* a_log; const float* skip;      // [H]
  float* state; int state_stride;     // [slots, H * N * dv]
  const int* cu_q; const int* state_slots;
  int num_seqs, H, per_group, N, dv;
  float* out;                         // [T, H, dv]
  float* left;                        // [chunks, H, N, dv]: what a chunk leaves, then its starting state
  float* decay;                       // [chunks, H]
  int heads_per_cta;                  // read kernel: heads of one group
};

__device__ __forceinline__ float sc_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// The request and the tokens of chunk g of the step; false for a number that belongs to no chunk.
__device__ __forceinline__ bool find_chunk(const ScanChunkArgs& a, int g, int& t0, int& nt) {
  int lo = 0, hi = a.num_seqs - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (a.cu_q[mid] / SC_Q + mid <= g) lo = mid; else hi = mid - 1;
  }
  const int start = a.cu_q[lo], end = a.cu_q[lo + 1];
  t0 = start + (g - (start / SC_Q + lo)) * SC_Q;
  nt = min(SC_Q, end - t0);
  return nt > 0;
}

// By one warp: dt and the running sums of the chunk's tokens for head h (two tokens a lane); tokens past the end have dt 0.
__device__ __forceinline__ void chunk_steps(const ScanChunkArgs& a, int h, int t0, int nt, int lane, float* dt_s, double* cum_s) {
  const float rate = expf(a.a_log[h]), bias = a.dt_bias[h];
  float dt[2];
  double sum[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int t = 2 * lane + i;
    dt[i] = t < nt ? sc_softplus(a.dt_pre[(size_t)(t0 + t) * a.dt_stride + h] + bias) : 0.f;
    sum[i] = -(double)(rate * dt[i]);
  }
  double run = sum[0] + sum[1];
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double other = __shfl_up_sync(0xffffffffu, run, o);
    if (lane >= o) run += other;
  }
  dt_s[2 * lane] = dt[0];
  dt_s[2 * lane + 1] = dt[1];
  cum_s[2 * lane] = run - sum[1];
  cum_s[2 * lane + 1] = run;
}

// acc[4 A][4] += A^T B over k rows: A's rows hold the 4 A-wide operand (row `lda` floats, this thread's part from `ar`), B's
// the 4-wide one. Both 16-byte aligned.
template <int A>
__device__ __forceinline__ void tile_product(float (&acc)[4 * A][4], const float* ar, int lda, const float* br, int ldb, int k) {
#pragma unroll 4
  for (int i = 0; i < k; ++i) {
    const float4 b = *reinterpret_cast<const float4*>(br + i * ldb);
#pragma unroll
    for (int q = 0; q < A; ++q) {
      const float4 a = *reinterpret_cast<const float4*>(ar + i * lda + 4 * q);
      const float av[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        acc[4 * q + r][0] = fmaf(av[r], b.x, acc[4 * q + r][0]);
        acc[4 * q + r][1] = fmaf(av[r], b.y, acc[4 * q + r][1]);
        acc[4 * q + r][2] = fmaf(av[r], b.z, acc[4 * q + r][2]);
        acc[4 * q + r][3] = fmaf(av[r], b.w, acc[4 * q + r][3]);
      }
    }
  }
}

// Loads in flight per thread before the first is stored to shared memory: one after the other each would wait for memory.
constexpr int SC_LOADS = 8;

// [nt rows of `width`] -> tile [SC_Q][ld], zero past the edges; four columns an access where the source allows it.
__device__ __forceinline__ void load_rows(const float* src, int stride, int rows, int width, bool vec, float* dst, int ld, int cols,
                                          int total_rows, int tid, int threads) {
  const int quads = cols / 4, total = total_rows * quads;
  for (int base = tid; base < total; base += threads * SC_LOADS) {
    float4 v[SC_LOADS];
#pragma unroll
    for (int u = 0; u < SC_LOADS; ++u) {
      const int idx = base + u * threads, r = idx / quads, c = (idx - r * quads) * 4;
      v[u] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (idx < total && r < rows) {
        const float* p = src + (size_t)r * stride + c;
        if (vec && c + 4 <= width) {
          v[u] = *reinterpret_cast<const float4*>(p);
        } else {
          if (c < width) v[u].x = p[0];
          if (c + 1 < width) v[u].y = p[1];
          if (c + 2 < width) v[u].z = p[2];
          if (c + 3 < width) v[u].w = p[3];
        }
      }
    }
#pragma unroll
    for (int u = 0; u < SC_LOADS; ++u) {
      const int idx = base + u * threads, r = idx / quads, c = (idx - r * quads) * 4;
      if (idx < total) *reinterpret_cast<float4*>(dst + r * ld + c) = v[u];
    }
  }
}

__device__ __forceinline__ bool rows_aligned(const float* p, int stride) { return (((uintptr_t)p) & 15) == 0 && (stride & 3) == 0; }

// What a chunk leaves: [N x dv] per head. A CTA is (chunk, head, 64 value columns); NP = the state size rounded up to 64.
template <int NP>
__global__ void __launch_bounds__(2 * NP) chunk_leave_kernel(ScanChunkArgs a) {
  constexpr int THREADS = 2 * NP;     // (NP / 8) x (64 / 4) tiles of 8 x 4
  extern __shared__ __align__(16) float sc_smem[];
  float* b_s = sc_smem;               // [SC_Q][NP], weighted
  float* x_s = b_s + SC_Q * NP;       // [SC_Q][SC_V]
  __shared__ float dt_s[SC_Q];
  __shared__ double cum_s[SC_Q];
  pdl_trigger();
  pdl_wait();
  int t0, nt;
  const int g = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * SC_V;
  if (!find_chunk(a, g, t0, nt)) return;
  const int tid = threadIdx.x, lane = tid & 31;
  const int grp = h / a.per_group, N = a.N;
  if (tid < 32) chunk_steps(a, h, t0, nt, lane, dt_s, cum_s);
  const float* xp = a.x + (size_t)t0 * a.x_stride + h * a.dv + v0;
  const float* bp = a.b + (size_t)t0 * a.b_stride + grp * N;
  load_rows(xp, a.x_stride, nt, min(SC_V, a.dv - v0), rows_aligned(xp, a.x_stride), x_s, SC_V, SC_V, nt, tid, THREADS);
  load_rows(bp, a.b_stride, nt, N, rows_aligned(bp, a.b_stride), b_s, NP, NP, nt, tid, THREADS);
  __syncthreads();
  // the weights go on x, the smaller tile of the two
  const double end = cum_s[SC_Q - 1];
  for (int idx = tid; idx < nt * (SC_V / 4); idx += THREADS) {
    const int t = idx / (SC_V / 4);
    const float w = expf((float)(end - cum_s[t])) * dt_s[t];
    float4* p = reinterpret_cast<float4*>(x_s) + idx;
    float4 v = *p;
    v.x *= w; v.y *= w; v.z *= w; v.w *= w;
    *p = v;
  }
  if (tid == 0 && blockIdx.z == 0) a.decay[(size_t)g * a.H + h] = expf((float)end);
  __syncthreads();
  const int n_at = (tid / 16) * 8, v_at = (tid % 16) * 4;
  float acc[8][4] = {};
  tile_product<2>(acc, b_s + n_at, NP, x_s + v_at, SC_V, nt);
  float* dst = a.left + ((size_t)g * a.H + h) * N * a.dv + v0 + v_at;
  const bool vec = (a.dv & 3) == 0 && v0 + v_at + 4 <= a.dv;
#pragma unroll
  for (int r = 0; r < 8; ++r) {
    if (n_at + r >= N) break;
    float* p = dst + (size_t)(n_at + r) * a.dv;
    if (vec) {
      *reinterpret_cast<float4*>(p) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (v0 + v_at + j < a.dv) p[j] = acc[r][j];
    }
  }
}

// A request's chunks in order; a thread per VEC state elements. Eight chunks' loads in flight, then the chain.
template <int VEC>
__global__ void chunk_combine_kernel(ScanChunkArgs a) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x, h = blockIdx.y;
  const int idx = (blockIdx.z * blockDim.x + threadIdx.x) * VEC;
  const int start = a.cu_q[b], n = a.cu_q[b + 1] - start;
  const int per_head = a.N * a.dv;
  if (n <= 0 || idx >= per_head) return;
  const int chunks = (n + SC_Q - 1) / SC_Q, first = start / SC_Q + b;
  float* slot = a.state + (size_t)a.state_slots[b] * a.state_stride + (size_t)h * per_head + idx;
  const size_t stride = (size_t)a.H * per_head;
  float* p0 = a.left + ((size_t)first * a.H + h) * per_head + idx;
  const float* d0 = a.decay + (size_t)first * a.H + h;
  float s[VEC];
#pragma unroll
  for (int e = 0; e < VEC; ++e) s[e] = slot[e];
  for (int c0 = 0; c0 < chunks; c0 += 8) {
    float left[8][VEC], dec[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const bool in = c0 + j < chunks;
      dec[j] = in ? d0[(size_t)(c0 + j) * a.H] : 0.f;
      if constexpr (VEC == 4) {
        const float4 v = in ? *reinterpret_cast<const float4*>(p0 + (size_t)(c0 + j) * stride) : make_float4(0.f, 0.f, 0.f, 0.f);
        left[j][0] = v.x; left[j][1] = v.y; left[j][2] = v.z; left[j][3] = v.w;
      } else {
        left[j][0] = in ? p0[(size_t)(c0 + j) * stride] : 0.f;
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (c0 + j < chunks) {
        float* p = p0 + (size_t)(c0 + j) * stride;
        if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(s[0], s[1], s[2], s[3]); else p[0] = s[0];
#pragma unroll
        for (int e = 0; e < VEC; ++e) s[e] = fmaf(dec[j], s[e], left[j][e]);
      }
    }
  }
#pragma unroll
  for (int e = 0; e < VEC; ++e) slot[e] = s[e];
}

// The token rows of C or B, transposed: tile [n][SC_LD] with the token as fast index, zero past the chunk's end and past N.
__device__ __forceinline__ void load_transposed(const float* src, int stride, int nt, int N, int NP, float* dst, int warp, int warps, int lane) {
  const bool vec = rows_aligned(src, stride);
  const int t_local = lane & 7, n4 = (lane >> 3) * 4;      // a warp takes 8 tokens x 16 columns
  const int tiles = (SC_Q / 8) * (NP / 16);
  for (int base = warp; base < tiles; base += warps * SC_LOADS) {
    float v[SC_LOADS][4];
#pragma unroll
    for (int u = 0; u < SC_LOADS; ++u) {
      const int tile = base + u * warps, t = (tile & 7) * 8 + t_local, n = (tile >> 3) * 16 + n4;
#pragma unroll
      for (int e = 0; e < 4; ++e) v[u][e] = 0.f;
      if (tile < tiles && t < nt) {
        const float* p = src + (size_t)t * stride + n;
        if (vec && n + 4 <= N) {
          const float4 q = *reinterpret_cast<const float4*>(p);
          v[u][0] = q.x; v[u][1] = q.y; v[u][2] = q.z; v[u][3] = q.w;
        } else {
#pragma unroll
          for (int e = 0; e < 4; ++e)
            if (n + e < N) v[u][e] = p[e];
        }
      }
    }
#pragma unroll
    for (int u = 0; u < SC_LOADS; ++u) {
      const int tile = base + u * warps, t = (tile & 7) * 8 + t_local, n = (tile >> 3) * 16 + n4;
      if (tile < tiles) {
#pragma unroll
        for (int e = 0; e < 4; ++e) dst[(n + e) * SC_LD + t] = v[u][e];
      }
    }
  }
}

// The read-outs of a chunk. A CTA is (chunk, some heads of one group, 64 value columns).
constexpr int SC_READ_THREADS = 256;  // (64 / 4) x (64 / 4) tiles of 4 x 4: two CTAs of eight warps an SM
template <int NP>
__global__ void __launch_bounds__(SC_READ_THREADS, 2) chunk_read_kernel(ScanChunkArgs a) {
  extern __shared__ __align__(16) float sc_smem[];
  float* c_s = sc_smem;               // [NP][SC_LD]: C, token fastest
  float* s_s = c_s + NP * SC_LD;      // [NP][SC_LD]: B, token fastest; then [NP][SC_V]: the starting state of a head
  float* x_s = s_s + NP * SC_LD;      // [SC_Q][SC_V]
  float* m_s = x_s + SC_Q * SC_V;     // [SC_Q][SC_LD]: weighted scores, row s, token t fastest
  __shared__ float dt_s[SC_Q], fall_s[SC_Q];
  __shared__ double cum_s[SC_Q];
  pdl_trigger();
  pdl_wait();
  int t0, nt;
  const int g = blockIdx.x, v0 = blockIdx.z * SC_V, N = a.N;
  if (!find_chunk(a, g, t0, nt)) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h0 = blockIdx.y * a.heads_per_cta, grp = h0 / a.per_group;
  load_transposed(a.c + (size_t)t0 * a.c_stride + grp * N, a.c_stride, nt, N, NP, c_s, warp, SC_READ_THREADS / 32, lane);
  load_transposed(a.b + (size_t)t0 * a.b_stride + grp * N, a.b_stride, nt, N, NP, s_s, warp, SC_READ_THREADS / 32, lane);
  auto load_x = [&](int h) {
    const float* xp = a.x + (size_t)t0 * a.x_stride + h * a.dv + v0;
    load_rows(xp, a.x_stride, nt, min(SC_V, a.dv - v0), rows_aligned(xp, a.x_stride), x_s, SC_V, SC_V, SC_Q, tid, SC_READ_THREADS);
    if (warp == 0) chunk_steps(a, h, t0, nt, lane, dt_s, cum_s);
  };
  load_x(h0);
  __syncthreads();
  const int t_at = (tid / 16) * 4, col = (tid % 16) * 4;   // this thread's tokens; its keys s, or its value columns
  const bool live = t_at < nt;
  const int cols = min(SC_V, a.dv - v0);
  float score[4][4] = {};
  if (live && col <= t_at + 3) tile_product<1>(score, c_s + t_at, SC_LD, s_s + col, SC_LD, N);
  for (int h = h0; h < h0 + a.heads_per_cta; ++h) {
    __syncthreads();                  // B, or the head before, has been read
    // the head's starting state travels while the weighted scores are made
    const float* sp = a.left + ((size_t)g * a.H + h) * N * a.dv + v0;
    if (cols == SC_V && rows_aligned(sp, a.dv)) {
      for (int idx = tid; idx < N * (SC_V / 4); idx += SC_READ_THREADS)
        __pipeline_memcpy_async(s_s + idx * 4, sp + (size_t)(idx / (SC_V / 4)) * a.dv + (idx % (SC_V / 4)) * 4, 16);
    } else {
      load_rows(sp, a.dv, N, cols, rows_aligned(sp, a.dv), s_s, SC_V, SC_V, N, tid, SC_READ_THREADS);
    }
    __pipeline_commit();
    if (h > h0) {
      load_x(h);
      __syncthreads();
    }
    if (tid < SC_Q) fall_s[tid] = expf((float)cum_s[tid]);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int s = col + j;
      float m[4];
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int t = t_at + r;
        m[r] = s <= t && t < nt ? score[r][j] * expf((float)(cum_s[t] - cum_s[s])) * dt_s[s] : 0.f;
      }
      *reinterpret_cast<float4*>(m_s + s * SC_LD + t_at) = make_float4(m[0], m[1], m[2], m[3]);
    }
    __pipeline_wait_prior(0);
    __syncthreads();
    if (live) {
      float acc[4][4] = {};
      tile_product<1>(acc, c_s + t_at, SC_LD, s_s + col, SC_V, N);
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const float f = fall_s[t_at + r];
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[r][j] *= f;
      }
      tile_product<1>(acc, m_s + t_at, SC_LD, x_s + col, SC_V, min(nt, t_at + 4));
      const float skip = a.skip[h];
      const bool vec = (a.dv & 3) == 0 && col + 4 <= cols;
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int t = t_at + r;
        if (t >= nt) break;
        const float4 xv = *reinterpret_cast<const float4*>(x_s + t * SC_V + col);
        const float y[4] = {fmaf(skip, xv.x, acc[r][0]), fmaf(skip, xv.y, acc[r][1]), fmaf(skip, xv.z, acc[r][2]), fmaf(skip, xv.w, acc[r][3])};
        float* p = a.out + ((size_t)(t0 + t) * a.H + h) * a.dv + v0 + col;
        if (vec) {
          *reinterpret_cast<float4*>(p) = make_float4(y[0], y[1], y[2], y[3]);
        } else {
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (col + j < cols) p[j] = y[j];
        }
      }
    }
  }
}

template <int NP>
static int launch_chunks(const ScanChunkArgs& a, int chunks, cudaStream_t stream) {
  const int vblocks = (a.dv + SC_V - 1) / SC_V;
  const size_t leave = sizeof(float) * SC_Q * (NP + SC_V);
  const size_t read = sizeof(float) * (2 * (size_t)NP * SC_LD + SC_Q * SC_V + SC_Q * SC_LD);
  auto lk = chunk_leave_kernel<NP>;
  auto rk = chunk_read_kernel<NP>;
  static bool allowed = false;
  if (!allowed) {
    if (int e = (int)cudaFuncSetAttribute(lk, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)leave)) return e;
    if (int e = (int)cudaFuncSetAttribute(rk, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)read)) return e;
    allowed = true;
  }
  if (int e = launch(lk, dim3(chunks, a.H, vblocks), 2 * NP, leave, stream, a)) return e;
  const int per_head = a.N * a.dv;
  const int vec = per_head % 4 == 0 ? 4 : 1;
  const dim3 cgrid(a.num_seqs, a.H, (per_head / vec + 127) / 128);
  if (int e = vec == 4 ? launch(chunk_combine_kernel<4>, cgrid, 128, 0, stream, a) : launch(chunk_combine_kernel<1>, cgrid, 128, 0, stream, a)) return e;
  return launch(rk, dim3(chunks, a.H / a.heads_per_cta, vblocks), SC_READ_THREADS, read, stream, a);
}

}  // namespace ts

using namespace ts;

extern "C" int ts_state_space_chunk_tokens() { return SC_Q; }

// c, b [T, groups * n], x [T, heads * dv], dt_pre [T, heads], all float with rows of their own strides; left [chunks, heads, n, dv]
// and decay [chunks, heads] are scratch with chunks = num_tokens / 64 + num_seqs. n up to 128. out [T, heads, dv].
extern "C" int ts_state_space_chunks(const float* c, int c_stride, const float* b, int b_stride, const float* x, int x_stride,
                                     const float* dt_pre, int dt_stride, const float* dt_bias, const float* a_log, const float* skip,
                                     float* state, int state_stride, const int* cu_q, const int* state_slots, int num_seqs, int num_tokens,
                                     int heads, int groups, int n, int dv, float* left, float* decay, float* out, cudaStream_t stream) {
  if (num_seqs <= 0 || num_tokens <= 0) return 0;
  if (heads <= 0 || groups <= 0 || heads % groups || n <= 0 || dv <= 0 || !left || !decay || !state || !out) return TS_ERR_BAD_ARGUMENT;
  if (n > SC_MAX_STATE) return TS_ERR_UNSUPPORTED;
  ScanChunkArgs a;
  a.c = c; a.c_stride = c_stride; a.b = b; a.b_stride = b_stride; a.x = x; a.x_stride = x_stride;
  a.dt_pre = dt_pre; a.dt_stride = dt_stride; a.dt_bias = dt_bias; a.a_log = a_log; a.skip = skip;
  a.state = state; a.state_stride = state_stride; a.cu_q = cu_q; a.state_slots = state_slots;
  a.num_seqs = num_seqs; a.H = heads; a.per_group = heads / groups; a.N = n; a.dv = dv;
  a.out = out; a.left = left; a.decay = decay;
  const int chunks = num_tokens / SC_Q + num_seqs, vblocks = (dv + SC_V - 1) / SC_V;
  // as many heads of a group per CTA as leave a few CTAs for every place on the machine (the scores are made once for them)
  int hp = a.per_group;
  while (hp > 1 && (long long)chunks * vblocks * (heads / hp) < 148 * 2 * 3) {
    do --hp; while (a.per_group % hp);
  }
  a.heads_per_cta = hp;
  return n <= 64 ? launch_chunks<64>(a, chunks, stream) : launch_chunks<128>(a, chunks, stream);
}
