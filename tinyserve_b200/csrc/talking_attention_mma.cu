// Attention with the heads' weights mixed after the softmax (talking_attention.cuh) on the tensor cores, bf16: prompt
// portions and single tokens, head sizes in steps of 16 up to 128, up to 64 heads.
//
// A CTA owns 16 queries and up to 16 heads, a warp one head; with more heads (or more key/value heads than fit in
// shared memory) the CTAs of a thread-block cluster own a share of the heads each and hand their weights to one
// another through distributed shared memory, so no score is computed twice. Keys and values arrive in tiles of 16
// positions, two tiles in flight: by the TMA unit where keys and values are 64 or 128 wide and a tile lies in one page
// (boxes of 64 columns of all heads at once, 128-byte swizzle, the warps ask for them in turn), else by cp.async into padded rows
// (which the warps stall on: an SM takes in some 30 bytes a cycle). First visit of the keys: every head's row maxima and sums. Second visit,
// tile by tile:
//   S_h = Q_h K^T (mma.sync), capped, p_h = 2^(s - lse) in 32-bit, stored as two bf16 parts (value and remainder);
//   W = T P for all positions of the tile (mma.sync with T as the A operand, both parts of P as B: the mixed weights
//       have 32-bit sums of 16-bit-exact products and are rounded once, where they meet the values);
//   O_h += W_h V (mma.sync), accumulators in registers.
// Single tokens: one row of 16 is live, the keys are cut into ranges (a launch for the maxima and sums, one for the
// values, and the ranges' outputs added up, as in the CUDA-core form).
#define TS_PDL_CLASS PDL_ATTENTION
#include "talking_attention.cuh"
#include "bounded_wait.cuh"
#include "cache_map.cuh"

namespace ts {

constexpr int TM_ROWS = 16, TM_KEYS = 16, TM_ROWP = TM_KEYS + 8, TM_POS = TM_ROWS * TM_ROWP + 8;   // padded rows
constexpr int TM_BOTH = 0, TM_STATS = 1, TM_VALUES = 2;
constexpr float TM_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ uint32_t tm_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void tm_arm(uint64_t* bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(tm_smem(bar)), "r"(bytes) : "memory");
}
// A box of several heads x 16 rows x 64 columns of a page into shared memory, 128-byte swizzled.
__device__ __forceinline__ void tm_tensor(void* dst, const CUtensorMap* map, int x, int y, int z, uint64_t* bar) {
  asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
               ::"r"(tm_smem(dst)), "l"(map), "r"(tm_smem(bar)), "r"(x), "r"(y), "r"(z) : "memory");
}
__device__ __forceinline__ bool tm_try(uint32_t addr, uint32_t parity) {      // the phase is complete already, or soon
  uint32_t ok;
  asm volatile("{\n.reg .pred p;\nmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\nselp.u32 %0, 1, 0, p;\n}\n"
               : "=r"(ok) : "r"(addr), "r"(parity) : "memory");
  return ok != 0;
}
constexpr int TM_AHEAD = 64;                               // tiles whose rows are looked up together
constexpr int TM_BOX = TM_KEYS * 64;                       // elements of a box
template <int N>                                           // all but this thread's last N groups of copies have arrived
__device__ __forceinline__ void tm_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
// Shared memory is addressed in its own 32-bit window throughout.
__device__ __forceinline__ void tm_ldm(uint32_t (&r)[4], uint32_t smem) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem) : "memory");
}
__device__ __forceinline__ void tm_ldm_t(uint32_t (&r)[4], uint32_t smem) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem) : "memory");
}
__device__ __forceinline__ void tm_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float tm_ex2(float x) {         // arguments are at most 0, or small: no range handling
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ uint32_t tm_pack(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t*>(&v);
}

template <int CL>
__device__ __forceinline__ void tm_sync() {
  if constexpr (CL == 1) {
    __syncthreads();
  } else {
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
  }
}
template <int CL>
__device__ __forceinline__ void tm_store_all(uint32_t addr, uint32_t v) {        // to this address in every CTA of the cluster
  if constexpr (CL == 1) {
    asm volatile("st.shared.u32 [%0], %1;" ::"r"(addr), "r"(v) : "memory");
  } else {
#pragma unroll
    for (int c = 0; c < CL; ++c) {
      uint32_t remote;
      asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(addr), "r"(c));
      asm volatile("st.shared::cluster.u32 [%0], %1;" ::"r"(remote), "r"(v) : "memory");
    }
  }
}

// The scores of a fragment in base-2 units: scale, or scale and soft cap. tanh by its Taylor series up to the 11th
// power while every argument of the warp is small (the next term is below 2e-8 of the value at 0.35), tanhf otherwise.
// Two elements an instruction (packed 32-bit arithmetic).
struct CapArgs { float mul, cap2; bool capped; };    // capped: cap2 * tanh(mul * s); else mul * s
__device__ __forceinline__ uint64_t tm_two(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void tm_split(uint64_t v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v)); }
__device__ __forceinline__ uint64_t tm_fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ uint64_t tm_mul2(uint64_t a, uint64_t b) {
  uint64_t r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
__device__ __forceinline__ void cap_scores(float (&s)[2][4], const CapArgs& c) {
  const uint64_t mul = tm_two(c.mul, c.mul);
  uint64_t x[4];
  float most = 0.f;
#pragma unroll
  for (int p = 0; p < 4; ++p) {
    x[p] = tm_mul2(tm_two(s[p >> 1][(p & 1) * 2], s[p >> 1][(p & 1) * 2 + 1]), mul);
    float x0, x1;
    tm_split(x[p], x0, x1);
    most = fmaxf(most, fmaxf(fabsf(x0), fabsf(x1)));
    s[p >> 1][(p & 1) * 2] = x0;
    s[p >> 1][(p & 1) * 2 + 1] = x1;
  }
  if (!c.capped) return;
  if (__any_sync(0xffffffffu, !(most <= 0.35f))) {
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[n][e] = c.cap2 * tanhf(s[n][e]);
    return;
  }
  const uint64_t cap2 = tm_two(c.cap2, c.cap2);
  const uint64_t c11 = tm_two(-1382.f / 155925.f, -1382.f / 155925.f), c9 = tm_two(62.f / 2835.f, 62.f / 2835.f),
                 c7 = tm_two(-17.f / 315.f, -17.f / 315.f), c5 = tm_two(2.f / 15.f, 2.f / 15.f), c3 = tm_two(-1.f / 3.f, -1.f / 3.f);
#pragma unroll
  for (int p = 0; p < 4; ++p) {
    const uint64_t u = tm_mul2(x[p], x[p]), y = tm_mul2(x[p], cap2);
    uint64_t q = tm_fma2(u, c11, c9);
    q = tm_fma2(u, q, c7);
    q = tm_fma2(u, q, c5);
    q = tm_fma2(u, q, c3);
    tm_split(tm_fma2(tm_mul2(y, u), q, y), s[p >> 1][(p & 1) * 2], s[p >> 1][(p & 1) * 2 + 1]);
  }
}

// --------------------------------------------------- maxima and sums of prompt portions
// The first visit needs one head at a time, so it runs on tiles of 64 queries (a warp 16 of them) that share every key
// tile of 64, a quarter of the key traffic of the tiles of 16 below. part_ml[token, head] receives the row's maximum
// (0 where capped scores are summed as they are) and its sum, in base-2 units.
constexpr int TS_ROWS = 64, TS_KEYS = 64, TS_THREADS = 128;

template <int KD>
__global__ void __launch_bounds__(TS_THREADS) talking_stats_kernel(TalkArgs a) {
  extern __shared__ __align__(16) unsigned char raw_stats[];
  __shared__ int rows[4][TS_KEYS];
  constexpr int KS = KD * 16 + 8;                          // padded row stride
  const int H = a.num_heads, D = a.head_dim;
  bf16* Ks = (bf16*)raw_stats;                             // [2][KEYS][KS]
  pdl_trigger();
  pdl_wait();
  const int seq = blockIdx.y, head = blockIdx.z, kvh = head / (H / a.num_kv_heads);
  const int row0 = a.cu_q[seq], n = a.cu_q[seq + 1] - row0;
  const int q0 = blockIdx.x * TS_ROWS;
  if (q0 >= n) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int first_pos = a.ctx_lens[seq] - n + q0, nq = min(TS_ROWS, n - q0), last_pos = first_pos + nq - 1;
  const int lo = a.window > 0 ? max(0, first_pos - a.window + 1) : 0;
  const int tiles = (last_pos + 1 - lo + TS_KEYS - 1) / TS_KEYS;
  const int* table = a.block_tables + (size_t)seq * a.table_width;
  const bf16* kc = (const bf16*)a.k_cache;
  const int r = warp * 16 + (lane >> 2), c2 = (lane & 3) * 2;
  uint32_t qf[KD][4];
#pragma unroll
  for (int kk = 0; kk < KD; ++kk)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int row = r + (j & 1) * 8, col = kk * 16 + c2 + (j >> 1) * 8;
      qf[kk][j] = 0u;
      if (row < nq && kk * 16 < D)
        qf[kk][j] = *reinterpret_cast<const uint32_t*>((const bf16*)a.q + ((size_t)(row0 + q0 + row) * H + head) * D + col);
    }
  // a thread copies its 16-byte piece of one key after the other; the keys' cache rows are looked up a tile ahead
  const int pieces = D >> 3, step = TS_THREADS / pieces, line0 = tid / pieces < step ? tid / pieces : TS_KEYS, ch = (tid % pieces) * 8;
  auto find = [&](int t) {
    const int kpos = lo + t * TS_KEYS + tid;
    if (tid < TS_KEYS) rows[t & 3][tid] = t < tiles && kpos <= last_pos ? (int)talk_row(table, kpos, kvh, a) : -1;
  };
  auto load = [&](int t) {
    if (t < tiles) {
      uint32_t to = tm_smem(Ks + ((size_t)(t & 1) * TS_KEYS + line0) * KS + ch);
      for (int line = line0; line < TS_KEYS; line += step, to += (uint32_t)(step * KS * 2)) {
        const int row = rows[t & 3][line];
        const bf16* from = kc + (size_t)(row < 0 ? 0 : row) * D + ch;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(to), "l"(from), "r"(row < 0 ? 0 : 16) : "memory");
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  CapArgs cap;
  cap.capped = a.softcap > 0.f;
  cap.mul = cap.capped ? a.scale / a.softcap : a.scale * TM_LOG2E;
  cap.cap2 = a.softcap * TM_LOG2E;
  const bool bounded = cap.capped && cap.cap2 <= 64.f;
  float m[2] = {bounded ? 0.f : -INFINITY, bounded ? 0.f : -INFINITY}, l[2] = {0.f, 0.f};
  for (int t = 0; t < 2; ++t) find(t);
  __syncthreads();
  load(0);
  for (int t = 0; t < tiles; ++t) {
    tm_wait<0>();
    __syncthreads();                                       // tile t has arrived, and nobody reads the other buffer any more
    load(t + 1);
    find(t + 2);
    const uint32_t kb = tm_smem(Ks) + (uint32_t)((((t & 1) * TS_KEYS + (lane & 7) + ((lane >> 4) << 3)) * KS + ((lane >> 3) & 1) * 8) * 2);
#pragma unroll
    for (int part = 0; part < TS_KEYS / 32; ++part) {
      const int k0 = lo + t * TS_KEYS + part * 32;
      // no row of this warp sees any of these keys
      if (k0 > first_pos + warp * 16 + 15 || (a.window > 0 && k0 + 31 <= first_pos + warp * 16 - a.window)) continue;
      float s[2][2][4];                                    // two blocks of 16 keys: four independent chains of products
#pragma unroll
      for (int i = 0; i < 16; ++i) s[i >> 3][(i >> 2) & 1][i & 3] = 0.f;
#pragma unroll
      for (int kk = 0; kk < KD; ++kk) {
        if (kk * 16 < D) {
          uint32_t b[2][4];
#pragma unroll
          for (int x = 0; x < 2; ++x) tm_ldm(b[x], kb + (uint32_t)((part * 2 + x) * 16 * KS * 2) + kk * 32);
#pragma unroll
          for (int x = 0; x < 2; ++x) {
            tm_mma(s[x][0], qf[kk], b[x][0], b[x][1]);
            tm_mma(s[x][1], qf[kk], b[x][2], b[x][3]);
          }
        }
      }
      cap_scores(s[0], cap);
      cap_scores(s[1], cap);
      if (!(k0 + 31 <= first_pos + warp * 16 && (a.window <= 0 || k0 > first_pos + warp * 16 + 15 - a.window))) {
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const int kpos = k0 + (i >> 3) * 16 + ((i >> 2) & 1) * 8 + c2 + (i & 1), qpos = first_pos + r + ((i >> 1) & 1) * 8;
          if (!(kpos <= qpos && (a.window <= 0 || kpos > qpos - a.window))) s[i >> 3][(i >> 2) & 1][i & 3] = -INFINITY;
        }
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float mn = m[half];
        if (!bounded) {
          float mx = -INFINITY;
#pragma unroll
          for (int i = 0; i < 8; ++i) mx = fmaxf(mx, s[i >> 2][(i >> 1) & 1][half * 2 + (i & 1)]);
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
          mn = fmaxf(m[half], mx);
          if (mn == -INFINITY) continue;
          l[half] *= tm_ex2(m[half] - mn);
          m[half] = mn;
        }
#pragma unroll
        for (int x = 0; x < 2; ++x)
          l[half] += (tm_ex2(s[x][0][half * 2] - mn) + tm_ex2(s[x][0][half * 2 + 1] - mn)) + (tm_ex2(s[x][1][half * 2] - mn) + tm_ex2(s[x][1][half * 2 + 1] - mn));
      }
    }
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    l[half] += __shfl_xor_sync(0xffffffffu, l[half], 1);
    l[half] += __shfl_xor_sync(0xffffffffu, l[half], 2);
    const int row = r + half * 8;
    if (row < nq && (lane & 3) == 0) {
      float* ml = a.part_ml + ((size_t)(row0 + q0 + row) * H + head) * 2;
      ml[0] = m[half];
      ml[1] = l[half];
    }
  }
}

// ------------------------------------------------------------------ the mixing kernel
constexpr int TM_MAX_COUNTERS = 1 << 14;
static __device__ unsigned int g_talk_counters[TM_MAX_COUNTERS];     // arrivals of a request's key ranges; zero between launches

struct TalkMmaShape {
  int heads_per_cta;       // <= 16: a warp each
  int kv_per_cta;          // key/value heads a CTA's heads read, at most
  int padded_heads;        // all heads, rounded up to 16
};

template <int KD, int KV, int CL, bool TMA>
__global__ void __launch_bounds__(512) talking_mma_kernel(TalkArgs a, TalkMmaShape sh, int phase, const __grid_constant__ CUtensorMap map_k,
                                                          const __grid_constant__ CUtensorMap map_v, int* error_flag) {
  extern __shared__ __align__(16) unsigned char raw_smem[];
  unsigned char* raw = TMA ? (unsigned char*)(((uintptr_t)raw_smem + 1023) & ~(uintptr_t)1023) : raw_smem;
  const int H = a.num_heads, G = a.num_kv_heads, per = H / G, D = TMA ? KD * 16 : a.head_dim, DV = TMA ? KV * 16 : a.v_head_dim;
  const int KS = TMA ? D : D + 8, VS = TMA ? DV : DV + 8;  // padded row strides (TMA: boxes of 64 columns one after the other)
  const int Hp = sh.padded_heads;
  const size_t k_elems = (size_t)sh.kv_per_cta * TM_KEYS * KS, v_elems = (size_t)sh.kv_per_cta * TM_KEYS * VS;
  bf16* Ks = (bf16*)raw;                                   // [2][kv][KEYS][KS]
  bf16* Vs = Ks + 2 * k_elems;                             // [2][kv][KEYS][VS]
  bf16* Ps = Vs + 2 * v_elems;                             // [2 parts][Hp][TM_POS]
  bf16* Ws = Ps + (size_t)2 * Hp * TM_POS;                 // [16][TM_POS]
  bf16* Tm = Ws + (size_t)16 * TM_POS;                     // [16][Hp + 8]
  __shared__ int key_rows[4][TM_KEYS];
  __shared__ int tile_rows[2 * TM_AHEAD];                  // TMA: the cache row of each tile's first key, TM_AHEAD tiles at a time
  __shared__ __align__(8) uint64_t bars[4];                // TMA: keys of even and odd tiles, values of even and odd tiles

  pdl_trigger();
  pdl_wait();
  const int rank = CL == 1 ? 0 : (int)(blockIdx.x % CL);
  const int seq = blockIdx.y;
  const int row0 = a.cu_q[seq], n = a.cu_q[seq + 1] - row0;
  const int q0 = (int)(blockIdx.x / CL) * TM_ROWS;
  if (q0 >= n) return;                                     // the same for every CTA of a cluster
  const int ctx = a.ctx_lens[seq];
  const int first_pos = ctx - n + q0;
  const int nq = min(TM_ROWS, n - q0);
  const int last_pos = first_pos + nq - 1;
  int lo = a.window > 0 ? max(0, first_pos - a.window + 1) : 0;
  if (TMA) lo &= ~(TM_KEYS - 1);                           // a tile does not cross a page
  const int all_tiles = (last_pos + 1 - lo + TM_KEYS - 1) / TM_KEYS;
  const int each = (all_tiles + a.num_splits - 1) / a.num_splits;
  const int k_begin = lo + (int)blockIdx.z * each * TM_KEYS;
  const int k_end = min(last_pos + 1, k_begin + each * TM_KEYS);
  const int tiles = max(0, (k_end - k_begin + TM_KEYS - 1) / TM_KEYS);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, threads = blockDim.x;
  const int head0 = rank * sh.heads_per_cta, my_heads = min(sh.heads_per_cta, H - head0);
  const int kv0 = head0 / per, my_kv = my_heads > 0 ? (head0 + my_heads - 1) / per - kv0 + 1 : 0;
  const int head = head0 + warp;
  const bool has_head = warp < my_heads;
  const int my_g = has_head ? head / per - kv0 : 0;
  const int* table = a.block_tables + (size_t)seq * a.table_width;
  const bf16* kc = (const bf16*)a.k_cache;
  const bf16* vc = (const bf16*)a.v_cache;
  const int r = lane >> 2, c2 = (lane & 3) * 2;            // this lane's rows r, r + 8 and columns c2, c2 + 1 of a fragment

  // this warp's queries as A fragments
  uint32_t qf[KD][4];
#pragma unroll
  for (int kk = 0; kk < KD; ++kk)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int row = r + (j & 1) * 8, col = kk * 16 + c2 + (j >> 1) * 8;
      qf[kk][j] = 0u;
      if (has_head && row < nq && kk * 16 < D)
        qf[kk][j] = *reinterpret_cast<const uint32_t*>((const bf16*)a.q + ((size_t)(row0 + q0 + row) * H + head) * D + col);
    }
  if (phase != TM_STATS) {
    for (int idx = tid; idx < 16 * Hp; idx += threads) {
      const int h = idx / Hp, g = idx - h * Hp;
      float t = 0.f;
      if (head0 + h < H && h < my_heads && g < H) t = a.talk ? a.talk[(size_t)(head0 + h) * H + g] : (g == head0 + h ? 1.f : 0.f);
      Tm[h * (Hp + 8) + g] = __float2bfloat16_rn(t);
    }
    // rows of P of no head (H not a multiple of 16) stay zero
    for (int idx = tid; idx < 2 * (Hp - H) * TM_POS; idx += threads) {
      const int part = idx / ((Hp - H) * TM_POS), rest = idx - part * (Hp - H) * TM_POS;
      Ps[((size_t)part * Hp + H) * TM_POS + rest] = __float2bfloat16_rn(0.f);
    }
  }
  auto find_tiles = [&](int t) {                           // TMA: the first cache rows of tiles t .. t + TM_AHEAD - 1, in units of kv head 0
    for (int i = tid; i < TM_AHEAD; i += threads)
      if (t + i < tiles) tile_rows[(t + i) & (2 * TM_AHEAD - 1)] = (int)talk_row(table, k_begin + (t + i) * TM_KEYS, 0, a);
  };
  auto find_rows = [&](int t) {                            // the cache rows of tile t (-1: no such key), in units of kv head 0
    if (tid < TM_KEYS) {
      const int kpos = k_begin + t * TM_KEYS + tid;
      key_rows[t & 3][tid] = t < tiles && kpos < k_end ? (int)talk_row(table, kpos, 0, a) : -1;
    }
  };
  // A tile's keys (or values): a line is one key of one head, `width` elements; a thread keeps its 16-byte piece of
  // a line and goes from line to line. Lines of no key are zeroed.
  const int k_pieces = D >> 3, v_pieces = DV >> 3, lines = my_kv * TM_KEYS;
  const int k_step = threads / k_pieces, v_step = threads / v_pieces;
  const int k_line = tid / k_pieces < k_step ? tid / k_pieces : lines, k_ch = (tid % k_pieces) * 8;
  const int v_line = tid / v_pieces < v_step ? tid / v_pieces : lines, v_ch = (tid % v_pieces) * 8;
  auto load_lines = [&](bf16* dst, const bf16* src, int t, int width, int stride, int line0, int step, int ch) {
    const int* rows = key_rows[t & 3];
    uint32_t to = tm_smem(dst) + (uint32_t)((line0 * stride + ch) * 2);
    const uint32_t to_step = (uint32_t)(step * stride * 2);
    const bf16* base = src + (size_t)kv0 * a.page_size * width + ch;
#pragma unroll 4
    for (int line = line0; line < lines; line += step, to += to_step) {
      const int row = rows[line & (TM_KEYS - 1)];
      const bf16* from = base + (size_t)(row < 0 ? 0 : row + (line / TM_KEYS) * a.page_size) * width;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(to), "l"(from), "r"(row < 0 ? 0 : 16) : "memory");
    }
  };
  const int warps = threads >> 5;
  uint32_t phases = 0;                                     // bit b: the parity barrier b is waited for next
  bool failed = false;
  auto arrived = [&](int b) {
    const uint32_t addr = tm_smem(&bars[b]), parity = (phases >> b) & 1u;
    if (!failed && !tm_try(addr, parity)) failed = !bounded_mbar_wait(addr, parity);
    phases ^= 1u << b;
    __syncwarp();
  };
  auto give_up = [&]() {                                   // a wait ran out: say so, and give the copies in flight the same time again
    if (!failed) return;
    atomicExch(error_flag, WAIT_FAILED_TALKING);
    if (tid == 0)
      for (int b = 0; b < 4; ++b) bounded_mbar_wait(tm_smem(&bars[b]), (phases >> b) & 1u);
  };
  // The same by the TMA unit (KD == KV): a box holds 64 columns of the tile's rows of kv_per_cta heads (heads beyond this
  // CTA's own are fetched and not read); the warps take turns in asking.
  const int boxes = sh.kv_per_cta;
  const bool lost = TMA && wait_test_unarmed();
  auto copy_boxes = [&](bf16* dst, const CUtensorMap* map, uint64_t* bar, int t) {
    if (lane == 0 && warp == t % warps) {
      tm_arm(bar, (uint32_t)(boxes * (KD / 4) * TM_BOX * 2));
      const int row = tile_rows[t & (2 * TM_AHEAD - 1)];
      const int z = a.page_shift >= 0 ? row >> a.page_shift : row / a.page_size;
#pragma unroll
      for (int part = 0; part < KD / 4; ++part)
        tm_tensor(dst + (size_t)part * boxes * TM_BOX, map, part * 64, row - z * a.page_size, z + min(kv0, G - 1), bar);
    }
  };
  auto copy_tiles = [&](int tk, int tv) {
    if (lost) return;
    if (tk >= 0 && tk < tiles) copy_boxes(Ks + (size_t)(tk & 1) * k_elems, &map_k, &bars[tk & 1], tk);
    if (tv >= 0 && tv < tiles) copy_boxes(Vs + (size_t)(tv & 1) * v_elems, &map_v, &bars[2 + (tv & 1)], tv);
  };
  auto load_tiles = [&](int tk, int tv) {                  // one group: keys of tile tk and values of tile tv (none outside 0 .. tiles - 1)
    if (tk >= 0 && tk < tiles) load_lines(Ks + (size_t)(tk & 1) * k_elems, kc, tk, D, KS, k_line, k_step, k_ch);
    if (tv >= 0 && tv < tiles) load_lines(Vs + (size_t)(tv & 1) * v_elems, vc, tv, DV, VS, v_line, v_step, v_ch);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  CapArgs cap;
  cap.capped = a.softcap > 0.f;
  cap.mul = cap.capped ? a.scale / a.softcap : a.scale * TM_LOG2E;
  cap.cap2 = a.softcap * TM_LOG2E;

  // This lane's places in the shared arrays (ldmatrix rows, fragment positions). A swizzled box: a row is 128 bytes, its
  // 16-byte pieces permuted by the row's low three bits; piece 2 k + h of row x lies at (h ^ x) ^ 2 k.
  const int krow = (lane & 7) + ((lane >> 4) << 3), khalf = (lane >> 3) & 1, vrow = (lane & 7) + ((lane >> 3) & 1) * 8, vhalf = lane >> 4;
  const uint32_t part_bytes = (uint32_t)(boxes * TM_BOX * 2);          // from 64 columns of all heads to the next 64
  const uint32_t s_k = tm_smem(Ks) + (uint32_t)(my_g * TM_KEYS * (TMA ? 64 : KS) * 2) + (uint32_t)(TMA ? krow * 128 + ((khalf ^ (lane & 7)) << 4) : (krow * KS + khalf * 8) * 2);
  const uint32_t s_v = tm_smem(Vs) + (uint32_t)(my_g * TM_KEYS * (TMA ? 64 : VS) * 2) + (uint32_t)(TMA ? vrow * 128 + ((vhalf ^ (lane & 7)) << 4) : (vrow * VS + vhalf * 8) * 2);
  const uint32_t s_p = tm_smem(Ps), s_w = tm_smem(Ws), k_stage = (uint32_t)(k_elems * 2), v_stage = (uint32_t)(v_elems * 2), rest = (uint32_t)(Hp * TM_POS * 2);
  const uint32_t s_p_out = s_p + (uint32_t)((head * TM_POS + r * TM_ROWP + c2) * 2);
  const uint32_t s_p_mix = s_p + (uint32_t)((((lane & 7) + ((lane >> 3) & 1) * 8) * TM_POS + (lane >> 4) * 8) * 2);
  const uint32_t s_t_mix = tm_smem(Tm) + (uint32_t)(((lane & 15) * (Hp + 8) + (lane >> 4) * 8) * 2);
  const uint32_t s_w_out = s_w + (uint32_t)((r * TM_POS + c2) * 2), s_w_in = s_w + (uint32_t)((warp * TM_POS + (lane & 15) * TM_ROWP + (lane >> 4) * 8) * 2);

  // the scores of this warp's head for tile t, in base-2 units, minus infinity where a row does not see the key
  auto scores = [&](float (&s)[2][4], int t) {
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[j][e] = 0.f;
    const uint32_t kb = s_k + (t & 1 ? k_stage : 0u);
#pragma unroll
    for (int kk = 0; kk < KD; ++kk) {
      if (kk * 16 < D) {
        uint32_t b[4];
        tm_ldm(b, TMA ? (kb ^ (uint32_t)((kk & 3) << 5)) + (kk >> 2) * part_bytes : kb + kk * 32);
        tm_mma(s[0], qf[kk], b[0], b[1]);
        tm_mma(s[1], qf[kk], b[2], b[3]);
      }
    }
    cap_scores(s, cap);
    const int k0 = k_begin + t * TM_KEYS;
    // the whole tile is seen by every row: no mask
    if (k0 + TM_KEYS - 1 <= first_pos && k0 + TM_KEYS <= k_end && (a.window <= 0 || k0 > last_pos - a.window)) return;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int kpos = k0 + j * 8 + c2 + (e & 1), qpos = first_pos + r + (e >> 1) * 8;
        if (!(kpos < k_end && kpos <= qpos && (a.window <= 0 || kpos > qpos - a.window))) s[j][e] = -INFINITY;
      }
  };

  // Capped scores cannot leave +-cap: their exponentials are summed as they are, without a running maximum.
  const bool bounded = cap.capped && cap.cap2 <= 64.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  if (bounded && phase != TM_VALUES) m[0] = m[1] = 0.f;
  if (TMA) {
    find_tiles(0);
  } else {
    for (int t = 0; t < 3; ++t) find_rows(t);
  }
  if (TMA && tid == 0) {
    for (int b = 0; b < 4; ++b) asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(tm_smem(&bars[b])));
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  __syncthreads();
  if (phase != TM_VALUES) {
    if (TMA) {
      copy_tiles(0, -1);
      copy_tiles(1, -1);
    } else {
      load_tiles(0, -1);
    }
    for (int t = 0; t < tiles; ++t) {
      if (TMA) {
        arrived(t & 1);
      } else {
        tm_wait<0>();
        __syncthreads();                                   // tile t has arrived, and nobody reads the other buffer any more
        load_tiles(t + 1, -1);
        find_rows(t + 3);
      }
      if (has_head) {
        float s[2][4];
        scores(s, t);
        if (bounded) {
#pragma unroll
          for (int half = 0; half < 2; ++half)
            l[half] += (tm_ex2(s[0][half * 2]) + tm_ex2(s[0][half * 2 + 1])) + (tm_ex2(s[1][half * 2]) + tm_ex2(s[1][half * 2 + 1]));
        } else {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          float mx = fmaxf(fmaxf(s[0][half * 2], s[0][half * 2 + 1]), fmaxf(s[1][half * 2], s[1][half * 2 + 1]));
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
          const float mn = fmaxf(m[half], mx);
          if (mn != -INFINITY) {
            float sum = 0.f;
#pragma unroll
            for (int j = 0; j < 2; ++j) sum += tm_ex2(s[j][half * 2] - mn) + tm_ex2(s[j][half * 2 + 1] - mn);
            l[half] = l[half] * tm_ex2(m[half] - mn) + sum;
            m[half] = mn;
          }
        }
        }
      }
      if (TMA) {
        __syncthreads();                                   // nobody reads this tile's buffer any more
        copy_tiles(t + 2, -1);
        if (((t + 8) & (TM_AHEAD - 1)) == 0) find_tiles(t + 8);      // well before the first of them is asked for
      }
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      l[half] += __shfl_xor_sync(0xffffffffu, l[half], 1);
      l[half] += __shfl_xor_sync(0xffffffffu, l[half], 2);
    }
    if (phase == TM_STATS) {
      if (has_head && (lane & 3) == 0)
#pragma unroll
        for (int half = 0; half < 2; ++half)
          if (r + half * 8 < nq) {
            float* ml = a.part_ml + (((size_t)(row0 + q0 + r + half * 8) * H + head) * a.num_splits + blockIdx.z) * 2;
            ml[0] = m[half];
            ml[1] = l[half];
          }
      give_up();
      return;
    }
  } else if (has_head) {
#pragma unroll
    for (int half = 0; half < 2; ++half)
      if (r + half * 8 < nq) {
        const float* ml = a.part_ml + ((size_t)(row0 + q0 + r + half * 8) * H + head) * a.num_splits * 2;
        for (int s = 0; s < a.num_splits; ++s) m[half] = fmaxf(m[half], ml[2 * s]);
        for (int s = 0; s < a.num_splits; ++s)
          if (ml[2 * s] != -INFINITY) l[half] += ml[2 * s + 1] * tm_ex2(ml[2 * s] - m[half]);
      }
  }
  // the logarithm of each row's denominator; rows that see nothing (none that is stored) get weights of zero
  float lse[2];
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    if (a.sinks && has_head) {
      const float sink = a.sinks[head] * TM_LOG2E, top = fmaxf(m[half], sink);
      l[half] = (m[half] == -INFINITY ? 0.f : l[half] * tm_ex2(m[half] - top)) + tm_ex2(sink - top);
      m[half] = top;
    }
    lse[half] = l[half] > 0.f ? m[half] + log2f(l[half]) : INFINITY;
  }

  float o[KV * 2][4];
#pragma unroll
  for (int j = 0; j < KV * 2; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
  __syncthreads();
  if (TMA) {
    if (tiles > TM_AHEAD) find_tiles(0);                   // unless they are all still there
  } else {
    for (int t = 0; t < 3; ++t) find_rows(t);
  }
  tm_sync<CL>();                                           // every CTA of the cluster is here before the first remote store
  if (TMA) {
    copy_tiles(0, 0);
    copy_tiles(1, -1);
  } else {
    load_tiles(0, -1);
    load_tiles(1, 0);
    tm_wait<1>();
    __syncthreads();                                       // the first keys have arrived
  }
  for (int t = 0; t < tiles; ++t) {
    if (TMA) arrived(t & 1);
    if (has_head) {
      float s[2][4];
      scores(s, t);
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const uint32_t at = s_p_out + half * (8 * TM_ROWP * 2);
#pragma unroll
        for (int j = 0; j < 2; ++j) {
          const float p0 = tm_ex2(s[j][half * 2] - lse[half]), p1 = tm_ex2(s[j][half * 2 + 1] - lse[half]);
          const uint32_t hi = tm_pack(p0, p1);
          const uint32_t rem = tm_pack(p0 - __uint_as_float(hi << 16), p1 - __uint_as_float(hi & 0xffff0000u));
          tm_store_all<CL>(at + j * 16, hi);
          tm_store_all<CL>(at + j * 16 + rest, rem);
        }
      }
    }
    tm_sync<CL>();                                         // all weights are there; keys of tile t and values of t - 1 are done with
    if (TMA) {
      copy_tiles(t + 2, t + 1);
      if (((t + 8) & (TM_AHEAD - 1)) == 0) find_tiles(t + 8);
    } else {
      load_tiles(t + 2, t + 1);
      find_rows(t + 3);
    }
    // mixed weights of this CTA's heads: a query row of the tile per turn
    for (int i = warp; i < TM_ROWS; i += warps) {
      float w[2][4];
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) w[j][e] = 0.f;
      for (int g0 = 0; g0 < Hp; g0 += 16) {
        uint32_t tf[4], b[4];
        tm_ldm(tf, s_t_mix + g0 * 2);
        const uint32_t pb = s_p_mix + g0 * (TM_POS * 2) + i * (TM_ROWP * 2);
        tm_ldm_t(b, pb);
        tm_mma(w[0], tf, b[0], b[1]);
        tm_mma(w[1], tf, b[2], b[3]);
        tm_ldm_t(b, pb + rest);
        tm_mma(w[0], tf, b[0], b[1]);
        tm_mma(w[1], tf, b[2], b[3]);
      }
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const uint32_t at = s_w_out + i * (TM_ROWP * 2) + j * 16;
        tm_store_all<1>(at, tm_pack(w[j][0], w[j][1]));
        tm_store_all<1>(at + 8 * TM_POS * 2, tm_pack(w[j][2], w[j][3]));
      }
    }
    if (TMA) {
      arrived(2 + (t & 1));
      const int live = k_end - k_begin - t * TM_KEYS;      // rows from here on hold whatever the page held: their weights are zero, but a
      if (live < TM_KEYS) {                                // number that is none would stay one
        const int per_box = (TM_KEYS - live) * 8;          // 16-byte pieces of the dead rows of a box
        for (int idx = tid; idx < boxes * (KV / 4) * per_box; idx += threads) {
          const int box = idx / per_box, rest = idx - box * per_box;
          *reinterpret_cast<uint4*>(Vs + (size_t)(t & 1) * v_elems + (size_t)box * TM_BOX + live * 64 + rest * 8) = make_uint4(0u, 0u, 0u, 0u);
        }
      }
    } else {
      tm_wait<1>();                                        // keys of tile t + 1 and values of tile t
    }
    tm_sync<CL>();
    if (has_head) {
      uint32_t wf[4];
      tm_ldm(wf, s_w_in);
      const uint32_t vb = s_v + (t & 1 ? v_stage : 0u);
#pragma unroll
      for (int j = 0; j < KV; ++j) {
        if (j * 16 < DV) {
          uint32_t b[4];
          tm_ldm_t(b, TMA ? (vb ^ (uint32_t)((j & 3) << 5)) + (j >> 2) * part_bytes : vb + j * 32);
          tm_mma(o[2 * j], wf, b[0], b[1]);
          tm_mma(o[2 * j + 1], wf, b[2], b[3]);
        }
      }
    }
  }
  if (has_head) {
#pragma unroll
    for (int j = 0; j < KV * 2; ++j) {
      if (j * 8 < DV) {
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int row = r + half * 8;
          if (row < nq) {
            const size_t t = (size_t)(row0 + q0 + row);
            const int col = head * DV + j * 8 + c2;
            if (a.num_splits == 1)
              *reinterpret_cast<uint32_t*>((bf16*)a.out + t * H * DV + col) = tm_pack(o[j][half * 2], o[j][half * 2 + 1]);
            else
              *reinterpret_cast<float2*>(a.part_out + (t * a.num_splits + blockIdx.z) * H * DV + col) =
                  make_float2(o[j][half * 2], o[j][half * 2 + 1]);
          }
        }
      }
    }
  }
  give_up();
  if (a.num_splits == 1) return;
  // the CTA of a request's last range to arrive adds the ranges' outputs up, in order, for the heads it owns
  __shared__ int last;
  if (!cta_arrives_last(&g_talk_counters[(size_t)seq * CL + rank], (unsigned int)a.num_splits, &last)) return;
  const int width = my_heads * DV;
  for (int idx = tid; idx < nq * width; idx += threads) {
    const int row = idx / width, col = head0 * DV + idx - row * width;
    const float* part = a.part_out + (size_t)(row0 + q0 + row) * a.num_splits * H * DV + col;
    float sum = 0.f;
    for (int s = 0; s < a.num_splits; ++s) sum += __ldcg(part + (size_t)s * H * DV);
    ((bf16*)a.out)[(size_t)(row0 + q0 + row) * H * DV + col] = __float2bfloat16_rn(sum);
  }
}

// How a cluster shares the heads: as few CTAs as hold 16 heads each and whose keys and values fit in shared memory.
static bool talk_mma_shape(int H, int G, int D, int DV, bool tma, TalkMmaShape& sh, int& cluster, size_t& smem) {
  constexpr size_t LIMIT = 226 * 1024;
  const int per = H / G;
  sh.padded_heads = (H + 15) / 16 * 16;
  if (sh.padded_heads > 64) return false;
  for (cluster = 1; cluster <= 4; cluster *= 2) {
    const int hc = (H + cluster - 1) / cluster;
    if (hc > 16) continue;
    int kv = 0;
    for (int c = 0; c < cluster; ++c) {
      const int h0 = c * hc, hn = H - h0 < hc ? H - h0 : hc;
      if (hn > 0 && (h0 + hn - 1) / per - h0 / per + 1 > kv) kv = (h0 + hn - 1) / per - h0 / per + 1;
    }
    sh.heads_per_cta = hc;
    sh.kv_per_cta = kv;
    smem = (tma ? 1024 : 0) + sizeof(bf16) * (2 * (size_t)kv * TM_KEYS * (tma ? D + DV : D + 8 + DV + 8) + (size_t)2 * sh.padded_heads * TM_POS + (size_t)16 * TM_POS +
                           (size_t)16 * (sh.padded_heads + 8));
    if (smem <= LIMIT) return true;
  }
  return false;
}

struct TalkMaps { CUtensorMap k, v; int* error_flag; };

template <int KD, int KV, int CL, bool TMA>
static int launch_talk_mma(const TalkArgs& a, const TalkMmaShape& sh, size_t smem, int num_seqs, int max_query_len, int phase,
                           const TalkMaps& maps, cudaStream_t stream) {
  auto kern = talking_mma_kernel<KD, KV, CL, TMA>;
  static size_t allowed = 0;
  if (smem > 48 * 1024 && smem > allowed) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    allowed = smem;
  }
  const dim3 grid((unsigned)((max_query_len + TM_ROWS - 1) / TM_ROWS * CL), num_seqs, a.num_splits);
  const int threads = sh.heads_per_cta * 32;
  if constexpr (CL == 1) return launch(kern, grid, threads, smem, stream, a, sh, phase, maps.k, maps.v, maps.error_flag);
  else return launch_cluster(kern, grid, dim3(threads), smem, stream, dim3(CL, 1, 1), a, sh, phase, maps.k, maps.v, maps.error_flag);
}

template <int KD, int KV, bool TMA>
static int launch_talk_mma_cl(const TalkArgs& a, const TalkMmaShape& sh, int cluster, size_t smem, int num_seqs, int max_query_len,
                              int phase, const TalkMaps& maps, cudaStream_t stream) {
  if (cluster == 1) return launch_talk_mma<KD, KV, 1, TMA>(a, sh, smem, num_seqs, max_query_len, phase, maps, stream);
  if (cluster == 2) return launch_talk_mma<KD, KV, 2, TMA>(a, sh, smem, num_seqs, max_query_len, phase, maps, stream);
  return launch_talk_mma<KD, KV, 4, TMA>(a, sh, smem, num_seqs, max_query_len, phase, maps, stream);
}

}  // namespace ts

using namespace ts;

extern "C" int ts_talking_attention_mma_takes(int heads, int kv_heads, int d, int dv) {
  TalkMmaShape sh;
  int cluster;
  size_t smem;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || d <= 0 || dv <= 0 || d % 16 || dv % 16 || d > 128 || dv > 128) return 0;
  return talk_mma_shape(heads, kv_heads, d, dv, false, sh, cluster, smem) ? cluster : 0;
}

// As ts_talking_attention, bf16 only; num_splits > 1 for steps of single tokens only; with num_splits 1 and part_ml
// [T, heads, 2] the maxima and sums are made by a kernel of their own (prompt portions). cache_rows = pages * kv_heads * page_size must stay below 2^31. talk is used as bf16.
extern "C" int ts_talking_attention_mma(const void* q, void* out, const void* k_cache, const void* v_cache, const int* block_tables,
                                        int table_width, const int* cu_q, const int* ctx_lens, int num_seqs, int max_query_len,
                                        int num_tokens, int heads, int kv_heads, int d, int dv, int page_size, float scale,
                                        int window, float softcap, const float* talk, const float* sinks, int num_splits,
                                        float* part_ml, float* part_out, long long cache_rows, int* error_flag,
                                        cudaStream_t stream) {
  if (num_seqs <= 0 || num_tokens <= 0) return 0;
  if (!error_flag || cache_rows <= 0 || cache_rows >= (1ll << 31)) return TS_ERR_BAD_ARGUMENT;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads || page_size <= 0 || max_query_len <= 0 || window < 0) return TS_ERR_BAD_ARGUMENT;
  if (num_splits < 1 || (num_splits > 1 && (!part_ml || !part_out || max_query_len != 1))) return TS_ERR_BAD_ARGUMENT;
  if (num_splits > 1 && (long long)num_seqs * 4 > TM_MAX_COUNTERS) return TS_ERR_UNSUPPORTED;
  if (((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)out) & 15) return TS_ERR_UNSUPPORTED;
  TalkMmaShape sh;
  int cluster;
  size_t smem;
  TalkMaps maps = {};
  maps.error_flag = error_flag;
  bool tma = d == dv && (d == 64 || d == 128) && page_size % TM_KEYS == 0;
  if (tma) {
    tma = talk_mma_shape(heads, kv_heads, d, dv, true, sh, cluster, smem);
    const CUtensorMap* mk = tma ? cache_heads_map(k_cache, cache_rows / page_size, page_size, d, TM_KEYS, sh.kv_per_cta) : nullptr;
    const CUtensorMap* mv = tma ? cache_heads_map(v_cache, cache_rows / page_size, page_size, dv, TM_KEYS, sh.kv_per_cta) : nullptr;
    tma = mk && mv;
    if (tma) { maps.k = *mk; maps.v = *mv; }
  }
  if (!ts_talking_attention_mma_takes(heads, kv_heads, d, dv) || !talk_mma_shape(heads, kv_heads, d, dv, tma, sh, cluster, smem))
    return TS_ERR_UNSUPPORTED;
  TalkArgs a;
  a.q = q; a.out = out; a.k_cache = k_cache; a.v_cache = v_cache; a.block_tables = block_tables; a.table_width = table_width;
  a.cu_q = cu_q; a.ctx_lens = ctx_lens; a.num_heads = heads; a.num_kv_heads = kv_heads; a.head_dim = d; a.v_head_dim = dv;
  a.page_size = page_size; a.page_shift = page_shift_of(page_size); a.scale = scale; a.window = window; a.softcap = softcap;
  a.talk = talk; a.sinks = sinks; a.num_splits = num_splits; a.part_ml = part_ml; a.part_out = part_out;
  auto run = [&](int phase) {
    const bool small = d <= 64 && dv <= 64;
    if (tma) return small ? launch_talk_mma_cl<4, 4, true>(a, sh, cluster, smem, num_seqs, max_query_len, phase, maps, stream)
                          : launch_talk_mma_cl<8, 8, true>(a, sh, cluster, smem, num_seqs, max_query_len, phase, maps, stream);
    return small ? launch_talk_mma_cl<4, 4, false>(a, sh, cluster, smem, num_seqs, max_query_len, phase, maps, stream)
                 : launch_talk_mma_cl<8, 8, false>(a, sh, cluster, smem, num_seqs, max_query_len, phase, maps, stream);
  };
  if (num_splits == 1 && !part_ml) return run(TM_BOTH);
  if (num_splits == 1) {
    const dim3 grid((max_query_len + TS_ROWS - 1) / TS_ROWS, num_seqs, heads);
    const size_t ssmem = sizeof(bf16) * 2 * (size_t)TS_KEYS * ((d <= 64 ? 64 : 128) + 8);
    if (int e = d <= 64 ? launch(talking_stats_kernel<4>, grid, TS_THREADS, ssmem, stream, a)
                        : launch(talking_stats_kernel<8>, grid, TS_THREADS, ssmem, stream, a)) return e;
    return run(TM_VALUES);
  }
  if (int e = run(TM_STATS)) return e;
  return run(TM_VALUES);
}
