// Two attention maps of a head over the same values, combined: o = a1 - factor a2, divided by its root mean square over
// the head's value columns, times a constant. One warp per (row, head); x is [T, heads, 2, dv], out [T, heads, dv]. The rows
// are all rows of a step or, with a list of requests, each one's only new row. 32-bit, rounded once. What earlier kernels
// wrote is read through pointers without __restrict__, so that no read can move in front of the wait for them.
#define TS_PDL_CLASS PDL_ELEMENTWISE
#include "common.cuh"

namespace ts {

constexpr int PC_WARPS = 4;
constexpr int PC_COLS = 8;        // value columns a lane keeps (dv up to 256)

template <typename T>
__global__ void __launch_bounds__(PC_WARPS * 32) pair_combine_kernel(const T* x, const float* __restrict__ factor, float eps,
                                                                     float mult, T* out, int num_rows, int heads, int dv,
                                                                     const int* __restrict__ seqs, const int* __restrict__ cu_q) {
  pdl_trigger();
  pdl_wait();
  const long long warp = ((long long)blockIdx.x * blockDim.x + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  if (warp >= (long long)num_rows * heads) return;
  const int i = (int)(warp / heads), h = (int)(warp - (long long)i * heads);
  const int row = seqs ? cu_q[seqs[i]] : i;
  const T* a1 = x + ((size_t)row * heads + h) * 2 * dv;
  const T* a2 = a1 + dv;
  const float f = *factor;
  float v[PC_COLS];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < PC_COLS; ++j) {
    const int c = lane + 32 * j;
    v[j] = c < dv ? fmaf(-f, to_float(a2[c]), to_float(a1[c])) : 0.f;
    ss = fmaf(v[j], v[j], ss);
  }
  const float by = rsqrtf(warp_sum(ss) / (float)dv + eps) * mult;
  T* o = out + ((size_t)row * heads + h) * dv;
#pragma unroll
  for (int j = 0; j < PC_COLS; ++j) {
    const int c = lane + 32 * j;
    if (c < dv) o[c] = from_float<T>(v[j] * by);
  }
}

}  // namespace ts

using namespace ts;

extern "C" int ts_pair_combine(const void* x, const float* factor, float eps, float mult, void* out, int num_rows, int heads, int dv,
                               const int* seqs, const int* cu_q, int dtype, cudaStream_t stream) {
  if (num_rows <= 0) return 0;
  if (!x || !factor || !out || heads <= 0 || (seqs && !cu_q)) return TS_ERR_BAD_ARGUMENT;
  if (dv <= 0 || dv > 32 * PC_COLS) return TS_ERR_UNSUPPORTED;
  const long long warps = (long long)num_rows * heads;
  const int blocks = (int)((warps + PC_WARPS - 1) / PC_WARPS);
  if (dtype == TS_DTYPE_F32)
    return launch(pair_combine_kernel<float>, blocks, PC_WARPS * 32, 0, stream, (const float*)x, factor, eps, mult, (float*)out, num_rows,
                  heads, dv, seqs, cu_q);
  if (dtype == TS_DTYPE_BF16)
    return launch(pair_combine_kernel<bf16>, blocks, PC_WARPS * 32, 0, stream, (const bf16*)x, factor, eps, mult, (bf16*)out, num_rows,
                  heads, dv, seqs, cu_q);
  return TS_ERR_BAD_ARGUMENT;
}
