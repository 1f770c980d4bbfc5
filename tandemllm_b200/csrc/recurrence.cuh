// What the recurrences over a matrix state share (recurrence.cu, recurrence_write.cu): the activations, copies into shared memory, the
// sum over the lanes that share a column of the state, and the size of the scans' blocks.
#pragma once

#include "common.cuh"

namespace tl {

constexpr int REC_THREADS = 256;

__device__ __forceinline__ float sigmoidf_(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float siluf_(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ float softplusf_(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

__device__ __forceinline__ void rec_cp16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void rec_cp4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// Sums v[0..T) over the P neighbouring lanes that share a column (`part` = the lane's place among them; P divides 32). Each
// crossing halves what a lane still holds: afterwards v[i], i < T / P, of lane `part` are the whole sums of tokens
// part * (T / P) + i; with more lanes than tokens, v[0] of the P / T lanes from part = token * (P / T) on is that token's sum.
template <int T, int P>
__device__ __forceinline__ void rec_reduce_scatter(float (&v)[T], int part) {
#pragma unroll
  for (int step = 0; (P >> 1 >> step) > 0; ++step) {
    const int off = P >> 1 >> step;
    const int cnt = (T >> step) > 1 ? (T >> step) : 1;
    if (cnt > 1) {
      const int half = cnt / 2;
      const bool up = (part & off) != 0;
#pragma unroll
      for (int i = 0; i < half; ++i) {
        const float send = up ? v[i] : v[i + half];
        const float keep = up ? v[i + half] : v[i];
        v[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
      }
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], off);
    }
  }
}

// Threads a block (a multiple of 32, at least P) and the value columns it takes: the largest block that still gives the GPU
// `want_blocks` blocks, else a single warp; never more columns than there are. (Steps of a few rows want many blocks in
// flight for the states they read and write; the staged form's blocks each fetch every prepared token of their head, so
// they stay as large as fills three SMs in four.)
static void recurrence_block(int requests, int H, int VD, int P, long long want_blocks, int* threads, int* cols) {
  const int needed = ((VD * P + 31) / 32) * 32;
  int th = REC_THREADS;
  while (th > 32 && th / 2 >= P && (long long)requests * H * ceil_div(VD, th / P) < want_blocks) th >>= 1;
  if (th > needed) th = needed;
  if (th < P) th = P;
  *threads = th;
  *cols = th / P;
}

}  // namespace tl
