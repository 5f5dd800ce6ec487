// Products of a few rows with a small float matrix, for what must stay in 32-bit: gates, step sizes, decays, routers.
#pragma once

#include "common.cuh"

// rows[r] . w[n] for ROWS rows in shared memory ([ROWS][kpad] float, kpad a multiple of 4, zeros from K on) and every row n of
// w [N][K]: a warp has OUTS outputs of all rows at a time, lanes over K in pieces of four, so the matrix comes out of L2 once for all
// rows. emit(r, n, sum) is called by one lane. A sum is made in the same order whatever ROWS and OUTS are.
template <int ROWS, int OUTS, typename F>
__device__ __forceinline__ void rows_times_matrix(const float* rows, int kpad, const float* __restrict__ w, int K, int N, F emit) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  const bool pieces = (K & 3) == 0 && (reinterpret_cast<uintptr_t>(w) & 15) == 0;   // every row of w starts on a 16-byte boundary
  for (int n0 = warp * OUTS; n0 < N; n0 += n_warps * OUTS) {
    float acc[OUTS][ROWS];
#pragma unroll
    for (int o = 0; o < OUTS; ++o)
#pragma unroll
      for (int r = 0; r < ROWS; ++r) acc[o][r] = 0.f;
#pragma unroll 2
    for (int k = lane * 4; k < kpad; k += 128) {
      float4 v[OUTS];
#pragma unroll
      for (int o = 0; o < OUTS; ++o) {
        const float* wr = w + size_t(n0 + o < N ? n0 + o : N - 1) * K + k;
        if (pieces) v[o] = *reinterpret_cast<const float4*>(wr);
        else v[o] = make_float4(wr[0], k + 1 < K ? wr[1] : 0.f, k + 2 < K ? wr[2] : 0.f, k + 3 < K ? wr[3] : 0.f);
      }
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        const float4 m = *reinterpret_cast<const float4*>(rows + r * kpad + k);
#pragma unroll
        for (int o = 0; o < OUTS; ++o)
          acc[o][r] = fmaf(m.w, v[o].w, fmaf(m.z, v[o].z, fmaf(m.y, v[o].y, fmaf(m.x, v[o].x, acc[o][r]))));
      }
    }
#pragma unroll
    for (int o = 0; o < OUTS; ++o)
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        const float sum = warp_sum(acc[o][r]);
        if (lane == (o * ROWS + r) % 32 && n0 + o < N) emit(r, n0 + o, sum);
      }
  }
}

// Shared memory beyond the default 48 KB is asked for before the launch; false: more than an SM has.
template <typename... A>
static inline bool room_for(void (*kernel)(A...), size_t smem) {
  if (smem <= 48 * 1024) return true;
  if (smem > 227 * 1024) return false;
  return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, int(smem)) == cudaSuccess;
}
