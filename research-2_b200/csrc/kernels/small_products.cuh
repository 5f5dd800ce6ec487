// Products of a few rows with a small matrix, in float, for what must stay in 32-bit: gates, step sizes, decays, routers.
#pragma once

#include "common.cuh"

__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(a.x, a.y, b.x, b.y);
}

// Sums over a warp of N values per lane (N a power of two up to 32): each exchange halves the values that a lane still has a share
// of. On return v[0] is a whole sum, the one whose index is returned; lanes that differ in the low log2(32 / N) bits have the same
// one. The additions of one value are warp_sum's, in its order.
template <int N>
__device__ __forceinline__ int warp_sums(float (&v)[N], int lane) {
  int index = 0;
#pragma unroll
  for (int off = 16, n = N; off > 0; off >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool upper = (lane & off) != 0;
#pragma unroll
      for (int i = 0; i < N / 2; ++i) {
        if (i < n) {
          const float send = upper ? v[i] : v[i + n], keep = upper ? v[i + n] : v[i];
          v[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
        }
      }
      if (upper) index += n;
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], off);
    }
  }
  return index;
}

// rows[r] . w[n] for ROWS rows in shared memory ([ROWS][kpad] float, kpad a multiple of 4, zeros from K on) and every row n of
// w [N][K] (float or bfloat16): a warp has OUTS outputs of all rows at a time, lanes over K in pieces of four, so the matrix comes out of L2 once for all
// rows. emit(r, n, sum) is called by one lane, the lanes of a warp side by side. A sum is made in the same order whatever ROWS and OUTS are.
template <int ROWS, int OUTS, typename W, typename F>
__device__ __forceinline__ void rows_times_matrix(const float* rows, int kpad, const W* __restrict__ w, int K, int N, F emit) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_warps = blockDim.x >> 5;
  const bool pieces = (K & 3) == 0 && (reinterpret_cast<uintptr_t>(w) & (4 * sizeof(W) - 1)) == 0;   // pieces of four stay whole
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
        const W* wr = w + size_t(n0 + o < N ? n0 + o : N - 1) * K + k;
        if (pieces) v[o] = load4(wr);
        else v[o] = make_float4(to_float(wr[0]), k + 1 < K ? to_float(wr[1]) : 0.f, k + 2 < K ? to_float(wr[2]) : 0.f, k + 3 < K ? to_float(wr[3]) : 0.f);
      }
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        const float4 m = *reinterpret_cast<const float4*>(rows + r * kpad + k);
#pragma unroll
        for (int o = 0; o < OUTS; ++o)
          acc[o][r] = fmaf(m.w, v[o].w, fmaf(m.z, v[o].z, fmaf(m.y, v[o].y, fmaf(m.x, v[o].x, acc[o][r]))));
      }
    }
    constexpr int AT_ONCE = OUTS * ROWS > 32 ? 32 / ROWS : OUTS, SUMS = AT_ONCE * ROWS;   // outputs whose sums are exchanged together
#pragma unroll
    for (int first = 0; first < OUTS; first += AT_ONCE) {
      float sums[SUMS];
#pragma unroll
      for (int o = 0; o < AT_ONCE; ++o)
#pragma unroll
        for (int r = 0; r < ROWS; ++r) sums[o * ROWS + r] = acc[first + o][r];
      const int mine = warp_sums<SUMS>(sums, lane);   // which of them this lane has in sums[0]
      const int o = first + mine / ROWS, r = mine % ROWS;
      if ((lane & (32 / SUMS - 1)) == 0 && n0 + o < N) emit(r, n0 + o, sums[0]);
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
