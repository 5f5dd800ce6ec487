// A residual stream that runs in several copies side by side ("streams"): x [T][S][D] float.
//
//   u = sum_a read[a] x_a                               what a sublayer reads, through an RMS norm
//   x_b <- sum_a mix[a][b] x_a + join[b] y              how its output y joins the streams, all of them at once from the old ones
//
//   r2_stream_join   one launch between two sublayers: the streams take the first one's output (y; null: they stay as they are), and the
//                    second one's input leaves with them: u of the NEW streams, normed (u / sqrt(mean(u^2) + eps) * gain) in the compute
//                    dtype, or u itself in float where no gain is given (the end of the layers: u is the streams' sum). The streams may
//                    come as one row per token that stands for all of them (the embedding's output), so that copies which hold the
//                    same are never written. One CTA a row; a column's S values are one thread's, so the streams may be renewed in
//                    place; the row's u stays in registers between the sum of its squares and the way out.
#include <math.h>

#include "common.cuh"

namespace {

constexpr int MAX_STREAMS = 32, STREAM_THREADS = 512, MANY_THREADS = 256;   // (MANY: more than eight streams)

struct StreamArgs {
  const float* x; int spread;      // [T][S][D], or [T][D] (spread): every stream holds that row
  const float* y;                  // [T][D] or null
  const float* mix;                // [S][S], [from][to]
  const float* join;               // [S]
  const float* read;               // [S]
  float* x_out;                    // [T][S][D] (may be x), or null: the new streams themselves are not needed
  const float* gain; float eps;    // [D] or null
  void* u_out;                     // [T][D]
  int streams, width;
};

template <int V> struct Pack { float v[V]; };
template <int V> __device__ __forceinline__ Pack<V> load_pack(const float* p);
template <> __device__ __forceinline__ Pack<1> load_pack<1>(const float* p) { return {{*p}}; }
template <> __device__ __forceinline__ Pack<4> load_pack<4>(const float* p) {
  const float4 f = *reinterpret_cast<const float4*>(p);
  return {{f.x, f.y, f.z, f.w}};
}
__device__ __forceinline__ void store_pack(float* p, const Pack<1>& a) { *p = a.v[0]; }
__device__ __forceinline__ void store_pack(float* p, const Pack<4>& a) { *reinterpret_cast<float4*>(p) = make_float4(a.v[0], a.v[1], a.v[2], a.v[3]); }
__device__ __forceinline__ void store_pack(bf16* p, const Pack<1>& a) { *p = __float2bfloat16_rn(a.v[0]); }
__device__ __forceinline__ void store_pack(bf16* p, const Pack<4>& a) {
  __nv_bfloat162 lo = __floats2bfloat162_rn(a.v[0], a.v[1]), hi = __floats2bfloat162_rn(a.v[2], a.v[3]);
  uint2 both;
  both.x = *reinterpret_cast<uint32_t*>(&lo);
  both.y = *reinterpret_cast<uint32_t*>(&hi);
  *reinterpret_cast<uint2*>(p) = both;
}

// S: the number of streams, up to eight, whose values at a thread's columns are registers; 0: a.streams of them, in shared memory.
// V: neighbouring columns a thread takes at once. KEEP: how many such pieces of u a thread keeps for the norm's second pass; it makes
// those beyond them again.
template <int S, int V, int KEEP, typename O>
__global__ void __launch_bounds__(STREAM_THREADS)
stream_join_kernel(const StreamArgs a) {
  pdl_launch_dependents();
  constexpr int MOST = S > 0 ? S : MAX_STREAMS;
  __shared__ float mix_s[MOST * MOST], join_s[MOST], read_s[MOST], scratch[33];
  __shared__ float many_s[S > 0 ? 1 : MAX_STREAMS * MANY_THREADS];
  const int n = S > 0 ? S : a.streams, width = a.width;
  const bool joins = a.y != nullptr;
  // the weights are no kernel's output
  for (int i = threadIdx.x; i < n * n; i += blockDim.x) mix_s[i] = joins ? a.mix[i] : 0.f;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    join_s[i] = joins ? a.join[i] : 0.f;
    read_s[i] = a.read[i];
  }
  __syncthreads();
  pdl_wait();
  const size_t t = blockIdx.x;
  const float* x = a.x + t * size_t(a.spread ? width : n * width);
  const size_t x_step = a.spread ? 0 : width;
  float* x_out = a.x_out != nullptr ? a.x_out + t * size_t(n) * width : nullptr;
  O* u_out = static_cast<O*>(a.u_out) + t * width;

  auto summed = [&](const float* streams, size_t step, int d) {   // u of streams as they are
    Pack<V> u = {};
#pragma unroll S > 0 ? S : 4
    for (int s = 0; s < n; ++s) {
      const Pack<V> x_s = load_pack<V>(streams + s * step + d);
#pragma unroll
      for (int i = 0; i < V; ++i) u.v[i] = fmaf(read_s[s], x_s.v[i], u.v[i]);
    }
    return u;
  };
  auto joined = [&](int d) {   // the streams' new values at columns d .., stored; -> their u
    Pack<V> old[S > 0 ? S : 1], u = {};
    if (S > 0) {
#pragma unroll
      for (int s = 0; s < S; ++s) old[s] = load_pack<V>(x + s * x_step + d);
    } else {
      for (int s = 0; s < n; ++s) many_s[s * MANY_THREADS + threadIdx.x] = x[s * x_step + d];
    }
    const Pack<V> y = load_pack<V>(a.y + t * width + d);
#pragma unroll S > 0 ? S : 1
    for (int b = 0; b < n; ++b) {
      Pack<V> now;
#pragma unroll
      for (int i = 0; i < V; ++i) now.v[i] = join_s[b] * y.v[i];
#pragma unroll S > 0 ? S : 4
      for (int s = 0; s < n; ++s) {
        const float m = mix_s[s * n + b];
        if (S > 0) {
#pragma unroll
          for (int i = 0; i < V; ++i) now.v[i] = fmaf(m, old[S > 0 ? s : 0].v[i], now.v[i]);
        } else {
          now.v[0] = fmaf(m, many_s[s * MANY_THREADS + threadIdx.x], now.v[0]);
        }
      }
      if (x_out != nullptr) store_pack(x_out + size_t(b) * width + d, now);
#pragma unroll
      for (int i = 0; i < V; ++i) u.v[i] = fmaf(read_s[b], now.v[i], u.v[i]);
    }
    return u;
  };
  float read_all = 0.f;
  for (int s = 0; s < n; ++s) read_all += read_s[s];
  auto columns = [&](int d) {
    if (joins) return joined(d);
    if (!a.spread) return summed(x, x_step, d);
    Pack<V> u = load_pack<V>(x + d);   // every stream holds this row
#pragma unroll
    for (int i = 0; i < V; ++i) u.v[i] *= read_all;
    return u;
  };

  const int step = blockDim.x * V, first = threadIdx.x * V;
  if (a.gain == nullptr) {   // u itself
    for (int d = first; d < width; d += step) store_pack(u_out + d, columns(d));
    return;
  }
  Pack<V> keep[KEEP];
  float sq = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int d = first + k * step;
    if (d < width) {
      keep[k] = columns(d);
#pragma unroll
      for (int i = 0; i < V; ++i) sq = fmaf(keep[k].v[i], keep[k].v[i], sq);
    }
  }
  for (int d = first + KEEP * step; d < width; d += step) {
    const Pack<V> u = columns(d);
#pragma unroll
    for (int i = 0; i < V; ++i) sq = fmaf(u.v[i], u.v[i], sq);
  }
  const float inv = 1.f / sqrtf(block_sum(sq, scratch) / float(width) + a.eps);
  auto leave = [&](int d, Pack<V> u) {
    const Pack<V> g = load_pack<V>(a.gain + d);
#pragma unroll
    for (int i = 0; i < V; ++i) u.v[i] = u.v[i] * inv * g.v[i];
    store_pack(u_out + d, u);
  };
#pragma unroll
  for (int k = 0; k < KEEP; ++k) {
    const int d = first + k * step;
    if (d < width) leave(d, keep[k]);
  }
  // (a thread's own columns again: of the new streams where they were stored, else of the ones that came)
  for (int d = first + KEEP * step; d < width; d += step) leave(d, joins ? summed(x_out, width, d) : columns(d));
}

template <int S, int V, typename O>
int launch_streams(const StreamArgs& a, int n_rows, cudaStream_t stream) {
  const int pieces = (a.width + V - 1) / V, most = S > 0 ? STREAM_THREADS : MANY_THREADS;
  const int threads = pieces >= most ? most : (pieces + 31) / 32 * 32;
  if (pieces <= threads) r2_launch(stream_join_kernel<S, V, 1, O>, dim3(n_rows), dim3(threads), size_t(0), stream, a);
  else r2_launch(stream_join_kernel<S, V, 4, O>, dim3(n_rows), dim3(threads), size_t(0), stream, a);
  return launch_status();
}

template <typename O>
int choose_streams(const StreamArgs& a, int n_rows, bool quads, cudaStream_t stream) {
  switch (a.streams) {
#define R2_STREAMS(S) \
  case S: return quads ? launch_streams<S, 4, O>(a, n_rows, stream) : launch_streams<S, 1, O>(a, n_rows, stream);
    R2_STREAMS(1) R2_STREAMS(2) R2_STREAMS(3) R2_STREAMS(4) R2_STREAMS(5) R2_STREAMS(6) R2_STREAMS(7) R2_STREAMS(8)
#undef R2_STREAMS
    default: return launch_streams<0, 1, O>(a, n_rows, stream);
  }
}

}  // namespace

// x float [n_rows][streams][width] (spread: [n_rows][width]); y float [n_rows][width] or null; mix float [streams][streams] ([from][to])
// and join float [streams] where y is given; read float [streams]; x_out float [n_rows][streams][width] (may be x) or null; gain float
// [width] and u_out [n_rows][width] in `out_dtype`, or gain null and u_out float.
extern "C" int r2_stream_join(const float* x, int spread, const float* y, const float* mix, const float* join, const float* read, float* x_out,
                              const float* gain, float eps, void* u_out, int n_rows, int streams, int width, int out_dtype, cudaStream_t stream) {
  if (n_rows <= 0) return R2_OK;
  if (streams < 1 || streams > MAX_STREAMS || width < 1 || x == nullptr || read == nullptr || u_out == nullptr) return R2_BAD_SHAPE;
  if (y != nullptr && (mix == nullptr || join == nullptr)) return R2_BAD_SHAPE;
  if (y != nullptr && gain != nullptr && x_out == nullptr) return R2_BAD_SHAPE;
  if ((spread && x_out == x) || (y == nullptr && x_out != nullptr) || (gain == nullptr && out_dtype != R2_F32)) return R2_BAD_SHAPE;
  StreamArgs a = {x, spread, y, mix, join, read, x_out, gain, eps, u_out, streams, width};
  auto on16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  const bool quads = width % 4 == 0 && on16(x) && on16(y) && on16(x_out) && on16(gain) && on16(u_out);
  if (out_dtype == R2_F32) return choose_streams<float>(a, n_rows, quads, stream);
  if (out_dtype == R2_BF16) return choose_streams<bf16>(a, n_rows, quads, stream);
  return R2_BAD_DTYPE;
}
