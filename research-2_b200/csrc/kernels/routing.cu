// Small projections that must stay in 32-bit, the choice of experts, and the experts' activation.
//
//   r2_small_linear   out[t][n] = bias[n] + sum_k h[t][k] * w[n][k] in float, for a handful of outputs per row (gates
//                     of a recurrence, one gate per head, step sizes, router logits): weights and result are float
//                     whatever the activations' type, every output one warp's sum in a fixed order.
//   r2_route_top_k    router logits in float, the `top` largest per row (the lower index wins a tie), softmax over the
//                     chosen logits only -> a dense row of weights [T, experts] (zero for experts not chosen), and the
//                     choices themselves.
//   r2_route_scored   the same with sigmoid scores: an expert is chosen by its score plus a learned correction, only
//                     inside the best groups of neighbouring experts (a group counts by its two best), and weighted by
//                     its plain score over the chosen experts' sum; further rows of the weight matrix give sigmoid gates
//                     of their own (one number per row of the batch, e.g. for an expert that every row uses). Or with
//                     scores that are the softmax over all experts, groups that count by their best expert alone, and
//                     weights that are the chosen scores times a constant (not made to sum to one).
//   r2_expert_act     the inner activation of gated feed-forwards whose [gate | up] projections of several experts
//                     (and of one more expert that every row uses) lie side by side in one row; each expert's
//                     columns are multiplied by the row's weight for that expert, so that ONE down product over the
//                     stacked matrices is the weighted sum of the experts' outputs.
//   r2_expert_unit    the same for experts without gates.
//
// In r2_route_scored the last outputs of the router may stand for no expert but for the row itself (identity outputs): the launch
// then also gives the row times their weights' sum, which joins the experts' sum as that product's addend.
#include <math.h>

#include "common.cuh"

namespace {

constexpr int MAX_EXPERTS = 1024;

template <typename T>
__global__ void __launch_bounds__(256)
small_linear_kernel(const T* __restrict__ h, int h_stride, const float* __restrict__ w, const float* __restrict__ bias,
                    float* __restrict__ out, int out_stride, int n_out, int width) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float row[];
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  const T* hr = h + size_t(t) * h_stride;
  for (int k = threadIdx.x; k < width; k += blockDim.x) row[k] = to_float(hr[k]);
  __syncthreads();
  for (int n = warp; n < n_out; n += n_warps) {
    const float* wr = w + size_t(n) * width;
    float acc = 0.f;
    for (int k = lane; k < width; k += 32) acc = fmaf(row[k], wr[k], acc);
    acc = warp_sum(acc);
    if (lane == 0) out[size_t(t) * out_stride + n] = acc + (bias != nullptr ? bias[n] : 0.f);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
route_top_k_kernel(const T* __restrict__ h, int h_stride, const float* __restrict__ w, const float* __restrict__ bias,
                   float* __restrict__ dense, int32_t* __restrict__ chosen, float* __restrict__ chosen_weight,
                   int n_experts, int top, int width) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float smem[];
  float* row = smem;             // [width]
  float* logit = smem + width;   // [n_experts]
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5;
  const T* hr = h + size_t(t) * h_stride;
  for (int k = threadIdx.x; k < width; k += blockDim.x) row[k] = to_float(hr[k]);
  __syncthreads();
  for (int n = warp; n < n_experts; n += n_warps) {
    const float* wr = w + size_t(n) * width;
    float acc = 0.f;
    for (int k = lane; k < width; k += 32) acc = fmaf(row[k], wr[k], acc);
    acc = warp_sum(acc);
    if (lane == 0) logit[n] = acc + (bias != nullptr ? bias[n] : 0.f);
  }
  for (int n = threadIdx.x; n < n_experts; n += blockDim.x) dense[size_t(t) * n_experts + n] = 0.f;
  __syncthreads();
  if (warp != 0) return;
  // the first warp picks the largest logit `top` times; a picked one is set to -inf. The first pick is the maximum
  // of the chosen, so the softmax over them needs no second pass for it.
  float best0 = 0.f, sum = 0.f;
  for (int c = 0; c < top; ++c) {
    float v = -INFINITY;
    int at = n_experts;
    for (int n = lane; n < n_experts; n += 32)
      if (logit[n] > v) { v = logit[n]; at = n; }
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, v, o);
      const int oat = __shfl_xor_sync(0xffffffffu, at, o);
      if (ov > v || (ov == v && oat < at)) { v = ov; at = oat; }
    }
    if (at >= n_experts) { at = c; v = best0; }   // logits that are not numbers: no index may leave the row
    if (c == 0) best0 = v;
    const float p = expf(v - best0);
    sum += p;
    if (lane == 0) {
      chosen[size_t(t) * top + c] = at;
      chosen_weight[size_t(t) * top + c] = p;
      logit[at] = -INFINITY;
    }
    __syncwarp();
  }
  const float inv = 1.f / sum;
  for (int c = lane; c < top; c += 32) {
    const float p = chosen_weight[size_t(t) * top + c] * inv;
    chosen_weight[size_t(t) * top + c] = p;
    dense[size_t(t) * n_experts + chosen[size_t(t) * top + c]] = p;
  }
}

// Router with sigmoid scores. w holds n_experts rows of router weights and then n_extra more rows; their logits leave as
// they are in `extra` [T, n_extra] (gates whose sigmoid another kernel takes). s = sigmoid(logit); an expert's choice score is
// s + correction; the experts form n_groups equal groups of neighbours, a group's mark is the sum of its two largest
// choice scores (of its one, where a group is a single expert), and only experts of the `keep` groups with the largest marks
// can be chosen (the lower index wins a tie, among groups and among experts). The `top` largest choice scores are chosen; a
// chosen expert's weight is its s over the sum of the chosen s (+ 1e-20).
// softmax_scores: s = softmax of the logits over all experts instead of their sigmoids. mark_best_only: a group's mark is its
// largest choice score alone. normalise = 0: the chosen s are not divided by their sum. The weights are multiplied by weight_scale.
// n_identity: the last of the n_experts outputs stand for no expert but for the input row itself: carried[t] = their weights' sum
// * h[t] (+ base[t] where given), float.
struct RouteArgs {
  const void* h; int h_stride;
  const float* w; const float* correction;
  float* dense; int32_t* chosen; float* chosen_weight; float* extra;
  int n_experts, n_extra, top, n_groups, keep, width, softmax_scores, mark_best_only, normalise;
  float weight_scale;
  int n_identity; const float* base; float* carried;
  int quads;   // rows of w start on 16-byte boundaries and hold a multiple of four numbers
};

// What a row's choice works on, in shared memory.
struct RouteRow {
  float* row;          // [width]
  float* score;        // [n_experts] the scores
  float* choice;       // [n_experts] score + correction; -inf once picked or outside the kept groups
  float* given;        // [n_experts] the weights, zero where not chosen
  float* mark;         // [n_groups]
  float* pick_weight;  // [top]
  int* pick;           // [top]
};
__device__ __host__ __forceinline__ size_t route_row_floats(int width, int n_experts, int n_groups, int top) {
  return (size_t(width) + 3 * n_experts + n_groups + 2 * top + 3) / 4 * 4;
}
__device__ __forceinline__ RouteRow route_row(float* at, const RouteArgs& a) {
  RouteRow r;
  r.row = at;
  r.score = at + a.width;
  r.choice = r.score + a.n_experts;
  r.given = r.choice + a.n_experts;
  r.mark = r.given + a.n_experts;
  r.pick_weight = r.mark + a.n_groups;
  r.pick = reinterpret_cast<int*>(r.pick_weight + a.top);
  return r;
}

// a logit: what becomes of it
__device__ __forceinline__ void put_logit(const RouteArgs& a, const RouteRow& r, int t, int n, float z) {
  if (n < a.n_experts) {
    const float s = a.softmax_scores ? z : 1.f / (1.f + expf(-z));   // (the softmax follows once all logits are there)
    r.score[n] = s;
    r.choice[n] = s + (a.correction != nullptr ? a.correction[n] : 0.f);
  } else {
    a.extra[size_t(t) * a.n_extra + (n - a.n_experts)] = z;
  }
}

// One warp: scores, groups, picks and weights of row t, from its logits. -> the identity outputs' weights' sum
__device__ __forceinline__ float choose_experts(const RouteArgs& a, const RouteRow& r, int t, int lane) {
  if (a.softmax_scores) {
    // s = exp(z - max) / sum over all experts, one warp, sums in a fixed order
    float top_z = -INFINITY;
    for (int n = lane; n < a.n_experts; n += 32) top_z = fmaxf(top_z, r.score[n]);
    for (int o = 16; o > 0; o >>= 1) top_z = fmaxf(top_z, __shfl_xor_sync(0xffffffffu, top_z, o));
    float total = 0.f;
    for (int n = lane; n < a.n_experts; n += 32) {
      const float e = expf(r.score[n] - top_z);
      r.score[n] = e;
      total += e;
    }
    total = warp_sum(total);
    const float inv_total = 1.f / total;
    for (int n = lane; n < a.n_experts; n += 32) {
      const float s = r.score[n] * inv_total;
      r.score[n] = s;
      r.choice[n] = s + (a.correction != nullptr ? a.correction[n] : 0.f);
    }
    __syncwarp();
  }
  const int size = a.n_experts / a.n_groups;
  if (a.keep < a.n_groups) {
    for (int g = lane; g < a.n_groups; g += 32) {
      float best = -INFINITY, second = -INFINITY;   // the group's largest and second largest
      for (int n = g * size; n < (g + 1) * size; ++n) {
        const float c = r.choice[n];
        if (c > best) { second = best; best = c; }
        else if (c > second) second = c;
      }
      r.mark[g] = (size > 1 && !a.mark_best_only) ? best + second : best;
    }
    __syncwarp();
    // the kept groups: `keep` times the largest mark; a kept group's mark becomes +inf, and what is not +inf at the end is out
    for (int c = 0; c < a.keep; ++c) {
      float v = -INFINITY;
      int at = a.n_groups;
      for (int g = lane; g < a.n_groups; g += 32)
        if (r.mark[g] != INFINITY && (r.mark[g] > v || at == a.n_groups)) { v = r.mark[g]; at = g; }
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, o);
        const int oat = __shfl_xor_sync(0xffffffffu, at, o);
        if (oat < a.n_groups && (at == a.n_groups || ov > v || (ov == v && oat < at))) { v = ov; at = oat; }
      }
      if (lane == 0 && at < a.n_groups) r.mark[at] = INFINITY;
      __syncwarp();
    }
    for (int n = lane; n < a.n_experts; n += 32)
      if (r.mark[n / size] != INFINITY) r.choice[n] = -INFINITY;
    __syncwarp();
  }
  float sum = 0.f;
  for (int c = 0; c < a.top; ++c) {
    float v = -INFINITY;
    int at = a.n_experts;
    for (int n = lane; n < a.n_experts; n += 32)
      if (r.choice[n] > v) { v = r.choice[n]; at = n; }
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, v, o);
      const int oat = __shfl_xor_sync(0xffffffffu, at, o);
      if (ov > v || (ov == v && oat < at)) { v = ov; at = oat; }
    }
    if (at >= a.n_experts) at = c;   // scores that are not numbers: no index may leave the row
    const float s = r.score[at];
    sum += s;
    if (lane == 0) {
      r.pick[c] = at;
      r.pick_weight[c] = s;
      r.choice[at] = -INFINITY;
    }
    __syncwarp();
  }
  const float inv = (a.normalise ? 1.f / (sum + 1e-20f) : 1.f) * a.weight_scale;
  for (int c = lane; c < a.top; c += 32) {
    const float p = r.pick_weight[c] * inv;
    a.chosen[size_t(t) * a.top + c] = r.pick[c];
    a.chosen_weight[size_t(t) * a.top + c] = p;
    r.given[r.pick[c]] = p;
  }
  __syncwarp();
  float share = 0.f;
  for (int n = a.n_experts - a.n_identity + lane; n < a.n_experts; n += 32) share += r.given[n];
  return warp_sum(share);
}

// four neighbouring products into four sums: the order in which a logit's terms are added is the same in both forms below
__device__ __forceinline__ void add_quad(float (&sum)[4], const float4 x, const float4 w) {
  sum[0] = fmaf(x.x, w.x, sum[0]);
  sum[1] = fmaf(x.y, w.y, sum[1]);
  sum[2] = fmaf(x.z, w.z, sum[2]);
  sum[3] = fmaf(x.w, w.w, sum[3]);
}

// A CTA a row. A warp has an output at a time; with `quads` its row of w comes as 16-byte pieces, the first ROUTE_AHEAD of them asked for
// before the kernel before this one has ended (weights are no kernel's output).
constexpr int ROUTE_AHEAD = 6, ROUTE_WARPS = 16;
template <typename T>
__global__ void __launch_bounds__(ROUTE_WARPS * 32)
route_scored_kernel(const RouteArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float smem[];
  __shared__ float identity_weight;
  const RouteRow r = route_row(smem, a);
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, n_warps = blockDim.x >> 5, width = a.width;
  float4 ahead[ROUTE_AHEAD];
  if (a.quads && warp < a.n_experts + a.n_extra) {
#pragma unroll
    for (int i = 0; i < ROUTE_AHEAD; ++i) {
      const int k = 4 * lane + 128 * i;
      ahead[i] = k < width ? *reinterpret_cast<const float4*>(a.w + size_t(warp) * width + k) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  for (int n = threadIdx.x; n < a.n_experts; n += blockDim.x) r.given[n] = 0.f;
  pdl_wait();
  const T* hr = static_cast<const T*>(a.h) + size_t(t) * a.h_stride;
  for (int k = threadIdx.x; k < width; k += blockDim.x) r.row[k] = to_float(hr[k]);
  __syncthreads();
  for (int n = warp; n < a.n_experts + a.n_extra; n += n_warps) {
    const float* wr = a.w + size_t(n) * width;
    float acc = 0.f;
    if (a.quads) {
      float sum[4] = {0.f, 0.f, 0.f, 0.f};
      auto at = [&](const float* p, int k) { return *reinterpret_cast<const float4*>(p + k); };
#pragma unroll
      for (int i = 0; i < ROUTE_AHEAD; ++i) {
        const int k = 4 * lane + 128 * i;
        if (k < width) add_quad(sum, at(r.row, k), n == warp ? ahead[i] : at(wr, k));
      }
#pragma unroll 4
      for (int k = 4 * lane + 128 * ROUTE_AHEAD; k < width; k += 128) add_quad(sum, at(r.row, k), at(wr, k));
      acc = (sum[0] + sum[1]) + (sum[2] + sum[3]);
    } else {
#pragma unroll 4
      for (int k = lane; k < width; k += 32) acc = fmaf(r.row[k], wr[k], acc);
    }
    acc = warp_sum(acc);
    if (lane == 0) put_logit(a, r, t, n, acc);
  }
  __syncthreads();
  if (warp == 0) {
    const float share = choose_experts(a, r, t, lane);
    if (lane == 0) identity_weight = share;
  }
  __syncthreads();
  for (int n = threadIdx.x; n < a.n_experts; n += blockDim.x) a.dense[size_t(t) * a.n_experts + n] = r.given[n];
  if (a.n_identity == 0) return;
  const float share = identity_weight;
  for (int k = threadIdx.x; k < width; k += blockDim.x)
    a.carried[size_t(t) * width + k] = share * r.row[k] + (a.base != nullptr ? a.base[size_t(t) * width + k] : 0.f);
}

// A warp a row, for many rows: the weights are in shared memory once a CTA, whose warps take row after row. (`quads` only.)
constexpr int ROUTE_ROWS = 8;
template <typename T>
__global__ void __launch_bounds__(ROUTE_ROWS * 32)
route_scored_rows_kernel(const RouteArgs a, int n_rows) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float smem[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, width = a.width, outputs = a.n_experts + a.n_extra;
  float* ws = smem;   // [outputs][width]
  const RouteRow r = route_row(smem + size_t(outputs) * width + warp * route_row_floats(width, a.n_experts, a.n_groups, a.top), a);
  for (int i = threadIdx.x; i < outputs * width / 4; i += blockDim.x) reinterpret_cast<float4*>(ws)[i] = reinterpret_cast<const float4*>(a.w)[i];
  __syncthreads();
  pdl_wait();
  for (int t = blockIdx.x * ROUTE_ROWS + warp; t < n_rows; t += gridDim.x * ROUTE_ROWS) {
    const T* hr = static_cast<const T*>(a.h) + size_t(t) * a.h_stride;
    for (int k = lane; k < width; k += 32) r.row[k] = to_float(hr[k]);
    for (int n = lane; n < a.n_experts; n += 32) r.given[n] = 0.f;
    __syncwarp();
    for (int n0 = 0; n0 < outputs; n0 += 4) {   // four outputs at a time: the row's numbers are read once for them
      float sum[4][4] = {};
      const float* wr[4];
#pragma unroll
      for (int o = 0; o < 4; ++o) wr[o] = ws + size_t(min(n0 + o, outputs - 1)) * width;
#pragma unroll 2
      for (int k = 4 * lane; k < width; k += 128) {
        const float4 x = *reinterpret_cast<const float4*>(r.row + k);
#pragma unroll
        for (int o = 0; o < 4; ++o) add_quad(sum[o], x, *reinterpret_cast<const float4*>(wr[o] + k));
      }
#pragma unroll
      for (int o = 0; o < 4; ++o) {
        const float acc = warp_sum((sum[o][0] + sum[o][1]) + (sum[o][2] + sum[o][3]));
        if (lane == 0 && n0 + o < outputs) put_logit(a, r, t, n0 + o, acc);
      }
    }
    __syncwarp();
    const float share = choose_experts(a, r, t, lane);
    for (int n = lane; n < a.n_experts; n += 32) a.dense[size_t(t) * a.n_experts + n] = r.given[n];
    if (a.n_identity > 0) {
      for (int k = 4 * lane; k < width; k += 128) {
        const float4 x = *reinterpret_cast<const float4*>(r.row + k);
        const size_t at = size_t(t) * width + k;
        const float4 b = a.base != nullptr ? *reinterpret_cast<const float4*>(a.base + at) : make_float4(0.f, 0.f, 0.f, 0.f);
        *reinterpret_cast<float4*>(a.carried + at) = make_float4(share * x.x + b.x, share * x.y + b.y, share * x.z + b.z, share * x.w + b.w);
      }
    }
    __syncwarp();   // (the warp's next row)
  }
}

constexpr int KIND_CLAMPED_SWISH = 0, KIND_RELU = 1, KIND_SILU = 2, KIND_GELU_TANH = 3;

__device__ __forceinline__ float gated_unit(float g, float u, int kind, float limit, float alpha, float up_offset) {
  if (kind == KIND_RELU) return fmaxf(g, 0.f) * u;
  if (kind == KIND_SILU) return g / (1.f + expf(-g)) * u;
  if (kind == KIND_GELU_TANH) return gelu_tanh(g) * u;
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return g / (1.f + expf(-alpha * g)) * (u + up_offset);
}

// A row of `gate_up` holds [gates of all `inner` columns | ups of all `inner` columns]. The first n_experts *
// expert_width columns belong to routed experts (limit `limit`, times the row's weight for the expert); the rest to the
// expert that every row uses (limit `tail_limit`; weight one, or sigmoid(tail_gate[row]) where a gate is given).
// n_experts = 0: one plain gated unit.
template <typename T>
__global__ void __launch_bounds__(256)
expert_act_kernel(const T* __restrict__ gate_up, int in_stride, T* __restrict__ out, int out_stride, int inner, int kind,
                  float limit, float alpha, float up_offset, const float* __restrict__ route, int route_stride, int n_experts, int expert_width,
                  float tail_limit, const float* __restrict__ tail_gate, int tail_gate_stride) {
  pdl_launch_dependents();
  pdl_wait();
  const T* in = gate_up + size_t(blockIdx.x) * in_stride;
  // the weight of the columns after the routed experts': one, or the sigmoid of the row's gate logit
  const float tail_weight = tail_gate != nullptr ? 1.f / (1.f + expf(-tail_gate[size_t(blockIdx.x) * tail_gate_stride])) : 1.f;
  T* o = out + size_t(blockIdx.x) * out_stride;
  const int routed = n_experts * expert_width;
  for (int f = blockIdx.y * blockDim.x + threadIdx.x; f < inner; f += gridDim.y * blockDim.x) {
    const bool tail = f >= routed;
    const float weight = tail ? tail_weight : route[size_t(blockIdx.x) * route_stride + f / expert_width];
    float y = 0.f;
    if (weight != 0.f) y = weight * gated_unit(to_float(in[f]), to_float(in[inner + f]), kind, tail ? tail_limit : limit, alpha, up_offset);
    o[f] = from_float<T>(y);
  }
}

// Experts without gates: a row of `up` holds the experts' inner values side by side; act(up) times the row's weight for the column's
// expert. (`route` rows are route_stride numbers apart.) With `vec` eight neighbouring columns, all of one expert, are one 16-byte piece.
template <typename T>
__global__ void __launch_bounds__(256)
expert_unit_kernel(const T* __restrict__ up, int in_stride, T* __restrict__ out, int out_stride, int inner, int act,
                   const float* __restrict__ route, int route_stride, int expert_width, int vec) {
  pdl_launch_dependents();
  pdl_wait();
  const T* in = up + size_t(blockIdx.x) * in_stride;
  T* o = out + size_t(blockIdx.x) * out_stride;
  const float* weights = route + size_t(blockIdx.x) * route_stride;
  if (sizeof(T) == 2 && vec) {
    for (int f = 8 * (blockIdx.y * blockDim.x + threadIdx.x); f < inner; f += 8 * gridDim.y * blockDim.x) {
      const float weight = weights[f / expert_width];
      uint4 yq = make_uint4(0u, 0u, 0u, 0u);
      if (weight != 0.f) {
        const uint4 zq = *reinterpret_cast<const uint4*>(in + f);
        const __nv_bfloat162* z2 = reinterpret_cast<const __nv_bfloat162*>(&zq);
        __nv_bfloat162* y2 = reinterpret_cast<__nv_bfloat162*>(&yq);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float2 z = __bfloat1622float2(z2[i]);
          y2[i] = __floats2bfloat162_rn(weight * activate(z.x, act), weight * activate(z.y, act));
        }
      }
      *reinterpret_cast<uint4*>(o + f) = yq;
    }
    return;
  }
  for (int f = blockIdx.y * blockDim.x + threadIdx.x; f < inner; f += gridDim.y * blockDim.x) {
    const float weight = weights[f / expert_width];
    o[f] = from_float<T>(weight != 0.f ? weight * activate(to_float(in[f]), act) : 0.f);
  }
}

}  // namespace

extern "C" int r2_small_linear(const void* h, int h_stride, const float* w, const float* bias, float* out, int out_stride,
                               int n_rows, int n_out, int width, int dtype, cudaStream_t stream) {
  if (n_rows <= 0 || n_out <= 0) return R2_OK;
  if (width < 1) return R2_BAD_SHAPE;
  const size_t smem = sizeof(float) * width;
  if (smem > 48 * 1024) return R2_UNSUPPORTED;
  const int threads = n_out >= 8 ? 256 : 32 * n_out;
  if (dtype == R2_F32) {
    r2_launch(small_linear_kernel<float>, dim3(n_rows), dim3(threads), smem, stream, (const float*)h, h_stride, w, bias, out, out_stride, n_out, width);
  } else if (dtype == R2_BF16) {
    r2_launch(small_linear_kernel<bf16>, dim3(n_rows), dim3(threads), smem, stream, (const bf16*)h, h_stride, w, bias, out, out_stride, n_out, width);
  } else {
    return R2_BAD_DTYPE;
  }
  return launch_status();
}

extern "C" int r2_route_top_k(const void* h, int h_stride, const float* w, const float* bias, float* dense, int32_t* chosen,
                              float* chosen_weight, int n_rows, int n_experts, int top, int width, int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return R2_OK;
  if (width < 1 || n_experts < 1 || n_experts > MAX_EXPERTS || top < 1 || top > n_experts) return R2_BAD_SHAPE;
  const size_t smem = sizeof(float) * (size_t(width) + n_experts);
  if (smem > 48 * 1024) return R2_UNSUPPORTED;
  if (dtype == R2_F32) {
    r2_launch(route_top_k_kernel<float>, dim3(n_rows), dim3(256), smem, stream, (const float*)h, h_stride, w, bias, dense, chosen, chosen_weight, n_experts, top, width);
  } else if (dtype == R2_BF16) {
    r2_launch(route_top_k_kernel<bf16>, dim3(n_rows), dim3(256), smem, stream, (const bf16*)h, h_stride, w, bias, dense, chosen, chosen_weight, n_experts, top, width);
  } else {
    return R2_BAD_DTYPE;
  }
  return launch_status();
}

// w float [n_experts + n_extra, width]; correction float [n_experts] (may be null); dense [T, n_experts], chosen / chosen_weight
// [T, top], extra [T, n_extra] (the further rows' logits; null when n_extra is 0); carried float [T, width] where n_identity > 0 (base
// likewise, or null). softmax_scores, mark_best_only, normalise and
// weight_scale choose the router's form (see the kernel).
extern "C" int r2_route_scored(const void* h, int h_stride, const float* w, const float* correction, float* dense, int32_t* chosen,
                               float* chosen_weight, float* extra, int n_rows, int n_experts, int n_extra, int top, int n_groups,
                               int keep, int width, int softmax_scores, int mark_best_only, int normalise, float weight_scale,
                               int n_identity, const float* base, float* carried, int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return R2_OK;
  if (width < 1 || n_experts < 1 || n_experts > MAX_EXPERTS || top < 1 || n_groups < 1 || n_experts % n_groups != 0 || keep < 1 ||
      keep > n_groups || top > n_experts / n_groups * keep || n_extra < 0 || (n_extra > 0 && extra == nullptr) ||
      n_identity < 0 || n_identity > n_experts || (n_identity > 0 && carried == nullptr)) return R2_BAD_SHAPE;
  RouteArgs a = {};
  a.h = h; a.h_stride = h_stride; a.w = w; a.correction = correction; a.dense = dense; a.chosen = chosen; a.chosen_weight = chosen_weight; a.extra = extra;
  a.n_experts = n_experts; a.n_extra = n_extra; a.top = top; a.n_groups = n_groups; a.keep = keep; a.width = width; a.softmax_scores = softmax_scores;
  a.mark_best_only = mark_best_only; a.normalise = normalise; a.weight_scale = weight_scale; a.n_identity = n_identity; a.base = base; a.carried = carried;
  auto on16 = [](const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
  a.quads = width % 4 == 0 && on16(w);
  if (dtype != R2_F32 && dtype != R2_BF16) return R2_BAD_DTYPE;
  const size_t per_row = sizeof(float) * route_row_floats(width, n_experts, n_groups, top);
  const int outputs = n_experts + n_extra;
  const size_t many = sizeof(float) * size_t(outputs) * width + ROUTE_ROWS * per_row;
  constexpr size_t MOST = 200 * 1024;   // (two CTAs an SM up to 113 KB)
  if (n_rows >= 512 && a.quads && many <= MOST && on16(base) && on16(carried)) {
    static bool configured = false;
    if (!configured) {
      cudaError_t e = cudaFuncSetAttribute(route_scored_rows_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(MOST));
      if (e == cudaSuccess) e = cudaFuncSetAttribute(route_scored_rows_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, int(MOST));
      if (e != cudaSuccess) return int(e);
      configured = true;
    }
    const dim3 grid(min((n_rows + ROUTE_ROWS - 1) / ROUTE_ROWS, 2048));
    if (dtype == R2_F32) r2_launch(route_scored_rows_kernel<float>, grid, dim3(ROUTE_ROWS * 32), many, stream, a, n_rows);
    else r2_launch(route_scored_rows_kernel<bf16>, grid, dim3(ROUTE_ROWS * 32), many, stream, a, n_rows);
    return launch_status();
  }
  if (per_row > 47 * 1024) return R2_UNSUPPORTED;
  // a warp an output where there are few rows (a decode step waits for the slowest warp); many rows fill the SMs with fewer
  const int most = n_rows <= 256 ? ROUTE_WARPS : 8;
  const dim3 threads(32 * (outputs < 4 ? 4 : outputs < most ? outputs : most));
  if (dtype == R2_F32) r2_launch(route_scored_kernel<float>, dim3(n_rows), threads, per_row, stream, a);
  else r2_launch(route_scored_kernel<bf16>, dim3(n_rows), threads, per_row, stream, a);
  return launch_status();
}

extern "C" int r2_expert_act(const void* gate_up, int in_stride, void* out, int out_stride, int n_rows, int inner, int kind,
                             float limit, float alpha, float up_offset, const float* route, int route_stride, int n_experts, int expert_width,
                             float tail_limit, const float* tail_gate, int tail_gate_stride, int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return R2_OK;
  if (inner < 1 || n_experts < 0 || (n_experts > 0 && (expert_width < 1 || route == nullptr || route_stride < n_experts || n_experts * expert_width > inner))) return R2_BAD_SHAPE;
  if (n_experts == 0) expert_width = 1;
  dim3 grid(n_rows, (inner + 1023) / 1024);
  if (dtype == R2_F32) {
    r2_launch(expert_act_kernel<float>, grid, dim3(256), size_t(0), stream, (const float*)gate_up, in_stride, (float*)out, out_stride, inner, kind,
              limit, alpha, up_offset, route, route_stride, n_experts, expert_width, tail_limit, tail_gate, tail_gate_stride);
  } else if (dtype == R2_BF16) {
    r2_launch(expert_act_kernel<bf16>, grid, dim3(256), size_t(0), stream, (const bf16*)gate_up, in_stride, (bf16*)out, out_stride, inner, kind,
              limit, alpha, up_offset, route, route_stride, n_experts, expert_width, tail_limit, tail_gate, tail_gate_stride);
  } else {
    return R2_BAD_DTYPE;
  }
  return launch_status();
}

// up and out [n_rows, inner] with inner = experts * expert_width; act one of the feed-forward activations; route float [n_rows, >= experts].
extern "C" int r2_expert_unit(const void* up, int in_stride, void* out, int out_stride, int n_rows, int inner, int act, const float* route,
                              int route_stride, int expert_width, int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return R2_OK;
  if (inner < 1 || expert_width < 1 || inner % expert_width != 0 || route == nullptr || route_stride < inner / expert_width) return R2_BAD_SHAPE;
  if (act < R2_ACT_NONE || act > R2_ACT_GELU_ERF) return R2_UNSUPPORTED;
  if (dtype == R2_F32) {
    r2_launch(expert_unit_kernel<float>, dim3(n_rows, (inner + 1023) / 1024), dim3(256), size_t(0), stream, (const float*)up, in_stride, (float*)out,
              out_stride, inner, act, route, route_stride, expert_width, 0);
  } else if (dtype == R2_BF16) {
    const bool vec = expert_width % 8 == 0 && in_stride % 8 == 0 && out_stride % 8 == 0 && !((reinterpret_cast<uintptr_t>(up) | reinterpret_cast<uintptr_t>(out)) & 15);
    r2_launch(expert_unit_kernel<bf16>, dim3(n_rows, vec ? (inner + 2047) / 2048 : (inner + 1023) / 1024), dim3(256), size_t(0), stream, (const bf16*)up,
              in_stride, (bf16*)out, out_stride, inner, act, route, route_stride, expert_width, int(vec));
  } else {
    return R2_BAD_DTYPE;
  }
  return launch_status();
}
