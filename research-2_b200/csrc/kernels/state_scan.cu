// Two recurrences over a matrix per head whose rows' vectors are prepared by a kernel of their own, so that the walk itself
// does nothing but load, multiply and add: the gated delta rule and time mixing with a decay per channel.
//
//   delta rule       S' = g S,  u = beta (v - S'^T k),  S = S' + k u^T,  o = S^T q         (q, k unit vectors, q scaled; g, beta per row)
//   time mixing      o = (S + diag(bonus) k v^T)^T r,   S <- diag(w) S + k v^T             (w per row and channel)
//
// S is [rows x cols] per head, float, in the request's slot, stored in pieces of four rows: [rows / 4][cols][4]. A CTA owns one (entry, head, slice of the columns), takes the state from
// the slot (or zeros for a sequence's first rows), walks the entry's rows in order and puts the state back. A thread keeps RPT
// rows of one column in registers, a column's rows are spread over G neighbouring lanes in pieces of four. The rows' vectors come
// through shared memory in tiles, copied asynchronously one tile ahead. The delta rule's write needs what the state returns for
// the row's key: S'^T k and S'^T q are summed side by side (o = S'^T q + (k . q) u), which leaves one round of shuffles a row on the
// chain. How a head's state is spread over lanes depends on its sizes alone, so a row's result is the same bits however its
// prompt was cut and whatever else is in the batch.
//
// All arithmetic is float; what is prepared is stored in float.
#include <math.h>

#include "common.cuh"
#include "small_products.cuh"

namespace {

constexpr int MODE_DELTA = 0, MODE_CHANNEL = 1;
constexpr int SCAN_STAGES = 2;

__device__ __forceinline__ float softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }

struct StateScanArgs {
  const void* read; long long read_stride; int read_group;    // q or r of group 0 in row 0; between rows, between groups (elements)
  const void* write; long long write_stride; int write_group; // k likewise
  const void* value; long long value_stride;                  // v [T, heads * cols]
  const float* decay; long long decay_stride;                 // time mixing: w [T, heads * rows]
  const float* bonus;                                         // time mixing: [heads * rows]
  const float4* row_numbers;                                  // delta rule: [T][heads] (g, beta, k . q, -)
  float* state; long long slot_stride; int head_stride;
  const int32_t* q_start; const int32_t* state_slot; const int32_t* fresh;
  float* out; int out_stride;
  int heads_per_group, rows, cols, G, cv;
  int tile;            // rows staged at a time
  int pieces;          // every row of every operand starts on a 16-byte boundary: asynchronous copies
  // the last keep_rows input rows (of the convolution, of the mixes) are state too: renewed here, spread over the entry's CTAs
  const void* keep_in; int keep_in_stride, keep_width, keep_rows, keep_is_bf16; long long keep_off;
};

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return uint32_t(__cvta_generic_to_shared(p)); }

// n elements of a row into shared memory, by the threads of the CTA from `first` on in steps of blockDim.x over (row, piece).
template <typename T>
__device__ __forceinline__ void stage_rows(T* dst, int dst_stride, const T* src, long long src_stride, int n, int n_rows, bool pieces) {
  constexpr int PER = 16 / int(sizeof(T));
  if (pieces) {
    const int per_row = n / PER;
    for (int i = threadIdx.x; i < per_row * n_rows; i += blockDim.x) {
      const int r = i / per_row, c = (i - r * per_row) * PER;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst + r * dst_stride + c)), "l"(src + r * src_stride + c) : "memory");
    }
  } else {
    for (int i = threadIdx.x; i < n * n_rows; i += blockDim.x) {
      const int r = i / n, c = i - r * n;
      dst[r * dst_stride + c] = src[r * src_stride + c];
    }
  }
}

// The newest keep_rows input rows of an entry: this step's, and before them what the slot held. Channel c is one thread's: it reads
// a place before it writes over it.
template <typename T>
__device__ __forceinline__ void keep_inputs(const StateScanArgs& a, float* slot, int row0, int row1, bool is_fresh, int part, int n_parts) {
  const T* in = static_cast<const T*>(a.keep_in);
  float* cs = slot + a.keep_off;
  const int n = row1 - row0;
  for (int c = part * blockDim.x + threadIdx.x; c < a.keep_width; c += n_parts * blockDim.x)
    for (int s = 0; s < a.keep_rows; ++s) {
      const int l = n - a.keep_rows + s;
      float val = 0.f;
      if (l >= 0) val = to_float(in[size_t(row0 + l) * a.keep_in_stride + c]);
      else if (!is_fresh) val = cs[size_t(s + n) * a.keep_width + c];
      cs[size_t(s) * a.keep_width + c] = val;
    }
}

// GL: the lanes of a column where they are fixed (8, 16, 32); 0: a.G of them.
template <typename T, int RPT, int GL, int MODE>
__global__ void __launch_bounds__(256, 1)
state_scan_kernel(const StateScanArgs a) {
  pdl_launch_dependents();
  // q_start, slots and fresh flags belong to the batch, which no kernel writes
  const int e = blockIdx.x, h = blockIdx.y;
  const int row0 = a.q_start[e], row1 = a.q_start[e + 1];
  if (row1 <= row0) {  // an entry without rows touches no slot
    pdl_wait();
    return;
  }
  const bool is_fresh = a.fresh[e] != 0;
  float* slot = a.state + size_t(a.state_slot[e]) * a.slot_stride;
  float* head_state = slot + size_t(h) * a.head_stride;
  extern __shared__ __align__(16) uint8_t scan_smem[];
  constexpr int Q = RPT / 4;
  const int G = GL > 0 ? GL : a.G, cv = a.cv, rows = a.rows, cols = a.cols, tile = a.tile;
  const int padded = RPT * G, cvp = (cv + 7) & ~7;
  // a stage: read vectors, write vectors, values, then decays (time mixing) or row numbers (delta rule)
  const int stage_bytes = tile * ((2 * padded + cvp) * int(sizeof(T)) + (MODE == MODE_CHANNEL ? padded : 4) * 4);
  const int tid = threadIdx.x, g = tid % G, jl = tid / G;
  const int j0 = blockIdx.z * cv, j = j0 + jl;
  // places that no copy ever fills: dimensions and columns beyond the head's, so that they multiply as zeros
  for (int i = tid; i < SCAN_STAGES * stage_bytes / 4; i += blockDim.x) reinterpret_cast<float*>(scan_smem)[i] = 0.f;
  pdl_wait();  // (the state may have been written by this layer's kernel of the step before)
  if (a.keep_in != nullptr) {
    const int part = h * gridDim.z + blockIdx.z, n_parts = gridDim.y * gridDim.z;
    if (a.keep_is_bf16) keep_inputs<bf16>(a, slot, row0, row1, is_fresh, part, n_parts);
    else keep_inputs<float>(a, slot, row0, row1, is_fresh, part, n_parts);
  }
  const int group = h / a.heads_per_group;
  const T* read = static_cast<const T*>(a.read) + size_t(group) * a.read_group;
  const T* write = static_cast<const T*>(a.write) + size_t(group) * a.write_group;
  const T* value = static_cast<const T*>(a.value) + size_t(h) * cols + j0;
  const int copy_cols = min(cv, cols - j0);
  __syncthreads();
  auto stage_at = [&](int s) { return scan_smem + s * stage_bytes; };
  auto issue = [&](int t0, int s) {
    const int nt = min(tile, row1 - t0);
    T* rs = reinterpret_cast<T*>(stage_at(s));
    const bool pieces = a.pieces != 0;
    stage_rows<T>(rs, padded, read + size_t(t0) * a.read_stride, a.read_stride, rows, nt, pieces);
    stage_rows<T>(rs + tile * padded, padded, write + size_t(t0) * a.write_stride, a.write_stride, rows, nt, pieces);
    if (copy_cols > 0) stage_rows<T>(rs + 2 * tile * padded, cvp, value + size_t(t0) * a.value_stride, a.value_stride, copy_cols, nt, pieces);
    float* fs = reinterpret_cast<float*>(rs + tile * (2 * padded + cvp));
    if (MODE == MODE_CHANNEL) {
      stage_rows<float>(fs, padded, a.decay + size_t(t0) * a.decay_stride + size_t(h) * rows, a.decay_stride, rows, nt, pieces);
    } else {
      stage_rows<float>(fs, 4, reinterpret_cast<const float*>(a.row_numbers + size_t(t0) * gridDim.y + h), 4 * (long long)gridDim.y, 4, nt, true);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  issue(row0, 0);

  // this thread's rows of its column: pieces of four, piece r4 starts at row (r4 * G + g) * 4
  float S[RPT];
  const int n_pieces = (rows + 3) >> 2;
#pragma unroll
  for (int r4 = 0; r4 < Q; ++r4) {
    const int piece = r4 * G + g;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!is_fresh && piece < n_pieces && j < cols) v = load4(head_state + (size_t(piece) * cols + j) * 4);
    S[r4 * 4] = v.x; S[r4 * 4 + 1] = v.y; S[r4 * 4 + 2] = v.z; S[r4 * 4 + 3] = v.w;
  }
  float bonus[MODE == MODE_CHANNEL ? RPT : 1];
  if (MODE == MODE_CHANNEL) {
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      const int i = ((r >> 2) * G + g) * 4 + (r & 3);
      bonus[r] = i < rows ? a.bonus[size_t(h) * rows + i] : 0.f;
    }
  }
  float* out = a.out + size_t(h) * cols + j;
  const bool writes = g == 0 && j < cols;

  int s = 0;
  for (int t0 = row0; t0 < row1; t0 += tile, s ^= 1) {
    const int nt = min(tile, row1 - t0);
    if (t0 + tile < row1) {
      issue(t0 + tile, s ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const T* rs = reinterpret_cast<const T*>(stage_at(s));
    const T* ws = rs + tile * padded;
    const T* vs = rs + 2 * tile * padded;
    const float* fs = reinterpret_cast<const float*>(rs + tile * (2 * padded + cvp));
    if (MODE == MODE_DELTA) {
      // the next row's vectors are fetched before this row's sums are waited for
      float4 k4[Q], q4[Q], kn[Q], qn[Q], num = load4(fs), num_n = num;
      float v = to_float(vs[jl]), v_n = v;
#pragma unroll
      for (int r4 = 0; r4 < Q; ++r4) {
        k4[r4] = load4(ws + (r4 * G + g) * 4);
        q4[r4] = load4(rs + (r4 * G + g) * 4);
      }
#pragma unroll 2
      for (int tt = 0; tt < nt; ++tt) {
        const int next = tt + 1 < nt ? tt + 1 : tt;
        num_n = load4(fs + next * 4);
        v_n = to_float(vs[next * cvp + jl]);
#pragma unroll
        for (int r4 = 0; r4 < Q; ++r4) {
          kn[r4] = load4(ws + next * padded + (r4 * G + g) * 4);
          qn[r4] = load4(rs + next * padded + (r4 * G + g) * 4);
        }
        float ak[4] = {0.f, 0.f, 0.f, 0.f}, aq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int r4 = 0; r4 < Q; ++r4) {
          const float k[4] = {k4[r4].x, k4[r4].y, k4[r4].z, k4[r4].w}, q[4] = {q4[r4].x, q4[r4].y, q4[r4].z, q4[r4].w};
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            S[r4 * 4 + u] *= num.x;
            ak[u] = fmaf(S[r4 * 4 + u], k[u], ak[u]);
            aq[u] = fmaf(S[r4 * 4 + u], q[u], aq[u]);
          }
        }
        float sk = (ak[0] + ak[1]) + (ak[2] + ak[3]), sq = (aq[0] + aq[1]) + (aq[2] + aq[3]);
#pragma unroll
        for (int o = G >> 1; o > 0; o >>= 1) {
          sk += __shfl_xor_sync(0xffffffffu, sk, o);
          sq += __shfl_xor_sync(0xffffffffu, sq, o);
        }
        const float u_row = num.y * (v - sk);
        if (writes) out[size_t(t0 + tt) * a.out_stride] = fmaf(num.z, u_row, sq);
#pragma unroll
        for (int r4 = 0; r4 < Q; ++r4) {
          const float k[4] = {k4[r4].x, k4[r4].y, k4[r4].z, k4[r4].w};
#pragma unroll
          for (int u = 0; u < 4; ++u) S[r4 * 4 + u] = fmaf(u_row, k[u], S[r4 * 4 + u]);
          k4[r4] = kn[r4];
          q4[r4] = qn[r4];
        }
        num = num_n;
        v = v_n;
      }
    } else {
      auto one_row = [&](int tt) {   // -> this lane's share of the row's output
        const float v = to_float(vs[tt * cvp + jl]);
        float acc[2] = {0.f, 0.f}, own[2] = {0.f, 0.f};
#pragma unroll
        for (int r4 = 0; r4 < Q; ++r4) {
          const int at = tt * padded + (r4 * G + g) * 4;
          const float4 q4 = load4(rs + at), k4 = load4(ws + at), w4 = load4(fs + at);
          const float q[4] = {q4.x, q4.y, q4.z, q4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w}, w[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            const int r = r4 * 4 + u;
            acc[u & 1] = fmaf(S[r], q[u], acc[u & 1]);            // the state before this row's write
            own[u & 1] = fmaf(bonus[r] * k[u], q[u], own[u & 1]); // the row's own write, times its bonus
            S[r] = fmaf(w[u], S[r], k[u] * v);
          }
        }
        return fmaf(own[0] + own[1], v, acc[0] + acc[1]);
      };
      int tt = 0;
      for (; tt + 4 <= nt; tt += 4) {   // four rows' sums over the lanes at a time: their shuffles overlap
        float y[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) y[i] = one_row(tt + i);
#pragma unroll
        for (int o = G >> 1; o > 0; o >>= 1) {
#pragma unroll
          for (int i = 0; i < 4; ++i) y[i] += __shfl_xor_sync(0xffffffffu, y[i], o);
        }
        if (writes) {
#pragma unroll
          for (int i = 0; i < 4; ++i) out[size_t(t0 + tt + i) * a.out_stride] = y[i];
        }
      }
      for (; tt < nt; ++tt) {
        float y = one_row(tt);
        for (int o = G >> 1; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
        if (writes) out[size_t(t0 + tt) * a.out_stride] = y;
      }
    }
    __syncthreads();  // the stage may be filled again
  }
#pragma unroll
  for (int r4 = 0; r4 < Q; ++r4) {
    const int piece = r4 * G + g;
    if (piece < n_pieces && j < cols)
      *reinterpret_cast<float4*>(head_state + (size_t(piece) * cols + j) * 4) = make_float4(S[r4 * 4], S[r4 * 4 + 1], S[r4 * 4 + 2], S[r4 * 4 + 3]);
  }
}

// The same for launches in which (nearly) every entry is one row, a decode step: nothing is staged, every thread asks for its part
// of the state and of the row at once. The arithmetic and its order are the walk's.
template <typename T, int RPT, int GL, int MODE>
__global__ void __launch_bounds__(256)
state_step_kernel(const StateScanArgs a) {
  pdl_launch_dependents();
  const int e = blockIdx.x, h = blockIdx.y;
  const int row0 = a.q_start[e], row1 = a.q_start[e + 1];
  if (row1 <= row0) {
    pdl_wait();
    return;
  }
  const bool is_fresh = a.fresh[e] != 0;
  float* slot = a.state + size_t(a.state_slot[e]) * a.slot_stride;
  float* head_state = slot + size_t(h) * a.head_stride;
  constexpr int Q = RPT / 4;
  const int G = GL > 0 ? GL : a.G, cv = a.cv, rows = a.rows, cols = a.cols;
  const int tid = threadIdx.x, g = tid % G, j = blockIdx.z * cv + tid / G;
  const int n_pieces = (rows + 3) >> 2, group = h / a.heads_per_group;
  const bool has_column = j < cols;
  pdl_wait();
  float S[RPT];
#pragma unroll
  for (int r4 = 0; r4 < Q; ++r4) {
    const int piece = r4 * G + g;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!is_fresh && piece < n_pieces && has_column) v = load4(head_state + (size_t(piece) * cols + j) * 4);
    S[r4 * 4] = v.x; S[r4 * 4 + 1] = v.y; S[r4 * 4 + 2] = v.z; S[r4 * 4 + 3] = v.w;
  }
  // four numbers of a row from dimension i on, zeros after the last
  auto row4 = [&](const auto* p, int i) {
    if (a.pieces) return i < rows ? load4(p + i) : make_float4(0.f, 0.f, 0.f, 0.f);
    return make_float4(i < rows ? to_float(p[i]) : 0.f, i + 1 < rows ? to_float(p[i + 1]) : 0.f, i + 2 < rows ? to_float(p[i + 2]) : 0.f,
                       i + 3 < rows ? to_float(p[i + 3]) : 0.f);
  };
  for (int t = row0; t < row1; ++t) {
    const T* read = static_cast<const T*>(a.read) + size_t(t) * a.read_stride + size_t(group) * a.read_group;
    const T* write = static_cast<const T*>(a.write) + size_t(t) * a.write_stride + size_t(group) * a.write_group;
    const float v = has_column ? to_float(static_cast<const T*>(a.value)[size_t(t) * a.value_stride + size_t(h) * cols + j]) : 0.f;
    float y;
    if (MODE == MODE_DELTA) {
      const float4 num = a.row_numbers[size_t(t) * gridDim.y + h];
      float ak[4] = {0.f, 0.f, 0.f, 0.f}, aq[4] = {0.f, 0.f, 0.f, 0.f};
      float4 k4[Q];
#pragma unroll
      for (int r4 = 0; r4 < Q; ++r4) {
        k4[r4] = row4(write, (r4 * G + g) * 4);
        const float4 q4 = row4(read, (r4 * G + g) * 4);
        const float k[4] = {k4[r4].x, k4[r4].y, k4[r4].z, k4[r4].w}, q[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          S[r4 * 4 + u] *= num.x;
          ak[u] = fmaf(S[r4 * 4 + u], k[u], ak[u]);
          aq[u] = fmaf(S[r4 * 4 + u], q[u], aq[u]);
        }
      }
      float sk = (ak[0] + ak[1]) + (ak[2] + ak[3]), sq = (aq[0] + aq[1]) + (aq[2] + aq[3]);
#pragma unroll
      for (int o = G >> 1; o > 0; o >>= 1) {
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
      }
      const float u_row = num.y * (v - sk);
      y = fmaf(num.z, u_row, sq);
#pragma unroll
      for (int r4 = 0; r4 < Q; ++r4) {
        const float k[4] = {k4[r4].x, k4[r4].y, k4[r4].z, k4[r4].w};
#pragma unroll
        for (int u = 0; u < 4; ++u) S[r4 * 4 + u] = fmaf(u_row, k[u], S[r4 * 4 + u]);
      }
    } else {
      const float* decay = a.decay + size_t(t) * a.decay_stride + size_t(h) * rows;
      const float* bonus = a.bonus + size_t(h) * rows;
      float acc[2] = {0.f, 0.f}, own[2] = {0.f, 0.f};
#pragma unroll
      for (int r4 = 0; r4 < Q; ++r4) {
        const int i = (r4 * G + g) * 4;
        const float4 q4 = row4(read, i), k4 = row4(write, i), w4 = row4(decay, i);
        const float q[4] = {q4.x, q4.y, q4.z, q4.w}, k[4] = {k4.x, k4.y, k4.z, k4.w}, w[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const int r = r4 * 4 + u;
          acc[u & 1] = fmaf(S[r], q[u], acc[u & 1]);
          own[u & 1] = fmaf((i + u < rows ? bonus[i + u] : 0.f) * k[u], q[u], own[u & 1]);
          S[r] = fmaf(w[u], S[r], k[u] * v);
        }
      }
      y = fmaf(own[0] + own[1], v, acc[0] + acc[1]);
#pragma unroll
      for (int o = G >> 1; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    }
    if (g == 0 && has_column) a.out[size_t(t) * a.out_stride + size_t(h) * cols + j] = y;
  }
#pragma unroll
  for (int r4 = 0; r4 < Q; ++r4) {
    const int piece = r4 * G + g;
    if (piece < n_pieces && has_column)
      *reinterpret_cast<float4*>(head_state + (size_t(piece) * cols + j) * 4) = make_float4(S[r4 * 4], S[r4 * 4 + 1], S[r4 * 4 + 2], S[r4 * 4 + 3]);
  }
  if (a.keep_in != nullptr) {
    const int part = h * gridDim.z + blockIdx.z, n_parts = gridDim.y * gridDim.z;
    if (a.keep_is_bf16) keep_inputs<bf16>(a, slot, row0, row1, is_fresh, part, n_parts);
    else keep_inputs<float>(a, slot, row0, row1, is_fresh, part, n_parts);
  }
}

// How a head's state is spread: RPT rows a thread and G lanes a column by the state's sizes alone; cv columns a CTA so that a
// launch has a CTA for every SM where the columns allow it, and no CTA more than 256 threads.
template <typename T, int MODE>
int launch_state_scan(const StateScanArgs& in, int n_entries, int n_heads, int single_rows, int n_sms, cudaStream_t stream) {
  StateScanArgs a = in;
  const int rpt = a.rows <= 32 ? 4 : (a.rows <= 64 ? 8 : (a.rows <= 512 ? 16 : 32));
  a.G = 1;
  while (a.G * rpt < a.rows) a.G *= 2;
  if (a.G > 32) return R2_UNSUPPORTED;
  // (columns are cut at whole warps and at whole 16-byte pieces of the values)
  const int per_warp = 32 / a.G, granule = 16 / int(sizeof(T)) > per_warp ? 16 / int(sizeof(T)) : per_warp;
  int splits = 1;
  for (;; splits *= 2) {
    const int unit = splits == 1 ? per_warp : granule, want = (a.cols + splits - 1) / splits;
    a.cv = (want + unit - 1) / unit * unit;
    const long long ctas = (long long)n_entries * n_heads * ((a.cols + a.cv - 1) / a.cv);
    if (a.cv * a.G <= 256 && (ctas >= n_sms || a.cv <= granule)) break;
    if (splits > a.cols) return R2_UNSUPPORTED;
  }
  splits = (a.cols + a.cv - 1) / a.cv;
  const int threads = a.cv * a.G;
  const int padded = rpt * a.G, cvp = (a.cv + 7) & ~7;
  const size_t per_row = size_t(2 * padded + cvp) * sizeof(T) + size_t(MODE == MODE_CHANNEL ? padded : 4) * 4;
  int tile = 32;
  while (tile > 1 && SCAN_STAGES * tile * per_row > 100 * 1024) tile /= 2;
  a.tile = tile;
  const size_t smem = SCAN_STAGES * tile * per_row;
  dim3 grid(n_entries, n_heads, splits);
#define R2_STATE_SCAN(RPT_, GL_)                                                               \
  do {                                                                                         \
    if (single_rows) {                                                                         \
      r2_launch(state_step_kernel<T, RPT_, GL_, MODE>, grid, dim3(threads), 0, stream, a);     \
    } else {                                                                                   \
      if (!room_for(state_scan_kernel<T, RPT_, GL_, MODE>, smem)) return R2_UNSUPPORTED;       \
      r2_launch(state_scan_kernel<T, RPT_, GL_, MODE>, grid, dim3(threads), smem, stream, a);  \
    }                                                                                          \
  } while (0)
  if (rpt == 4 && a.G == 8) R2_STATE_SCAN(4, 8);
  else if (rpt == 4) R2_STATE_SCAN(4, 0);
  else if (rpt == 8) R2_STATE_SCAN(8, 8);
  else if (rpt == 16 && a.G == 8) R2_STATE_SCAN(16, 8);
  else if (rpt == 16 && a.G == 16) R2_STATE_SCAN(16, 16);
  else if (rpt == 16) R2_STATE_SCAN(16, 32);
  else R2_STATE_SCAN(32, 32);
#undef R2_STATE_SCAN
  return launch_status();
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

// ---- what the delta rule walks over --------------------------------------------------------------
// Per row: the short causal convolution and silu of q, k and v (inputs of positions before this step from the slot, zeros before a
// sequence's start), q and k made unit vectors (q times a scale), the decay g and the write strength beta from two small float
// products with the layer's input, and k . q of the unit vectors. A CTA takes ROWS rows. qk [T][groups][2][dim4] float (q, then k; dim4 =
// dim rounded up to 4, zeros after dim), v_out [T][heads * vdim] float, numbers [T][heads] (g, beta, k . q, 0). The slot is only read.
struct DeltaPrepareArgs {
  const void* in; int in_stride;              // [T, 2 groups dim + heads vdim]: the projections of q, k, v
  const void* h; int h_stride, width;         // [T, width]: the layer's input
  const float* taps; int n_taps;              // [channels][n_taps]
  const void* w_gates;                        // [2 heads][width] (dtype): write strengths, then step sizes
  const float* step_bias; const float* log_rate;
  float q_scale, unit_eps;
  int heads, groups, dim, vdim, n_rows;
  float* qk; float* v_out; float4* numbers;
  const float* state; long long slot_stride, conv_off;
  const int32_t* row_entry; const int32_t* q_start; const int32_t* state_slot; const int32_t* fresh;
};

constexpr int PREP_THREADS = 512;

template <typename T, int ROWS>
__global__ void __launch_bounds__(PREP_THREADS)
delta_prepare_kernel(const DeltaPrepareArgs a) {
  pdl_launch_dependents();
  const int t0 = blockIdx.x * ROWS;
  __shared__ int entry_row[ROWS];             // the row's place in its entry this step; -1: no row of an entry
  __shared__ const float* kept[ROWS];         // the slot's kept inputs, or null for a sequence's first rows
  if (threadIdx.x < ROWS) {
    const int t = t0 + int(threadIdx.x), e = t < a.n_rows ? a.row_entry[t] : -1;
    entry_row[threadIdx.x] = e >= 0 ? t - a.q_start[e] : -1;
    kept[threadIdx.x] = (e >= 0 && a.fresh[e] == 0) ? a.state + size_t(a.state_slot[e]) * a.slot_stride + a.conv_off : nullptr;
  }
  extern __shared__ __align__(16) float prep_smem[];
  const int qk_width = 2 * a.groups * a.dim, channels = qk_width + a.heads * a.vdim, wpad = (a.width + 3) & ~3;
  float* rows_h = prep_smem;                        // [ROWS][wpad]
  float* conv = rows_h + ROWS * wpad;               // [ROWS][qk_width]
  float* gates = conv + ROWS * qk_width;            // [ROWS][2 heads]
  float* products = gates + ROWS * 2 * a.heads;     // [ROWS][groups]
  pdl_wait();
  __syncthreads();
  const T* in = static_cast<const T*>(a.in);
  const T* h = static_cast<const T*>(a.h);
  for (int i = threadIdx.x; i < ROWS * wpad; i += PREP_THREADS) {
    const int r = i / wpad, c = i - r * wpad;
    rows_h[i] = (c < a.width && entry_row[r] >= 0) ? to_float(h[size_t(t0 + r) * a.h_stride + c]) : 0.f;
  }
  // four taps and rows that all lie inside one entry behind its first three: every input is a row of this step
  const bool inside = ROWS > 1 && a.n_taps == 4 && entry_row[0] >= 3 && entry_row[ROWS - 1] == entry_row[0] + ROWS - 1;
  for (int c = threadIdx.x; c < channels; c += PREP_THREADS) {
    float acc[ROWS];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) acc[r] = 0.f;
    if (inside) {
      float x[ROWS + 3];
#pragma unroll
      for (int r = 0; r < ROWS + 3; ++r) x[r] = to_float(in[size_t(t0 + r - 3) * a.in_stride + c]);
      float tap[4];
#pragma unroll
      for (int d = 0; d < 4; ++d) tap[d] = a.taps[size_t(c) * 4 + d];
#pragma unroll
      for (int r = 0; r < ROWS; ++r)
#pragma unroll
        for (int d = 0; d < 4; ++d) acc[r] = fmaf(tap[d], x[r + d], acc[r]);
    } else for (int d = 0; d < a.n_taps; ++d) {
      const float tap = a.taps[size_t(c) * a.n_taps + d];
      const int back = a.n_taps - 1 - d;
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        const int src = entry_row[r] - back;
        float val = 0.f;
        if (entry_row[r] >= 0) {
          if (src >= 0) val = to_float(in[size_t(t0 + r - back) * a.in_stride + c]);
          else if (kept[r] != nullptr) val = kept[r][size_t(a.n_taps - 1 + src) * channels + c];
        }
        acc[r] = fmaf(tap, val, acc[r]);
      }
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      const float y = silu(acc[r]);
      if (c < qk_width) conv[r * qk_width + c] = y;
      else if (t0 + r < a.n_rows) a.v_out[size_t(t0 + r) * (channels - qk_width) + (c - qk_width)] = y;
    }
  }
  __syncthreads();
  rows_times_matrix<ROWS, (ROWS > 1 ? 2 : 1)>(rows_h, wpad, static_cast<const T*>(a.w_gates), a.width, 2 * a.heads, [&](int r, int n, float sum) { gates[r * 2 * a.heads + n] = sum; });
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, dim4 = (a.dim + 3) & ~3;
  for (int unit = warp; unit < ROWS * a.groups; unit += PREP_THREADS / 32) {   // a warp per row and group
    const int r = unit / a.groups, grp = unit - r * a.groups;
    const float* q = conv + r * qk_width + grp * a.dim;
    const float* k = q + a.groups * a.dim;
    float qq = 0.f, kk = 0.f, kq = 0.f;
    for (int i = lane; i < a.dim; i += 32) {
      qq = fmaf(q[i], q[i], qq);
      kk = fmaf(k[i], k[i], kk);
      kq = fmaf(k[i], q[i], kq);
    }
    qq = warp_sum(qq);
    kk = warp_sum(kk);
    kq = warp_sum(kq);
    const float qn = a.q_scale / sqrtf(qq + a.unit_eps), kn = 1.f / sqrtf(kk + a.unit_eps);
    if (t0 + r < a.n_rows) {
      float* o = a.qk + (size_t(t0 + r) * a.groups + grp) * 2 * dim4;
      for (int i = lane; i < dim4; i += 32) {
        o[i] = i < a.dim ? q[i] * qn : 0.f;
        o[dim4 + i] = i < a.dim ? k[i] * kn : 0.f;
      }
    }
    if (lane == 0) products[r * a.groups + grp] = kq * kn * qn;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < ROWS * a.heads; i += PREP_THREADS) {
    const int r = i / a.heads, hd = i - r * a.heads;
    if (t0 + r >= a.n_rows) continue;
    const float* gr = gates + r * 2 * a.heads;
    const float step = softplus(gr[a.heads + hd] + a.step_bias[hd]);
    a.numbers[size_t(t0 + r) * a.heads + hd] =
        make_float4(expf(-expf(a.log_rate[hd]) * step), 1.f / (1.f + expf(-gr[hd])), products[r * a.groups + hd / (a.heads / a.groups)], 0.f);
  }
}

// ---- what time mixing walks over -----------------------------------------------------------------
// Mix s of row t: h + (h' - h) * mu[s], h' the row before it in its sequence: the row above inside the entry, the slot's row for
// an entry's first (zeros for a sequence's first). Mixes 0 .. n_mixes - 1 go to out [T][n_mixes][width] in the rows' dtype. One
// more, with mu[n_mixes], stays in float in shared memory and becomes the row's decays on the spot:
//
//     decay[t] = exp(-exp(w0 + W2 tanh(W1 mix)))       W1 [rank][width], W2 stored transposed [rank][n_out], sums in float
//
// A CTA takes ROWS rows, so that the two small matrices come out of L2 once for all of them; in the second product a thread has one
// column of every row. A row's sums are made in the same order whatever ROWS is. The slot is only read.
struct TimeMixPrepareArgs {
  const void* h; int h_stride, width, n_rows;
  const float* mu; int n_mixes; void* out;
  const void* w1; const void* w2t; const float* w0; int rank, n_out; float* decay;   // both matrices in the dtype
  const float* state; long long slot_stride, row_off;
  const int32_t* row_entry; const int32_t* q_start; const int32_t* state_slot; const int32_t* fresh;
};

template <typename T, int ROWS>
__global__ void __launch_bounds__(PREP_THREADS)
time_mix_prepare_kernel(const TimeMixPrepareArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float prep_smem[];
  const int width = a.width, wpad = (width + 3) & ~3, rpad = (a.rank + 3) & ~3;
  float* mix = prep_smem;              // [ROWS][wpad], zeros after the width
  float* low = mix + ROWS * wpad;      // [ROWS][rpad], zeros after the rank
  const int t0 = blockIdx.x * ROWS;
  __shared__ int kind[ROWS];               // 0: no row of an entry; 1: the row above is the row before; 2: a sequence's first; 3: kept in the slot
  __shared__ const float* kept_row[ROWS];
  if (threadIdx.x < ROWS) {
    const int t = t0 + int(threadIdx.x), e = t < a.n_rows ? a.row_entry[t] : -1;
    const bool first = e >= 0 && t == a.q_start[e];
    kind[threadIdx.x] = e < 0 ? 0 : (!first ? 1 : (a.fresh[e] != 0 ? 2 : 3));
    kept_row[threadIdx.x] = e >= 0 ? a.state + size_t(a.state_slot[e]) * a.slot_stride + a.row_off : nullptr;
  }
  for (int i = threadIdx.x; i < ROWS * rpad; i += PREP_THREADS) low[i] = 0.f;
  pdl_wait();
  __syncthreads();
  const T* h = static_cast<const T*>(a.h);
  T* out = static_cast<T*>(a.out);
  // (with few rows several CTAs share them: each makes the whole inner row, and its share of the mixes and of the columns)
  const int share = blockIdx.y, n_shares = gridDim.y;
  for (int c = threadIdx.x; c < wpad; c += PREP_THREADS) {
    const bool inside = c < width;
    float now[ROWS + 1], step[ROWS];   // now[r + 1]: row t0 + r; now[0]: the row above the first
    now[0] = (inside && kind[0] == 1) ? to_float(h[size_t(t0 - 1) * a.h_stride + c]) : 0.f;
#pragma unroll
    for (int r = 0; r < ROWS; ++r) now[r + 1] = (inside && kind[r] != 0) ? to_float(h[size_t(t0 + r) * a.h_stride + c]) : 0.f;
#pragma unroll
    for (int r = 0; r < ROWS; ++r) step[r] = (kind[r] == 1 ? now[r] : ((inside && kind[r] == 3) ? kept_row[r][c] : 0.f)) - now[r + 1];
    for (int s = share; s < a.n_mixes; s += n_shares) {
      const float m = inside ? a.mu[size_t(s) * width + c] : 0.f;
#pragma unroll
      for (int r = 0; r < ROWS; ++r)
        if (inside && t0 + r < a.n_rows) out[(size_t(t0 + r) * a.n_mixes + s) * width + c] = from_float<T>(fmaf(step[r], m, now[r + 1]));
    }
    const float m = inside ? a.mu[size_t(a.n_mixes) * width + c] : 0.f;
#pragma unroll
    for (int r = 0; r < ROWS; ++r) mix[r * wpad + c] = fmaf(step[r], m, now[r + 1]);
  }
  __syncthreads();
  rows_times_matrix<ROWS, 4>(mix, wpad, static_cast<const T*>(a.w1), width, a.rank, [&](int r, int n, float sum) { low[r * rpad + n] = tanhf(sum); });
  __syncthreads();
  for (int n = share * PREP_THREADS + threadIdx.x; n < a.n_out; n += n_shares * PREP_THREADS) {
    float acc[ROWS];
    const T* w2t = static_cast<const T*>(a.w2t);
    const float start = a.w0[n];
#pragma unroll
    for (int r = 0; r < ROWS; ++r) acc[r] = start;
#pragma unroll (ROWS == 1 ? 16 : 4)
    for (int i = 0; i < rpad; i += 4) {
      float w[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) w[u] = i + u < a.rank ? to_float(w2t[size_t(i + u) * a.n_out + n]) : 0.f;
#pragma unroll
      for (int r = 0; r < ROWS; ++r) {
        const float4 l = *reinterpret_cast<const float4*>(low + r * rpad + i);
        acc[r] = fmaf(l.w, w[3], fmaf(l.z, w[2], fmaf(l.y, w[1], fmaf(l.x, w[0], acc[r]))));
      }
    }
#pragma unroll
    for (int r = 0; r < ROWS; ++r)
      if (t0 + r < a.n_rows) a.decay[size_t(t0 + r) * a.n_out + n] = expf(-expf(acc[r]));
  }
}

// Rows a CTA of a preparing kernel: more while every SM still has one, and as many as fit.
int rows_per_cta(int n_rows, int n_sms, size_t per_row) {
  int rows = n_rows > 4 * n_sms ? 8 : (n_rows > n_sms ? 4 : 1);
  while (rows > 1 && per_row * rows > 200 * 1024) rows = rows == 8 ? 4 : 1;
  return rows;
}

#define R2_PREPARE(KERNEL_, T_, ROWS_)                                                                                                  \
  do {                                                                                                                                  \
    if (!room_for(KERNEL_<T_, ROWS_>, per_row * ROWS_)) return R2_UNSUPPORTED;                                                          \
    r2_launch(KERNEL_<T_, ROWS_>, dim3((a.n_rows + ROWS_ - 1) / ROWS_, shares), dim3(PREP_THREADS), per_row * ROWS_, stream, a);        \
  } while (0)
#define R2_PREPARE_ROWS(KERNEL_, T_)                \
  do {                                              \
    if (rows == 8) R2_PREPARE(KERNEL_, T_, 8);      \
    else if (rows == 4) R2_PREPARE(KERNEL_, T_, 4); \
    else R2_PREPARE(KERNEL_, T_, 1);                \
  } while (0)

}  // namespace

// in [T, 2 groups dim + heads vdim], h [T, width], w_gates [2 heads, width] (dtype); everything else float: see DeltaPrepareArgs.
extern "C" int r2_delta_prepare(const void* in, int in_stride, const void* h, int h_stride, int width, const float* taps, int n_taps,
                                const void* w_gates, const float* step_bias, const float* log_rate, float q_scale, float unit_eps, int n_heads,
                                int n_groups, int dim, int vdim, int n_rows, float* qk, float* v_out, float* numbers, const float* state,
                                long long slot_stride, long long conv_off, const int32_t* row_entry, const int32_t* q_start,
                                const int32_t* state_slot, const int32_t* fresh, int n_sms, int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return R2_OK;
  if (n_heads < 1 || n_groups < 1 || n_heads % n_groups != 0 || dim < 1 || vdim < 1 || n_taps < 1 || width < 1 || n_sms < 1) return R2_BAD_SHAPE;
  if (!aligned16(numbers)) return R2_BAD_ALIGN;
  DeltaPrepareArgs a;
  a.in = in; a.in_stride = in_stride; a.h = h; a.h_stride = h_stride; a.width = width; a.taps = taps; a.n_taps = n_taps; a.w_gates = w_gates;
  a.step_bias = step_bias; a.log_rate = log_rate; a.q_scale = q_scale; a.unit_eps = unit_eps; a.heads = n_heads; a.groups = n_groups;
  a.dim = dim; a.vdim = vdim; a.n_rows = n_rows; a.qk = qk; a.v_out = v_out; a.numbers = reinterpret_cast<float4*>(numbers);
  a.state = state; a.slot_stride = slot_stride; a.conv_off = conv_off;
  a.row_entry = row_entry; a.q_start = q_start; a.state_slot = state_slot; a.fresh = fresh;
  const size_t per_row = sizeof(float) * (size_t((width + 3) & ~3) + size_t(2) * n_groups * dim + 2 * n_heads + n_groups);
  const int rows = rows_per_cta(n_rows, n_sms, per_row), shares = 1;
  if (dtype == R2_F32) R2_PREPARE_ROWS(delta_prepare_kernel, float);
  else if (dtype == R2_BF16) R2_PREPARE_ROWS(delta_prepare_kernel, bf16);
  else return R2_BAD_DTYPE;
  return launch_status();
}

// The delta rule over what r2_delta_prepare made. State per slot: S [heads][dim / 4 rounded up][vdim][4] and, at conv_off, the convolution's last
// n_taps - 1 inputs, renewed here from conv_in [T, channels] (in_dtype). out [T, heads * vdim] float, the heads' outputs before their norm.
extern "C" int r2_delta_scan(const float* qk, const float* v, const float* numbers, float* state, long long slot_stride, const int32_t* q_start,
                             const int32_t* state_slot, const int32_t* fresh, int n_entries, float* out, int out_stride, int n_heads, int n_groups,
                             int dim, int vdim, const void* conv_in, int conv_in_stride, int conv_channels, int n_taps, long long conv_off,
                             int in_dtype, int single_rows, int n_sms, cudaStream_t stream) {
  if (n_entries <= 0) return R2_OK;
  if (n_heads < 1 || n_groups < 1 || n_heads % n_groups != 0 || dim < 1 || vdim < 1 || n_sms < 1) return R2_BAD_SHAPE;
  if (in_dtype != R2_F32 && in_dtype != R2_BF16) return R2_BAD_DTYPE;
  if (!aligned16(qk) || !aligned16(numbers) || !aligned16(state) || slot_stride % 4 != 0) return R2_BAD_ALIGN;
  const int dim4 = (dim + 3) & ~3;
  StateScanArgs a = {};
  a.read = qk; a.read_stride = (long long)n_groups * 2 * dim4; a.read_group = 2 * dim4;
  a.write = qk + dim4; a.write_stride = a.read_stride; a.write_group = 2 * dim4;
  a.value = v; a.value_stride = (long long)n_heads * vdim; a.row_numbers = reinterpret_cast<const float4*>(numbers);
  a.state = state; a.slot_stride = slot_stride; a.head_stride = dim4 * vdim; a.q_start = q_start; a.state_slot = state_slot; a.fresh = fresh;
  a.out = out; a.out_stride = out_stride; a.heads_per_group = n_heads / n_groups; a.rows = dim; a.cols = vdim;
  a.pieces = dim % 4 == 0 && vdim % 4 == 0 && aligned16(v);
  a.keep_in = n_taps > 1 ? conv_in : nullptr; a.keep_in_stride = conv_in_stride; a.keep_width = conv_channels; a.keep_rows = n_taps - 1;
  a.keep_is_bf16 = in_dtype == R2_BF16; a.keep_off = conv_off;
  return launch_state_scan<float, MODE_DELTA>(a, n_entries, n_heads, single_rows, n_sms, stream);
}

// h [T, width], w1, w2t, out [T][n_mixes][width] (dtype); mu float [n_mixes + 1][width]; decay float [T][n_out]: see TimeMixPrepareArgs.
extern "C" int r2_time_mix_prepare(const void* h, int h_stride, const float* mu, int n_mixes, void* out, int n_rows, int width, const void* w1,
                                   const void* w2t, const float* w0, int rank, int n_out, float* decay, const float* state,
                                   long long slot_stride, long long row_off, const int32_t* row_entry, const int32_t* q_start,
                                   const int32_t* state_slot, const int32_t* fresh, int n_sms, int dtype, cudaStream_t stream) {
  if (n_rows <= 0) return R2_OK;
  if (width < 1 || n_mixes < 0 || rank < 1 || n_out < 1 || n_sms < 1) return R2_BAD_SHAPE;
  TimeMixPrepareArgs a;
  a.h = h; a.h_stride = h_stride; a.width = width; a.n_rows = n_rows; a.mu = mu; a.n_mixes = n_mixes; a.out = out;
  a.w1 = w1; a.w2t = w2t; a.w0 = w0; a.rank = rank; a.n_out = n_out; a.decay = decay; a.state = state; a.slot_stride = slot_stride;
  a.row_off = row_off; a.row_entry = row_entry; a.q_start = q_start; a.state_slot = state_slot; a.fresh = fresh;
  const size_t per_row = sizeof(float) * (size_t((width + 3) & ~3) + ((rank + 3) & ~3));
  const int rows = rows_per_cta(n_rows, n_sms, per_row), column_blocks = (n_out + PREP_THREADS - 1) / PREP_THREADS;
  const int shares = 2 * n_rows > n_sms ? 1 : (column_blocks < 4 ? column_blocks : 4);
  if (dtype == R2_F32) R2_PREPARE_ROWS(time_mix_prepare_kernel, float);
  else if (dtype == R2_BF16) R2_PREPARE_ROWS(time_mix_prepare_kernel, bf16);
  else return R2_BAD_DTYPE;
  return launch_status();
}

// Time mixing: o_t = (S_(t-1) + diag(bonus) k_t v_t^T)^T r_t, S_t = diag(decay_t) S_(t-1) + k_t v_t^T. r, k, v [T, heads * dim] (dtype, row
// strides); decay float [T, heads * dim]; bonus float [heads * dim]. State per slot: S [heads][dim / 4 rounded up][dim][4] and, at row_off, the input row of
// the sequence's last position [row_width], renewed here from row_in [T, row_width] (dtype). out [T, heads * dim] float.
extern "C" int r2_time_mix_scan(const void* r, int r_stride, const void* k, int k_stride, const void* v, int v_stride, const float* decay,
                                int decay_stride, const float* bonus, float* state, long long slot_stride, const int32_t* q_start,
                                const int32_t* state_slot, const int32_t* fresh, int n_entries, float* out, int out_stride, int n_heads, int dim,
                                const void* row_in, int row_in_stride, int row_width, long long row_off, int single_rows, int n_sms, int dtype,
                                cudaStream_t stream) {
  if (n_entries <= 0) return R2_OK;
  if (n_heads < 1 || dim < 1 || n_sms < 1) return R2_BAD_SHAPE;
  if (dtype != R2_F32 && dtype != R2_BF16) return R2_BAD_DTYPE;
  if (!aligned16(state) || slot_stride % 4 != 0) return R2_BAD_ALIGN;
  const int per = dtype == R2_BF16 ? 8 : 4;
  StateScanArgs a = {};
  a.read = r; a.read_stride = r_stride; a.read_group = dim; a.write = k; a.write_stride = k_stride; a.write_group = dim;
  a.value = v; a.value_stride = v_stride; a.decay = decay; a.decay_stride = decay_stride; a.bonus = bonus;
  a.state = state; a.slot_stride = slot_stride; a.head_stride = ((dim + 3) & ~3) * dim; a.q_start = q_start; a.state_slot = state_slot; a.fresh = fresh;
  a.out = out; a.out_stride = out_stride; a.heads_per_group = 1; a.rows = dim; a.cols = dim;
  a.pieces = dim % per == 0 && r_stride % per == 0 && k_stride % per == 0 && v_stride % per == 0 && decay_stride % 4 == 0 && aligned16(r) &&
             aligned16(k) && aligned16(v) && aligned16(decay);
  a.keep_in = row_in; a.keep_in_stride = row_in_stride; a.keep_width = row_width; a.keep_rows = 1; a.keep_is_bf16 = dtype == R2_BF16; a.keep_off = row_off;
  if (dtype == R2_F32) return launch_state_scan<float, MODE_CHANNEL>(a, n_entries, n_heads, single_rows, n_sms, stream);
  return launch_state_scan<bf16, MODE_CHANNEL>(a, n_entries, n_heads, single_rows, n_sms, stream);
}
