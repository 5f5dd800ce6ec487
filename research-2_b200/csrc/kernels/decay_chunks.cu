// Linear attention with one fixed decay per head over prompts, in chunks of 64 rows instead of row by row:
//
//     S_t = decay S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t          (S: [dim x vdim] per head, from the request's slot or zero)
//
// For a chunk that starts with the state S and rows i, j = 0, 1, .. of it:
//
//     o_i = decay^(i + 1) S^T q_i + sum over j <= i of decay^(i - j) (q_i . k_j) v_j
//     state after n rows = decay^n S + U,   U = sum over j of decay^(n - 1 - j) k_j v_j^T
//
// Three launches, the first and the last over all chunks of all entries and heads at once:
//   decay_chunk_sums     U of every chunk (a product over the chunk's rows)
//   decay_chunk_states   entry by entry: every chunk's state at its start (written over U) and the request's new state; elementwise
//   decay_chunk_outputs  o of every chunk: two products with a triangle of decays between them, and one with the chunk's first state
//
// and one for decode steps, in which (nearly) every entry is one row:
//   decay_step           S and o of a row as they are written above, every load of the state in flight at once
//
// The products run on the warp-level tensor cores (mma.sync, bfloat16 with float sums). Everything that enters them is float: silu of
// queries, keys and values (where asked for), powers of the decay, states, weighted scores; each operand is the sum of two bfloat16
// terms (16 bits of mantissa), of whose four products three are taken. States and sums stay float.
#include <math.h>

#include "common.cuh"
#include "mma_sync.cuh"

namespace {

constexpr int CHUNK = 64, THREADS = 128, COLS = 64;   // rows of a chunk; four warps; value columns a CTA takes
constexpr int MAX_DIM = 256;

struct ChunkArgs {
  const bf16* q; int q_stride;
  const bf16* k; int k_stride;
  const bf16* v; int v_stride;     // [T, heads * vdim]
  const float* decay;              // [heads]
  float k_scale; int silu_in;
  float* sums;                     // [tiles][heads][dim][vdim]: U, then the states at the chunks' starts
  float* state; long long slot_stride;
  const int32_t* q_start; const int32_t* state_slot; const int32_t* fresh;
  int n_entries;
  float* out; int out_stride;
  int n_heads, dim, vdim, dim16;   // dim16: dim to a multiple of 16
  int vec;                         // rows, heads and slices start on 16-byte boundaries and hold multiples of eight numbers
};

struct Tile { int entry, row0, rows; };   // entry -1: no such chunk

// Chunks are numbered entry by entry. One warp finds a chunk's entry.
__device__ __forceinline__ Tile find_tile(const int32_t* q_start, int n_entries, int tile) {
  const int lane = threadIdx.x & 31;
  int left = tile;
  for (int base = 0; base < n_entries; base += 32) {
    const int e = base + lane;
    const int first = e < n_entries ? q_start[e] : 0, rows = e < n_entries ? q_start[e + 1] - first : 0;
    const int own = (rows + CHUNK - 1) / CHUNK;
    int upto = own;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int other = __shfl_up_sync(0xffffffffu, upto, o);
      if (lane >= o) upto += other;
    }
    const unsigned hit = __ballot_sync(0xffffffffu, upto > left);
    if (hit != 0) {
      const int at = __ffs(hit) - 1;
      const int within = left - (__shfl_sync(0xffffffffu, upto, at) - __shfl_sync(0xffffffffu, own, at));
      const int row0 = __shfl_sync(0xffffffffu, first, at) + within * CHUNK;
      return {base + at, row0, min(CHUNK, __shfl_sync(0xffffffffu, first + rows, at) - row0)};
    }
    left -= __shfl_sync(0xffffffffu, upto, 31);
  }
  return {-1, 0, 0};
}

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return uint32_t(__cvta_generic_to_shared(p)); }
__device__ __forceinline__ float silu(float x) { return __fdividef(x, 1.f + __expf(-x)); }   // (a few units of the last place)
__device__ __forceinline__ uint32_t pack_pair(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

// decay^n by squaring (decay^0 is one, also for a decay of zero)
__device__ __forceinline__ float power(float decay, int n) {
  float out = 1.f, square = decay;
  for (; n > 0; n >>= 1, square *= square)
    if (n & 1) out *= square;
  return out;
}

// A matrix in shared memory as two bfloat16 terms, rows `stride` numbers apart.
struct Split { bf16* hi; bf16* lo; int stride; };

__device__ __forceinline__ void put2(const Split& m, int r, int c, float x, float y) {
  const uint32_t head = pack_pair(x, y);
  *reinterpret_cast<uint32_t*>(m.hi + r * m.stride + c) = head;
  *reinterpret_cast<uint32_t*>(m.lo + r * m.stride + c) = pack_rest(x, y, head);
}

// `rows` rows of `cols` numbers (zeros up to CHUNK rows and `padded` columns), silu, times `scale` and, with `powers`, times
// powers[rows - 1 - row].
__device__ __forceinline__ void stage(const Split& m, const bf16* src, long long stride, int rows, int cols, int padded, bool silu_in, float scale,
                                      const float* powers, bool vec) {
  const int pieces = padded / 8;
  for (int i = threadIdx.x; i < CHUNK * pieces; i += THREADS) {
    const int r = i / pieces, c = (i - r * pieces) * 8;
    float x[8];
#pragma unroll
    for (int u = 0; u < 8; ++u) x[u] = 0.f;
    if (r < rows && c < cols) {
      const bf16* p = src + r * stride + c;
      if (vec) {
        const uint4 w = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* w2 = reinterpret_cast<const __nv_bfloat162*>(&w);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          const float2 f = __bfloat1622float2(w2[u]);
          x[2 * u] = f.x;
          x[2 * u + 1] = f.y;
        }
      } else {
#pragma unroll
        for (int u = 0; u < 8; ++u)
          if (c + u < cols) x[u] = to_float(p[u]);
      }
      const float factor = powers != nullptr ? scale * powers[rows - 1 - r] : scale;
#pragma unroll
      for (int u = 0; u < 8; ++u) x[u] = (silu_in ? silu(x[u]) : x[u]) * factor;
    }
#pragma unroll
    for (int u = 0; u < 8; u += 2) put2(m, r, c + u, x[u], x[u + 1]);
  }
}

// Operand fragments of mma.sync m16n8k16 (lane addresses for ldmatrix).
// a: 16 x 16 of a matrix stored by rows, from (r, c) on
__device__ __forceinline__ void load_a(const bf16* m, int stride, int r, int c, uint32_t (&f)[4]) {
  const int lane = threadIdx.x & 31;
  ldmatrix_x4(smem_u32(m + (r + (lane & 15)) * stride + c + (lane >> 4) * 8), f[0], f[1], f[2], f[3]);
}
// a: 16 x 16 of the transpose of a matrix stored by rows: rows of the operand are the stored columns from c on, its k the stored rows
__device__ __forceinline__ void load_a_transposed(const bf16* m, int stride, int k, int c, uint32_t (&f)[4]) {
  const int lane = threadIdx.x & 31;
  ldmatrix_x4_trans(smem_u32(m + (k + (lane & 7) + (lane >> 4) * 8) * stride + c + ((lane >> 3) & 1) * 8), f[0], f[1], f[2], f[3]);
}
// b: k 16 x n 16 (two tiles of 8 columns: f[0..1], f[2..3]) of a matrix stored by rows of n
__device__ __forceinline__ void load_b(const bf16* m, int stride, int n, int k, uint32_t (&f)[4]) {
  const int lane = threadIdx.x & 31;
  ldmatrix_x4(smem_u32(m + (n + (lane & 7) + (lane >> 4) * 8) * stride + k + ((lane >> 3) & 1) * 8), f[0], f[1], f[2], f[3]);
}
// b: k 16 x n 16 of a matrix stored by rows of k
__device__ __forceinline__ void load_b_transposed(const bf16* m, int stride, int k, int n, uint32_t (&f)[4]) {
  const int lane = threadIdx.x & 31;
  ldmatrix_x4_trans(smem_u32(m + (k + (lane & 15)) * stride + n + (lane >> 4) * 8), f[0], f[1], f[2], f[3]);
}
// (a_hi + a_lo)(b_hi + b_lo) without the product of the two small terms, for one tile of 8 columns
__device__ __forceinline__ void mma_split(float (&c)[4], const uint32_t (&ah)[4], const uint32_t (&al)[4], uint32_t bh0, uint32_t bh1, uint32_t bl0, uint32_t bl1) {
  mma_bf16(c, al[0], al[1], al[2], al[3], bh0, bh1);
  mma_bf16(c, ah[0], ah[1], ah[2], ah[3], bl0, bl1);
  mma_bf16(c, ah[0], ah[1], ah[2], ah[3], bh0, bh1);
}

__device__ __forceinline__ Split carve(uint8_t*& at, int rows, int stride) {
  Split m = {reinterpret_cast<bf16*>(at), reinterpret_cast<bf16*>(at) + rows * stride, stride};
  at += size_t(rows) * stride * 2 * sizeof(bf16);
  return m;
}

// U of a chunk: [dim x COLS of the value columns]. Grid: chunks, heads, slices of the columns.
__global__ void __launch_bounds__(THREADS)
decay_chunk_sums_kernel(const ChunkArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float powers[CHUNK];
  const Tile tile = find_tile(a.q_start, a.n_entries, blockIdx.x);
  const int h = blockIdx.y, col0 = blockIdx.z * COLS, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i < CHUNK; i += THREADS) powers[i] = power(a.decay[h], i);
  __syncthreads();
  pdl_wait();
  if (tile.entry < 0) return;
  uint8_t* at = smem;
  const Split k = carve(at, CHUNK, a.dim16 + 8), v = carve(at, CHUNK, COLS + 8);
  const int cols = min(COLS, a.vdim - col0);
  stage(k, a.k + size_t(tile.row0) * a.k_stride + size_t(h) * a.dim, a.k_stride, tile.rows, a.dim, a.dim16, a.silu_in, a.k_scale, powers, a.vec);
  stage(v, a.v + size_t(tile.row0) * a.v_stride + size_t(h) * a.vdim + col0, a.v_stride, tile.rows, cols, COLS, a.silu_in, 1.f, nullptr, a.vec);
  __syncthreads();
  float* sums = a.sums + (size_t(blockIdx.x) * a.n_heads + h) * a.dim * a.vdim + col0;
  for (int m0 = warp * 16; m0 < a.dim16; m0 += (THREADS / 32) * 16) {
    float acc[COLS / 8][4] = {};
    for (int j = 0; j < tile.rows; j += 16) {
      uint32_t ah[4], al[4];
      load_a_transposed(k.hi, k.stride, j, m0, ah);
      load_a_transposed(k.lo, k.stride, j, m0, al);
#pragma unroll
      for (int n = 0; n < COLS; n += 16) {
        uint32_t bh[4], bl[4];
        load_b_transposed(v.hi, v.stride, j, n, bh);
        load_b_transposed(v.lo, v.stride, j, n, bl);
        mma_split(acc[n / 8], ah, al, bh[0], bh[1], bl[0], bl[1]);
        mma_split(acc[n / 8 + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
      }
    }
#pragma unroll
    for (int t = 0; t < COLS / 8; ++t) {
      const int c = t * 8 + (lane & 3) * 2;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int r = m0 + (lane >> 2) + half * 8;
        if (r < a.dim) {
          float* dst = sums + size_t(r) * a.vdim + c;
          if (c + 1 < cols && (a.vdim & 1) == 0) {
            *reinterpret_cast<float2*>(dst) = make_float2(acc[t][2 * half], acc[t][2 * half + 1]);
          } else {
            if (c < cols) dst[0] = acc[t][2 * half];
            if (c + 1 < cols) dst[1] = acc[t][2 * half + 1];
          }
        }
      }
    }
  }
}

// The states at the chunks' starts, and the request's new one. Grid: entries, heads, pieces of the state.
__global__ void __launch_bounds__(256)
decay_chunk_states_kernel(const ChunkArgs a) {
  pdl_launch_dependents();
  __shared__ float scratch[33];
  const int e = blockIdx.x, h = blockIdx.y;
  const int row0 = a.q_start[e], rows = a.q_start[e + 1] - row0;
  int before = 0;   // chunks of the entries before this one
  for (int i = threadIdx.x; i < e; i += blockDim.x) before += (a.q_start[i + 1] - a.q_start[i] + CHUNK - 1) / CHUNK;
  const int first = int(block_sum(float(before), scratch));   // (small whole numbers: exact)
  const bool is_fresh = a.fresh[e] != 0;
  const int size = a.dim * a.vdim, i = blockIdx.z * blockDim.x + threadIdx.x;
  const float decay = a.decay[h];
  const float whole = power(decay, CHUNK), last = power(decay, rows - (rows - 1) / CHUNK * CHUNK);
  pdl_wait();
  if (rows <= 0 || i >= size) return;   // an entry without rows touches no slot
  float* slot = a.state + size_t(a.state_slot[e]) * a.slot_stride + size_t(h) * size + i;
  float s = is_fresh ? 0.f : *slot;
  float* sums = a.sums + (size_t(first) * a.n_heads + h) * size + i;
  const size_t step = size_t(a.n_heads) * size;
  const int n = (rows + CHUNK - 1) / CHUNK;
  for (int base = 0; base < n; base += 8) {   // eight chunks' sums in flight
    float u[8];
#pragma unroll
    for (int c = 0; c < 8; ++c) u[c] = base + c < n ? sums[(base + c) * step] : 0.f;
#pragma unroll
    for (int c = 0; c < 8; ++c) {
      if (base + c < n) {
        sums[(base + c) * step] = s;
        s = fmaf(base + c == n - 1 ? last : whole, s, u[c]);
      }
    }
  }
  *slot = s;
}

// Outputs of a chunk. Grid: chunks, heads, slices of the columns. A warp has 16 of the chunk's rows.
__global__ void __launch_bounds__(THREADS)
decay_chunk_outputs_kernel(const ChunkArgs a) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float powers[CHUNK + 1];
  const Tile tile = find_tile(a.q_start, a.n_entries, blockIdx.x);
  const int h = blockIdx.y, col0 = blockIdx.z * COLS, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i <= CHUNK; i += THREADS) powers[i] = power(a.decay[h], i);
  __syncthreads();
  pdl_wait();
  if (tile.entry < 0) return;
  uint8_t* at = smem;
  const Split q = carve(at, CHUNK, a.dim16 + 8), k = carve(at, CHUNK, a.dim16 + 8), v = carve(at, CHUNK, COLS + 8), s = carve(at, a.dim16, COLS + 8);
  const int cols = min(COLS, a.vdim - col0);
  stage(q, a.q + size_t(tile.row0) * a.q_stride + size_t(h) * a.dim, a.q_stride, tile.rows, a.dim, a.dim16, a.silu_in, 1.f, nullptr, a.vec);
  stage(k, a.k + size_t(tile.row0) * a.k_stride + size_t(h) * a.dim, a.k_stride, tile.rows, a.dim, a.dim16, a.silu_in, a.k_scale, nullptr, a.vec);
  stage(v, a.v + size_t(tile.row0) * a.v_stride + size_t(h) * a.vdim + col0, a.v_stride, tile.rows, cols, COLS, a.silu_in, 1.f, nullptr, a.vec);
  const float* start = a.sums + (size_t(blockIdx.x) * a.n_heads + h) * a.dim * a.vdim + col0;
  for (int i = threadIdx.x; i < a.dim16 * (COLS / 2); i += THREADS) {
    const int r = i / (COLS / 2), c = (i - r * (COLS / 2)) * 2;
    const float* p = start + size_t(r) * a.vdim + c;
    put2(s, r, c, r < a.dim && c < cols ? p[0] : 0.f, r < a.dim && c + 1 < cols ? p[1] : 0.f);
  }
  __syncthreads();
  const int i0 = warp * 16;
  if (i0 >= tile.rows) return;   // (no barrier follows)
  // what the chunk's first state gives, and the scores of the rows up to each row
  float acc[COLS / 8][4] = {}, p[CHUNK / 8][4] = {};
  for (int d = 0; d < a.dim16; d += 16) {
    uint32_t ah[4], al[4];
    load_a(q.hi, q.stride, i0, d, ah);
    load_a(q.lo, q.stride, i0, d, al);
#pragma unroll
    for (int n = 0; n < COLS; n += 16) {
      uint32_t bh[4], bl[4];
      load_b_transposed(s.hi, s.stride, d, n, bh);
      load_b_transposed(s.lo, s.stride, d, n, bl);
      mma_split(acc[n / 8], ah, al, bh[0], bh[1], bl[0], bl[1]);
      mma_split(acc[n / 8 + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
    }
#pragma unroll
    for (int j = 0; j < CHUNK; j += 16) {
      if (j <= i0) {   // (later rows are seen by none of the warp's)
        uint32_t bh[4], bl[4];
        load_b(k.hi, k.stride, j, d, bh);
        load_b(k.lo, k.stride, j, d, bl);
        mma_split(p[j / 8], ah, al, bh[0], bh[1], bl[0], bl[1]);
        mma_split(p[j / 8 + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
      }
    }
  }
  const int r = i0 + (lane >> 2);   // this lane's rows: r and r + 8
  const float lead0 = powers[r + 1], lead1 = powers[r + 9];
#pragma unroll
  for (int t = 0; t < COLS / 8; ++t) {
    acc[t][0] *= lead0;
    acc[t][1] *= lead0;
    acc[t][2] *= lead1;
    acc[t][3] *= lead1;
  }
#pragma unroll
  for (int j = 0; j < CHUNK; j += 16) {
    if (j > i0) break;
    uint32_t ah[4], al[4];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      float* w = p[j / 8 + half];
      const int c = j + half * 8 + (lane & 3) * 2;
      const float w0 = c <= r ? w[0] * powers[r - c] : 0.f, w1 = c + 1 <= r ? w[1] * powers[r - c - 1] : 0.f;
      const float w2 = c <= r + 8 ? w[2] * powers[r + 8 - c] : 0.f, w3 = c + 1 <= r + 8 ? w[3] * powers[r + 7 - c] : 0.f;
      ah[2 * half] = pack_pair(w0, w1);
      al[2 * half] = pack_rest(w0, w1, ah[2 * half]);
      ah[2 * half + 1] = pack_pair(w2, w3);
      al[2 * half + 1] = pack_rest(w2, w3, ah[2 * half + 1]);
    }
#pragma unroll
    for (int n = 0; n < COLS; n += 16) {
      uint32_t bh[4], bl[4];
      load_b_transposed(v.hi, v.stride, j, n, bh);
      load_b_transposed(v.lo, v.stride, j, n, bl);
      mma_split(acc[n / 8], ah, al, bh[0], bh[1], bl[0], bl[1]);
      mma_split(acc[n / 8 + 1], ah, al, bh[2], bh[3], bl[2], bl[3]);
    }
  }
  float* out = a.out + size_t(h) * a.vdim + col0;
  const bool pairs = (a.vdim & 1) == 0 && (a.out_stride & 1) == 0;
#pragma unroll
  for (int t = 0; t < COLS / 8; ++t) {
    const int c = t * 8 + (lane & 3) * 2;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      if (r + half * 8 < tile.rows) {
        float* dst = out + size_t(tile.row0 + r + half * 8) * a.out_stride + c;
        if (c + 1 < cols && pairs) {
          *reinterpret_cast<float2*>(dst) = make_float2(acc[t][2 * half], acc[t][2 * half + 1]);
        } else {
          if (c < cols) dst[0] = acc[t][2 * half];
          if (c + 1 < cols) dst[1] = acc[t][2 * half + 1];
        }
      }
    }
  }
}

// Decode steps. A CTA has one (entry, head, slice of the columns); a thread has V neighbouring columns of every row_groups-th row, and
// the row groups' sums meet in shared memory, in order.
constexpr int STEP_THREADS = 128, STEP_ROWS = 8;
template <int V>
__global__ void __launch_bounds__(STEP_THREADS)
decay_step_kernel(const ChunkArgs a, int slice) {
  pdl_launch_dependents();
  __shared__ float qs[MAX_DIM], ks[MAX_DIM], sums[STEP_THREADS][V];
  const int e = blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * slice;
  const int row0 = a.q_start[e], row1 = a.q_start[e + 1];
  const bool is_fresh = a.fresh[e] != 0;
  const float decay = a.decay[h];
  const int groups = slice / V, row_groups = STEP_THREADS / groups;   // (groups divides the threads)
  const int g = threadIdx.x % groups, rg = threadIdx.x / groups, j = col0 + g * V;
  const bool mine = j < a.vdim;
  float* head_state = a.state + size_t(a.state_slot[e]) * a.slot_stride + size_t(h) * a.dim * a.vdim;
  pdl_wait();
  for (int t = row0; t < row1; ++t) {
    const bool zero = is_fresh && t == row0;
    float s[STEP_ROWS][V], v[V], acc[V] = {};
#pragma unroll
    for (int i = 0; i < STEP_ROWS; ++i) {   // the first rows' states, asked for before anything is waited for
      const int r = rg + i * row_groups;
#pragma unroll
      for (int u = 0; u < V; ++u) s[i][u] = 0.f;
      if (mine && r < a.dim && !zero) {
        const float* p = head_state + size_t(r) * a.vdim + j;
        if (V == 4) {
          const float4 f = *reinterpret_cast<const float4*>(p);
          s[i][0] = f.x;
          s[i][V > 1 ? 1 : 0] = f.y;
          s[i][V > 2 ? 2 : 0] = f.z;
          s[i][V > 3 ? 3 : 0] = f.w;
        } else {
          s[i][0] = *p;
        }
      }
    }
    const bf16* q = a.q + size_t(t) * a.q_stride + size_t(h) * a.dim;
    const bf16* k = a.k + size_t(t) * a.k_stride + size_t(h) * a.dim;
    for (int i = threadIdx.x; i < a.dim; i += STEP_THREADS) {
      const float x = to_float(q[i]), y = to_float(k[i]);
      qs[i] = a.silu_in ? silu(x) : x;
      ks[i] = (a.silu_in ? silu(y) : y) * a.k_scale;
    }
#pragma unroll
    for (int u = 0; u < V; ++u) {
      const float x = mine ? to_float(a.v[size_t(t) * a.v_stride + size_t(h) * a.vdim + j + u]) : 0.f;
      v[u] = a.silu_in ? silu(x) : x;
    }
    __syncthreads();
    auto row = [&](int r, float (&state)[V]) {
#pragma unroll
      for (int u = 0; u < V; ++u) {
        state[u] = fmaf(decay, state[u], ks[r] * v[u]);
        acc[u] = fmaf(state[u], qs[r], acc[u]);
      }
      float* p = head_state + size_t(r) * a.vdim + j;
      if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(state[0], state[V > 1 ? 1 : 0], state[V > 2 ? 2 : 0], state[V > 3 ? 3 : 0]);
      else *p = state[0];
    };
    if (mine) {
#pragma unroll
      for (int i = 0; i < STEP_ROWS; ++i)
        if (rg + i * row_groups < a.dim) row(rg + i * row_groups, s[i]);
      for (int r = rg + STEP_ROWS * row_groups; r < a.dim; r += row_groups) {
        const float* p = head_state + size_t(r) * a.vdim + j;
        float state[V];
#pragma unroll
        for (int u = 0; u < V; ++u) state[u] = zero ? 0.f : p[u];
        row(r, state);
      }
    }
#pragma unroll
    for (int u = 0; u < V; ++u) sums[threadIdx.x][u] = acc[u];
    __syncthreads();
    if (rg == 0 && mine) {
#pragma unroll
      for (int u = 0; u < V; ++u) {
        float o = 0.f;
        for (int i = 0; i < row_groups; ++i) o += sums[i * groups + g][u];
        a.out[size_t(t) * a.out_stride + size_t(h) * a.vdim + j + u] = o;
      }
    }
    __syncthreads();   // (the vectors and sums of the next row)
  }
}

size_t split_bytes(int rows, int stride) { return size_t(rows) * stride * 2 * sizeof(bf16); }

}  // namespace

// Floats of scratch for a batch whose entries have n_tiles chunks in all (each entry's last chunk may be short).
extern "C" long long r2_decay_chunks_floats(int n_tiles, int n_heads, int dim, int vdim) { return (long long)n_tiles * n_heads * dim * vdim; }

// q, k [T, heads * dim], v [T, heads * vdim] bfloat16 (slices of a projection); decay float [heads]; silu_in: silu of all three on their
// way in, k then times k_scale; state float [slots][heads][dim][vdim]; n_tiles at least the sum over entries of ceil(rows / 64); scratch
// float (r2_decay_chunks_floats); out float [T, heads * vdim]. Three launches. R2_UNSUPPORTED: heads of more than 256 rows.
extern "C" int r2_decay_chunks(const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride, const float* decay, float k_scale,
                               int silu_in, float* state, long long slot_stride, const int32_t* q_start, const int32_t* state_slot, const int32_t* fresh,
                               int n_entries, int n_tiles, float* scratch, long long scratch_floats, float* out, int out_stride, int n_heads, int dim,
                               int vdim, cudaStream_t stream) {
  if (n_entries <= 0 || n_tiles <= 0) return R2_OK;
  if (n_heads < 1 || dim < 1 || vdim < 1 || scratch == nullptr || scratch_floats < r2_decay_chunks_floats(n_tiles, n_heads, dim, vdim)) return R2_BAD_SHAPE;
  if (dim > MAX_DIM || n_heads > 65535 || n_tiles > (1 << 20)) return R2_UNSUPPORTED;
  ChunkArgs a = {};
  a.q = (const bf16*)q; a.q_stride = q_stride; a.k = (const bf16*)k; a.k_stride = k_stride; a.v = (const bf16*)v; a.v_stride = v_stride;
  a.decay = decay; a.k_scale = k_scale; a.silu_in = silu_in; a.sums = scratch; a.state = state; a.slot_stride = slot_stride;
  a.q_start = q_start; a.state_slot = state_slot; a.fresh = fresh; a.n_entries = n_entries; a.out = out; a.out_stride = out_stride;
  a.n_heads = n_heads; a.dim = dim; a.vdim = vdim; a.dim16 = (dim + 15) / 16 * 16;
  a.vec = dim % 8 == 0 && vdim % 8 == 0 && q_stride % 8 == 0 && k_stride % 8 == 0 && v_stride % 8 == 0 &&
          !((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v)) & 15);
  const size_t rows_q = split_bytes(CHUNK, a.dim16 + 8), rows_v = split_bytes(CHUNK, COLS + 8);
  const size_t smem_sums = rows_q + rows_v, smem_out = 2 * rows_q + rows_v + split_bytes(a.dim16, COLS + 8);
  static bool configured = false;
  if (!configured) {
    const int most = int(2 * split_bytes(CHUNK, MAX_DIM + 8) + split_bytes(CHUNK, COLS + 8) + split_bytes(MAX_DIM, COLS + 8));
    cudaError_t e = cudaFuncSetAttribute(decay_chunk_outputs_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(decay_chunk_sums_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, most);
    if (e != cudaSuccess) {
      cudaGetLastError();
      return R2_UNSUPPORTED;
    }
    configured = true;
  }
  const dim3 grid(n_tiles, n_heads, (vdim + COLS - 1) / COLS);
  r2_launch(decay_chunk_sums_kernel, grid, dim3(THREADS), smem_sums, stream, a);
  r2_launch(decay_chunk_states_kernel, dim3(n_entries, n_heads, (dim * vdim + 255) / 256), dim3(256), size_t(0), stream, a);
  r2_launch(decay_chunk_outputs_kernel, grid, dim3(THREADS), smem_out, stream, a);
  return launch_status();
}

// The same for batches in which (nearly) every entry is one row: one launch, no scratch.
extern "C" int r2_decay_step(const void* q, int q_stride, const void* k, int k_stride, const void* v, int v_stride, const float* decay, float k_scale,
                             int silu_in, float* state, long long slot_stride, const int32_t* q_start, const int32_t* state_slot, const int32_t* fresh,
                             int n_entries, float* out, int out_stride, int n_heads, int dim, int vdim, int n_sms, cudaStream_t stream) {
  if (n_entries <= 0) return R2_OK;
  if (n_heads < 1 || dim < 1 || vdim < 1 || n_sms < 1) return R2_BAD_SHAPE;
  if (dim > MAX_DIM || n_heads > 65535) return R2_UNSUPPORTED;
  ChunkArgs a = {};
  a.q = (const bf16*)q; a.q_stride = q_stride; a.k = (const bf16*)k; a.k_stride = k_stride; a.v = (const bf16*)v; a.v_stride = v_stride;
  a.decay = decay; a.k_scale = k_scale; a.silu_in = silu_in; a.state = state; a.slot_stride = slot_stride;
  a.q_start = q_start; a.state_slot = state_slot; a.fresh = fresh; a.n_entries = n_entries; a.out = out; a.out_stride = out_stride;
  a.n_heads = n_heads; a.dim = dim; a.vdim = vdim;
  // as many columns a CTA as leave twice as many CTAs as the GPU has SMs
  int slice = 64;
  while (slice > 16 && (long long)n_entries * n_heads * ((vdim + slice - 1) / slice) < 2ll * n_sms) slice /= 2;
  const dim3 grid(n_entries, n_heads, (vdim + slice - 1) / slice);
  const bool quads = vdim % 4 == 0 && slot_stride % 4 == 0 && !(reinterpret_cast<uintptr_t>(state) & 15);
  if (quads) r2_launch(decay_step_kernel<4>, grid, dim3(STEP_THREADS), size_t(0), stream, a, slice);
  else r2_launch(decay_step_kernel<1>, grid, dim3(STEP_THREADS), size_t(0), stream, a, slice);
  return launch_status();
}
