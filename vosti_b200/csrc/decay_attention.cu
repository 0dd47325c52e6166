// Linear attention with one fixed decay per head: per request and head a float32 state S [dk, dv],
//
//   S_t = decay * S_(t-1) + k_t v_t^T,    o_t = S_t^T q_t
//
// q, k and v are columns of one projection (the serving type, or float32 unsummed K splits, added in
// split order and rounded to the serving type); on the way in they may pass SiLU, or q and k a rotation
// of the first 2 * rot_half elements of each head (element i with i + rot_half, by position * freq[i],
// formed in float32); k is then multiplied by a constant. The state slot of a request holds S of all heads
// ([heads, dk, dv]).
//
// decay_scan: token by token, for steps of few tokens a request and for float32 serving. A block takes a
// piece of the value columns of one (request, head); a thread keeps a few rows of S in registers, the
// state is read and written once.
//
// Long portions in bfloat16 run as chunks of 128 tokens, on the 5th-generation tensor cores (tcgen05, accumulators in
// tensor memory, operands made by the block's threads in the 128-byte-swizzled layout):
//   decay_chunk_state  U_c = sum over the chunk's tokens of decay^(tokens after it) k v^T, all chunks side by side;
//   decay_chunk_scan   S before every chunk, S_(c+1) = decay^(n_c) S_c + U_c, written over U; the last one to the slot;
//   decay_chunk_out    o_t = decay^(t+1) q_t S_c + sum over j <= t of decay^(t-j) (q_t . k_j) v_j, all chunks side by side.
// What is float32 in the recurrence (decayed keys, rotated queries and keys, S, the weights of the second
// product) enters a product as two bfloat16 terms; the product of the two remainders is left out. SiLU'd
// queries, keys and values are activations of a projection and are rounded to bfloat16.
//
// decay_out: the read-outs normed (each head by its own root mean square, or all heads together with a
// weight) and gated (SiLU or sigmoid of further columns of the projection), rounded for the output product.
#include "common.cuh"
#include "mma_util.cuh"
#include "tcgen05.cuh"

namespace {

constexpr int MAX_DK = 256;
constexpr int CHUNK = 128;

__device__ __forceinline__ float silu_of(float x) { return x / (1.f + expf(-x)); }
template <typename T> __device__ __forceinline__ float rounded_to(float x) { return to_f32(from_f32<T>(x)); }

struct Projection {
  const void* data;            // T [tokens, stride], or float32 [splits, tokens, stride] with `plane` between splits
  int splits;
  int64_t stride, plane;
  int off_q, off_k, off_v, off_g;
};
// Column `col` of token t, rounded to the serving type.
template <typename T>
__device__ __forceinline__ float column(const Projection& p, int64_t t, int col) {
  const int64_t at = t * p.stride + col;
  if (p.splits == 0) return to_f32(reinterpret_cast<const T*>(p.data)[at]);
  const float* src = reinterpret_cast<const float*>(p.data) + at;
  float x = src[0];
  for (int s = 1; s < p.splits; ++s) x += src[s * p.plane];
  return rounded_to<T>(x);
}

struct Recurrence {
  int heads, dk, dv, silu;
  const float* decay;          // [heads]
  const float* log2_decay;     // [heads]
  float key_scale;
  const float* freq;           // [rot_half]
  int rot_half;
  const int* positions;
  float* state;
  int64_t state_stride;
  const int* cu_q;
  const int* state_slots;
  int num_slots;
};

// ------------------------------------------------------------------ token by token
constexpr int SCAN_THREADS = 256;
constexpr int SCAN_LANES = 8;                        // threads side by side along the value columns
constexpr int SCAN_ROWS = SCAN_THREADS / SCAN_LANES; // row groups: a thread keeps rows rg, rg + 32, ...
constexpr int SCAN_TOKENS = 8;                       // tokens staged together

template <typename T, int V, int R>
__global__ void __launch_bounds__(SCAN_THREADS)
decay_scan_kernel(const Projection p, const Recurrence c, float* __restrict__ out, int max_len) {
  constexpr int COLS = SCAN_LANES * V;
  __shared__ float qs[SCAN_TOKENS][32 * R], ks[SCAN_TOKENS][32 * R], vs[SCAN_TOKENS][COLS];
  __shared__ float red[SCAN_TOKENS][SCAN_THREADS / 32][COLS];
  extern __shared__ float turns[];                   // [SCAN_TOKENS][rot_half] cosines, then sines
  pdl_wait();
  pdl_launch_dependents();
  const int b = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * COLS;
  const int slot = c.state_slots[b];
  const int start = c.cu_q[b], n = c.cu_q[b + 1] - start;
  if (slot < 0 || slot >= c.num_slots || n <= 0 || (max_len > 0 && n > max_len)) return;
  const int lane8 = threadIdx.x % SCAN_LANES, rg = threadIdx.x / SCAN_LANES;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int dk = c.dk, dv = c.dv;
  const int col = col0 + lane8 * V;
  const bool live = col < dv;                        // (V = 4 only where dv is a multiple of 4)
  float* S = c.state + (int64_t)slot * c.state_stride + (int64_t)h * dk * dv + col;
  float s[R][V];
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = rg + SCAN_ROWS * i;
    if (V == 4) {
      const float4 x = (live && r < dk) ? *reinterpret_cast<const float4*>(S + (int64_t)r * dv) : make_float4(0.f, 0.f, 0.f, 0.f);
      s[i][0] = x.x; s[i][V > 1 ? 1 : 0] = x.y; s[i][V > 2 ? 2 : 0] = x.z; s[i][V > 3 ? 3 : 0] = x.w;
    } else {
      s[i][0] = (live && r < dk) ? S[(int64_t)r * dv] : 0.f;
    }
  }
  const float decay = c.decay[h];
  float* cosines = turns;
  float* sines = turns + SCAN_TOKENS * c.rot_half;
  for (int t0 = 0; t0 < n; t0 += SCAN_TOKENS) {
    const int count = min(SCAN_TOKENS, n - t0);
    if (c.rot_half > 0) {
      for (int i = threadIdx.x; i < count * c.rot_half; i += SCAN_THREADS) {
        const int tt = i / c.rot_half, f = i - tt * c.rot_half;
        const float angle = (float)c.positions[start + t0 + tt] * c.freq[f];
        cosines[tt * c.rot_half + f] = cosf(angle);
        sines[tt * c.rot_half + f] = sinf(angle);
      }
      __syncthreads();
    }
    for (int i = threadIdx.x; i < count * dk; i += SCAN_THREADS) {
      const int tt = i / dk, e = i - tt * dk;
      const int64_t t = start + t0 + tt;
      const int cq = p.off_q + h * dk, ck = p.off_k + h * dk;
      float q = column<T>(p, t, cq + e), k = column<T>(p, t, ck + e);
      if (c.silu) { q = silu_of(q); k = silu_of(k); }
      if (e < 2 * c.rot_half) {
        const bool low = e < c.rot_half;
        const int other = low ? e + c.rot_half : e - c.rot_half, f = low ? e : other;
        const float cs = cosines[tt * c.rot_half + f], sn = low ? -sines[tt * c.rot_half + f] : sines[tt * c.rot_half + f];
        q = q * cs + column<T>(p, t, cq + other) * sn;
        k = k * cs + column<T>(p, t, ck + other) * sn;
      }
      qs[tt][e] = q;
      ks[tt][e] = k * c.key_scale;
    }
    for (int i = threadIdx.x; i < count * COLS; i += SCAN_THREADS) {
      const int tt = i / COLS, e = i - tt * COLS;
      float v = col0 + e < dv ? column<T>(p, start + t0 + tt, p.off_v + h * dv + col0 + e) : 0.f;
      vs[tt][e] = c.silu ? silu_of(v) : v;
    }
    __syncthreads();
    for (int tt = 0; tt < count; ++tt) {
      float o[V], v[V];
#pragma unroll
      for (int e = 0; e < V; ++e) { o[e] = 0.f; v[e] = vs[tt][lane8 * V + e]; }
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int r = rg + SCAN_ROWS * i;
        if (r < dk) {
          const float k = ks[tt][r], q = qs[tt][r];
#pragma unroll
          for (int e = 0; e < V; ++e) {
            s[i][e] = fmaf(k, v[e], s[i][e] * decay);
            o[e] = fmaf(q, s[i][e], o[e]);
          }
        }
      }
#pragma unroll
      for (int e = 0; e < V; ++e) {
        o[e] += __shfl_xor_sync(0xffffffffu, o[e], 8);
        o[e] += __shfl_xor_sync(0xffffffffu, o[e], 16);
        if (lane < SCAN_LANES) red[tt][warp][lane8 * V + e] = o[e];
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < count * COLS; i += SCAN_THREADS) {
      const int tt = i / COLS, e = i - tt * COLS;
      if (col0 + e < dv) {
        float sum = 0.f;
#pragma unroll
        for (int w = 0; w < SCAN_THREADS / 32; ++w) sum += red[tt][w][e];
        out[(int64_t)(start + t0 + tt) * c.heads * dv + h * dv + col0 + e] = sum;
      }
    }
  }
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int r = rg + SCAN_ROWS * i;
    if (!live || r >= dk) continue;
    if (V == 4) *reinterpret_cast<float4*>(S + (int64_t)r * dv) = make_float4(s[i][0], s[i][V > 1 ? 1 : 0], s[i][V > 2 ? 2 : 0], s[i][V > 3 ? 3 : 0]);
    else S[(int64_t)r * dv] = s[i][0];
  }
}

// ------------------------------------------------------------------ chunks on the tensor cores
constexpr int CHUNK_THREADS = 512;
constexpr int CHUNK_MAX_DK = 128;
constexpr int VT = 128;                 // value columns of a block
constexpr int BLOCK_BYTES = CHUNK * 128;        // [128 rows][64 elements], 128-byte swizzle

struct Chunks {
  const int* request;                   // [chunks] the request a chunk belongs to
  const int* first;                     // [chunks] its first token, counted in the request's portion
  const float2* turns;                  // [tokens][rot_half] (cosine, sine), or null
  float* states;                        // [chunks][heads][dk][dv]
};

__global__ void __launch_bounds__(256)
rotation_table_kernel(const float* __restrict__ freq, int half, const int* __restrict__ positions, int64_t n, float2* __restrict__ out) {
  pdl_wait();
  pdl_launch_dependents();
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int64_t t = i / half;
    const float angle = (float)positions[t] * freq[i - t * half];
    out[i] = make_float2(cosf(angle), sinf(angle));
  }
}

__device__ __forceinline__ float gate_value(float g, int silu) { return silu ? silu_of(g) : 1.f / (1.f + expf(-g)); }
// SiLU and sigmoid gates on the special-function unit, for results that are rounded to bfloat16.
__device__ __forceinline__ float quick_silu(float x) { return __fdividef(x, 1.f + __expf(-x)); }
__device__ __forceinline__ float quick_gate(float g, int silu) { return silu ? quick_silu(g) : __fdividef(1.f, 1.f + __expf(-g)); }
// Two values as two bfloat16 terms each: hi = round(x), lo = round(x - hi).
__device__ __forceinline__ void two_terms(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  lo = pack_bf16(a - __uint_as_float(hi << 16), b - __uint_as_float(hi & 0xffff0000u));
}
__device__ __forceinline__ void unpack8(uint4 raw, float (&x)[8]) {
  const __nv_bfloat162* p = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 f = __bfloat1622float2(p[e]);
    x[2 * e] = f.x;
    x[2 * e + 1] = f.y;
  }
}
// Byte offset of 16-byte word `word` (8 elements) of row `row` in the tensor cores' layout: blocks of 64 elements,
// [rows][128 bytes] each with the 128-byte swizzle, `block_bytes` apart.
__device__ __forceinline__ uint32_t operand_offset(int row, int word, int block_bytes) {
  return (uint32_t)((word >> 3) * block_bytes + row * 128 + (((word & 7) ^ (row & 7)) << 4));
}
// Eight values as one or two bfloat16 terms, a 16-byte word each.
__device__ __forceinline__ void put_terms(const float (&x)[8], uint8_t* hi, uint8_t* lo, uint32_t at) {
  uint32_t h[4], l[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) two_terms(x[2 * e], x[2 * e + 1], h[e], l[e]);
  *reinterpret_cast<uint4*>(hi + at) = make_uint4(h[0], h[1], h[2], h[3]);
  if (lo != nullptr) *reinterpret_cast<uint4*>(lo + at) = make_uint4(l[0], l[1], l[2], l[3]);
}

// A chunk's rows of one head's queries or keys (columns col0 .. col0 + dk - 1 of the projection) as one or two (lo not
// null) bfloat16 terms in `blocks` blocks of 64 elements, zeros beyond row n and column dk. Times `scale`, and if
// WEIGHTED times decay^(n - 1 - row). ROTATED: with a rotation (no activation), else perhaps with SiLU. The loads of
// BATCH words of a thread are in flight together.
template <bool WEIGHTED, bool ROTATED>
__device__ __forceinline__ void stage_rows(const bf16* __restrict__ proj, int64_t stride, int64_t start, int n, int col0, int dk, int blocks,
                                           int silu, const float2* __restrict__ turns, int rot_half, float scale, float log2_decay,
                                           uint8_t* hi, uint8_t* lo) {
  constexpr int BATCH = ROTATED ? 2 : 4;
  const int shift = blocks == 1 ? 3 : 4, total = CHUNK << shift;        // words of a row: 8 or 16
  const bool wide = dk % 8 == 0 && stride % 8 == 0 && col0 % 8 == 0 && (!ROTATED || rot_half % 8 == 0);
  for (int i0 = threadIdx.x; i0 < total; i0 += BATCH * CHUNK_THREADS) {
    uint4 raw[BATCH], other[ROTATED ? BATCH : 1];
    float4 cs[ROTATED ? BATCH : 1][4];
    if (wide) {
#pragma unroll
      for (int b = 0; b < BATCH; ++b) {
        const int i = i0 + b * CHUNK_THREADS, r = i >> shift, e0 = (i & ((1 << shift) - 1)) * 8;
        raw[b] = make_uint4(0, 0, 0, 0);
        if (r < n && e0 < dk) {                        // (n <= CHUNK: words beyond the total are left out too)
          const bf16* src = proj + (start + r) * stride + col0;
          raw[b] = *reinterpret_cast<const uint4*>(src + e0);
          if (ROTATED && e0 < 2 * rot_half) {
            const bool low = e0 < rot_half;
            other[ROTATED ? b : 0] = *reinterpret_cast<const uint4*>(src + (low ? e0 + rot_half : e0 - rot_half));
            const float4* t = reinterpret_cast<const float4*>(turns + (start + r) * rot_half + (low ? e0 : e0 - rot_half));
#pragma unroll
            for (int e = 0; e < 4; ++e) cs[ROTATED ? b : 0][e] = t[e];
          }
        }
      }
    }
#pragma unroll
    for (int b = 0; b < BATCH; ++b) {
      const int i = i0 + b * CHUNK_THREADS, r = i >> shift, word = i & ((1 << shift) - 1), e0 = word * 8;
      if (i >= total) continue;
      float x[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) x[e] = 0.f;
      if (r < n && e0 < dk) {
        if (wide) {
          unpack8(raw[b], x);
          if (!ROTATED && silu) {
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] = rounded_to<bf16>(quick_silu(x[e]));
          }
          if (ROTATED && e0 < 2 * rot_half) {
            const bool low = e0 < rot_half;
            float y[8];
            unpack8(other[ROTATED ? b : 0], y);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float4 a = cs[ROTATED ? b : 0][e];
              x[2 * e] = x[2 * e] * a.x + y[2 * e] * (low ? -a.y : a.y);
              x[2 * e + 1] = x[2 * e + 1] * a.z + y[2 * e + 1] * (low ? -a.w : a.w);
            }
          }
        } else {
          const bf16* src = proj + (start + r) * stride + col0;
#pragma unroll
          for (int e = 0; e < 8; ++e) {
            const int j = e0 + e;
            if (j >= dk) continue;
            float v = to_f32(src[j]);
            if (!ROTATED && silu) v = rounded_to<bf16>(quick_silu(v));
            if (ROTATED && j < 2 * rot_half) {
              const bool low = j < rot_half;
              const float2 a = turns[(start + r) * rot_half + (low ? j : j - rot_half)];
              v = v * a.x + to_f32(src[low ? j + rot_half : j - rot_half]) * (low ? -a.y : a.y);
            }
            x[e] = v;
          }
        }
        const float by = WEIGHTED ? scale * exp2f(log2_decay * (float)(n - 1 - r)) : scale;
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] *= by;
      }
      put_terms(x, hi, lo, operand_offset(r, word, BLOCK_BYTES));
    }
  }
}

// A chunk's values, columns v0 .. of one head in `blocks` blocks of 64 elements, zeros beyond row n and column dv.
__device__ __forceinline__ void stage_values(const bf16* __restrict__ proj, int64_t stride, int64_t start, int n, int col0, int v0, int dv,
                                             int blocks, int silu, uint8_t* vs) {
  constexpr int BATCH = 4;
  const int shift = blocks == 1 ? 3 : 4, total = CHUNK << shift;
  const bool wide = dv % 8 == 0 && stride % 8 == 0 && col0 % 8 == 0;
  for (int i0 = threadIdx.x; i0 < total; i0 += BATCH * CHUNK_THREADS) {
    uint4 raw[BATCH];
#pragma unroll
    for (int b = 0; b < BATCH; ++b) {
      const int i = i0 + b * CHUNK_THREADS, r = i >> shift, e0 = (i & ((1 << shift) - 1)) * 8;
      raw[b] = make_uint4(0, 0, 0, 0);
      if (r < n && v0 + e0 < dv) {
        const bf16* src = proj + (start + r) * stride + col0 + v0 + e0;
        if (wide) {
          raw[b] = *reinterpret_cast<const uint4*>(src);
        } else {
          bf16* x = reinterpret_cast<bf16*>(&raw[b]);
#pragma unroll
          for (int e = 0; e < 8; ++e)
            if (v0 + e0 + e < dv) x[e] = src[e];
        }
      }
    }
#pragma unroll
    for (int b = 0; b < BATCH; ++b) {
      const int i = i0 + b * CHUNK_THREADS, r = i >> shift, word = i & ((1 << shift) - 1);
      if (i >= total) continue;
      if (silu) {
        float x[8];
        unpack8(raw[b], x);
#pragma unroll
        for (int e = 0; e < 8; ++e) x[e] = quick_silu(x[e]);
        raw[b] = make_uint4(pack_bf16(x[0], x[1]), pack_bf16(x[2], x[3]), pack_bf16(x[4], x[5]), pack_bf16(x[6], x[7]));
      }
      *reinterpret_cast<uint4*>(vs + operand_offset(r, word, BLOCK_BYTES)) = raw[b];
    }
  }
}

__device__ __forceinline__ int chunk_rows(const Recurrence& c, const Chunks& k, int chunk, int64_t& start) {
  const int b = k.request[chunk];
  start = c.cu_q[b] + k.first[chunk];
  return min(CHUNK, (int)(c.cu_q[b + 1] - start));
}
__host__ __device__ __forceinline__ int blocks_of(int elements) { return (elements + 63) / 64; }       // blocks of 64 elements

// Instruction descriptor for kind::f16 with A MN-major too (rows of A's tile are the K index).
__host__ __device__ constexpr uint32_t instr_both_mn(int n) { return umma_instr_desc(CHUNK, n, true) | (1u << 15); }

// An operand in shared memory: its descriptor, and how it moves on along K: `step` bytes for 16 elements, after
// `per_block` steps to the next block, `block_bytes` further on.
struct Operand {
  uint64_t desc;
  int step, per_block, block_bytes;
  __device__ __forceinline__ uint64_t at(int k) const {
    return desc + (uint64_t)(((k / per_block) * block_bytes + (k % per_block) * step) >> 4);
  }
};
__device__ __forceinline__ Operand k_major(uint32_t addr) { return Operand{smem_desc_sw128(addr), 32, 4, BLOCK_BYTES}; }
__device__ __forceinline__ Operand mn_major(uint32_t addr, int block_bytes) { return Operand{smem_desc_sw128_mn(addr, (uint32_t)block_bytes), 16 * 128, 1 << 20, 0}; }
// D += A B over `steps` steps of 16 along K (the first MMA of a sum overwrites D). One thread.
__device__ __forceinline__ void multiply(uint32_t tmem, const Operand& a, const Operand& b, uint32_t idesc, int steps, bool& started) {
  for (int k = 0; k < steps; ++k) {
    umma_bf16(tmem, a.at(k), b.at(k), idesc, started ? 1u : 0u);
    started = true;
  }
}

// What the two kernels have in common: barriers and tensor memory, operands, the way out.
template <int BARS>
__device__ __forceinline__ void tensor_setup(uint64_t (&bars)[BARS], uint32_t* holder, volatile int* abort_flag, uint32_t cols) {
  if (threadIdx.x == 0) {
    *abort_flag = 0;
    for (int i = 0; i < BARS; ++i) mbar_init(smem_u32(&bars[i]), 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (threadIdx.x < 32) tmem_alloc(smem_u32(holder), cols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_launch_dependents();            // after the tensor memory is ours: a dependent must not take it first
}
// Every thread's writes to shared memory are seen by the tensor cores after this.
__device__ __forceinline__ void operands_ready() {
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
}
__device__ __forceinline__ void tensor_leave(uint32_t tmem, uint32_t cols, volatile int* abort_flag) {
  tc_fence_before();
  __syncthreads();
  if (*abort_flag) {
    for (int i = 0; i < 64; ++i) __nanosleep(1000);
    __syncthreads();
  }
  if (threadIdx.x < 32) {
    tc_fence_after();
    tmem_dealloc(tmem, cols);
  }
}

constexpr uint32_t STATE_TMEM = 128;

// grid (chunks, heads, value tiles): U[dk, dv] = K^T V, the head's key channels on the MMA's M side (128, zeros beyond dk).
template <bool ROTATED>
__global__ void __launch_bounds__(CHUNK_THREADS, 2)
decay_chunk_state_kernel(const Projection p, const Recurrence c, const Chunks k, unsigned* status) {
  extern __shared__ uint8_t chunk_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(chunk_raw) + 1023) & ~(uintptr_t)1023);
  __shared__ __align__(8) uint64_t done[1];
  __shared__ uint32_t tmem_holder;
  __shared__ volatile int abort_flag;
  pdl_wait();
  const int chunk = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * VT;
  const int dk = c.dk, dv = c.dv;
  int64_t start;
  const int n = chunk_rows(c, k, chunk, start);
  if (n <= 0) return;                                  // (the whole block: nothing is allocated yet)
  const int vblocks = blocks_of(min(dv - v0, VT));
  uint8_t* kh = smem;                                  // two blocks of 64 key channels
  uint8_t* kl = kh + 2 * BLOCK_BYTES;
  uint8_t* vs = kl + 2 * BLOCK_BYTES;                  // [vblocks]
  tensor_setup(done, &tmem_holder, &abort_flag, STATE_TMEM);
  const uint32_t tmem = tmem_holder;
  const bf16* proj = reinterpret_cast<const bf16*>(p.data);
  stage_rows<true, ROTATED>(proj, p.stride, start, n, p.off_k + h * dk, dk, 2, c.silu, k.turns, c.rot_half, c.key_scale, c.log2_decay[h], kh, kl);
  stage_values(proj, p.stride, start, n, p.off_v + h * dv, v0, dv, vblocks, c.silu, vs);
  operands_ready();
  if (threadIdx.x == 0) {
    const uint32_t idesc = instr_both_mn(64 * vblocks);
    const Operand v = mn_major(smem_u32(vs), BLOCK_BYTES);
    bool started = false;
    multiply(tmem, mn_major(smem_u32(kh), BLOCK_BYTES), v, idesc, (n + 15) / 16, started);
    multiply(tmem, mn_major(smem_u32(kl), BLOCK_BYTES), v, idesc, (n + 15) / 16, started);
    umma_commit(smem_u32(&done[0]));
  }
  __syncwarp();
  const bool ok = mbar_wait_warp(smem_u32(&done[0]), 0, &abort_flag, status);
  tc_fence_after();
  // a thread a key channel and 32 value columns
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, row = (warp & 3) * 32 + lane, c0 = (warp >> 2) * 32;
  if (ok && c0 < 64 * vblocks) {
    uint32_t r[32];
    tmem_load32(tmem + ((uint32_t)((warp & 3) * 32) << 16) + (uint32_t)c0, r);
    if (row < dk) {
      float* dst = k.states + (((int64_t)chunk * c.heads + h) * dk + row) * dv + v0 + c0;
      if (dv % 4 == 0) {
#pragma unroll
        for (int j = 0; j < 8; ++j)
          if (v0 + c0 + 4 * j < dv)
            reinterpret_cast<float4*>(dst)[j] = make_float4(__uint_as_float(r[4 * j]), __uint_as_float(r[4 * j + 1]), __uint_as_float(r[4 * j + 2]), __uint_as_float(r[4 * j + 3]));
      } else {
#pragma unroll
        for (int j = 0; j < 32; ++j)
          if (v0 + c0 + j < dv) dst[j] = __uint_as_float(r[j]);
      }
    }
  }
  tensor_leave(tmem, STATE_TMEM, &abort_flag);
}

// V floats a thread. long_requests: which requests; chunk0: a request's first chunk.
template <int V>
__global__ void __launch_bounds__(256)
decay_chunk_scan_kernel(const Recurrence c, const int* __restrict__ long_requests, const int* __restrict__ chunk0, float* __restrict__ states) {
  pdl_wait();
  pdl_launch_dependents();
  const int b = long_requests[blockIdx.z], h = blockIdx.y;
  const int slot = c.state_slots[b], n = c.cu_q[b + 1] - c.cu_q[b];
  const int64_t size = (int64_t)c.dk * c.dv, i = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (i >= size || slot < 0 || slot >= c.num_slots) return;
  const int chunks = (n + CHUNK - 1) / CHUNK;
  const int64_t step = (int64_t)c.heads * size;
  float* S = c.state + (int64_t)slot * c.state_stride + (int64_t)h * size + i;
  float* at = states + ((int64_t)chunk0[blockIdx.z] * c.heads + h) * size + i;
  const float whole = exp2f(c.log2_decay[h] * (float)CHUNK), last = exp2f(c.log2_decay[h] * (float)(n - (chunks - 1) * CHUNK));
  float s[V];
#pragma unroll
  for (int e = 0; e < V; ++e) s[e] = S[e];
  constexpr int AHEAD = 8;
  for (int k0 = 0; k0 < chunks; k0 += AHEAD) {
    float u[AHEAD][V];
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
      if (k0 + k >= chunks) continue;
      if (V == 4) {
        const float4 x = *reinterpret_cast<const float4*>(at + (k0 + k) * step);
        u[k][0] = x.x; u[k][V > 1 ? 1 : 0] = x.y; u[k][V > 2 ? 2 : 0] = x.z; u[k][V > 3 ? 3 : 0] = x.w;
      } else {
        u[k][0] = at[(k0 + k) * step];
      }
    }
#pragma unroll
    for (int k = 0; k < AHEAD; ++k) {
      if (k0 + k >= chunks) continue;
      if (V == 4) *reinterpret_cast<float4*>(at + (k0 + k) * step) = make_float4(s[0], s[V > 1 ? 1 : 0], s[V > 2 ? 2 : 0], s[V > 3 ? 3 : 0]);
      else at[(k0 + k) * step] = s[0];
      const float by = k0 + k + 1 < chunks ? whole : last;
#pragma unroll
      for (int e = 0; e < V; ++e) s[e] = fmaf(by, s[e], u[k][e]);
    }
  }
#pragma unroll
  for (int e = 0; e < V; ++e) S[e] = s[e];
}

constexpr uint32_t OUT_TMEM = 512, SCORE_COL = 0, CARRIED_COL = 128, INNER_COL = 256;

// What may follow a head's read-out at once where a block holds the whole head: unit root mean square and gate.
struct HeadOut {
  bf16* y;                              // [tokens, heads * dv], or null: the read-outs go out as they are
  float eps;
  int gate_silu;
};

// grid (chunks, heads, value tiles). LO: queries and keys have a second term (they are rotated); else they are bfloat16
// (SiLU'd activations). Scores Q K^T, the carried part Q S and the inner part P V have tensor memory of their own;
// P, the decayed scores in two terms, takes the place of the queries and keys.
template <bool LO>
__global__ void __launch_bounds__(CHUNK_THREADS, 1)
decay_chunk_out_kernel(const Projection p, const Recurrence c, const Chunks k, float* __restrict__ out, const HeadOut fin, unsigned* status) {
  extern __shared__ uint8_t chunk_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(chunk_raw) + 1023) & ~(uintptr_t)1023);
  __shared__ __align__(8) uint64_t done[3];
  __shared__ uint32_t tmem_holder;
  __shared__ volatile int abort_flag;
  pdl_wait();
  const int chunk = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * VT;
  const int dk = c.dk, dv = c.dv;
  int64_t start;
  const int n = chunk_rows(c, k, chunk, start);
  if (n <= 0) return;
  const int kblocks = blocks_of(dk), vblocks = blocks_of(min(dv - v0, VT));
  const int q_bytes = kblocks * BLOCK_BYTES, s_block = 64 * kblocks * 128;
  uint8_t* qh = smem;
  uint8_t* ql = qh + (LO ? q_bytes : 0);
  uint8_t* kh = ql + q_bytes;
  uint8_t* kl = kh + (LO ? q_bytes : 0);
  uint8_t* ph = smem;                                  // after the queries and keys have been read: two blocks of 64 keys a term
  uint8_t* pl = ph + 2 * BLOCK_BYTES;
  uint8_t* vs = smem + max((LO ? 4 : 2) * q_bytes, 4 * BLOCK_BYTES);
  uint8_t* sh = vs + vblocks * BLOCK_BYTES;            // [vblocks][64 * kblocks rows][64 columns]
  uint8_t* sl = sh + vblocks * s_block;
  tensor_setup(done, &tmem_holder, &abort_flag, OUT_TMEM);
  const uint32_t tmem = tmem_holder;
  const bf16* proj = reinterpret_cast<const bf16*>(p.data);
  const float l2d = c.log2_decay[h];
  stage_rows<false, LO>(proj, p.stride, start, n, p.off_q + h * dk, dk, kblocks, c.silu, k.turns, c.rot_half, 1.f, 0.f, qh, LO ? ql : nullptr);
  stage_rows<false, LO>(proj, p.stride, start, n, p.off_k + h * dk, dk, kblocks, c.silu, k.turns, c.rot_half, c.key_scale, 0.f, kh, LO ? kl : nullptr);
  operands_ready();
  if (threadIdx.x == 0) {
    const uint32_t idesc = umma_instr_desc(CHUNK, CHUNK, false);
    bool started = false;
    multiply(tmem + SCORE_COL, k_major(smem_u32(qh)), k_major(smem_u32(kh)), idesc, 4 * kblocks, started);
    if (LO) {
      multiply(tmem + SCORE_COL, k_major(smem_u32(ql)), k_major(smem_u32(kh)), idesc, 4 * kblocks, started);
      multiply(tmem + SCORE_COL, k_major(smem_u32(qh)), k_major(smem_u32(kl)), idesc, 4 * kblocks, started);
    }
    umma_commit(smem_u32(&done[0]));
  }
  __syncwarp();
  // the state before the chunk and the values, while the scores are made
  {
    const float* S = k.states + ((int64_t)chunk * c.heads + h) * dk * dv + v0;
    constexpr int BATCH = 4;
    const int shift = vblocks == 1 ? 3 : 4, total = 64 * kblocks << shift;
    const bool wide = dv % 4 == 0;
    for (int i0 = threadIdx.x; i0 < total; i0 += BATCH * CHUNK_THREADS) {
      float x[BATCH][8];
#pragma unroll
      for (int b = 0; b < BATCH; ++b) {
        const int i = i0 + b * CHUNK_THREADS, r = i >> shift, e0 = (i & ((1 << shift) - 1)) * 8;
#pragma unroll
        for (int e = 0; e < 8; ++e) x[b][e] = 0.f;
        if (r < dk) {                                  // (dk <= 64 * kblocks: words beyond the total are left out too)
          const float* src = S + (int64_t)r * dv + e0;
          if (wide) {
            if (v0 + e0 < dv) {
              const float4 a = *reinterpret_cast<const float4*>(src);
              x[b][0] = a.x; x[b][1] = a.y; x[b][2] = a.z; x[b][3] = a.w;
            }
            if (v0 + e0 + 4 < dv) {
              const float4 a = *reinterpret_cast<const float4*>(src + 4);
              x[b][4] = a.x; x[b][5] = a.y; x[b][6] = a.z; x[b][7] = a.w;
            }
          } else {
#pragma unroll
            for (int e = 0; e < 8; ++e)
              if (v0 + e0 + e < dv) x[b][e] = src[e];
          }
        }
      }
#pragma unroll
      for (int b = 0; b < BATCH; ++b) {
        const int i = i0 + b * CHUNK_THREADS;
        if (i < total) put_terms(x[b], sh, sl, operand_offset(i >> shift, i & ((1 << shift) - 1), s_block));
      }
    }
  }
  stage_values(proj, p.stride, start, n, p.off_v + h * dv, v0, dv, vblocks, c.silu, vs);
  operands_ready();
  const uint32_t idesc_v = umma_instr_desc(CHUNK, 64 * vblocks, true);
  if (threadIdx.x == 0) {
    bool started = false;
    multiply(tmem + CARRIED_COL, k_major(smem_u32(qh)), mn_major(smem_u32(sh), s_block), idesc_v, 4 * kblocks, started);
    multiply(tmem + CARRIED_COL, k_major(smem_u32(qh)), mn_major(smem_u32(sl), s_block), idesc_v, 4 * kblocks, started);
    if (LO) multiply(tmem + CARRIED_COL, k_major(smem_u32(ql)), mn_major(smem_u32(sh), s_block), idesc_v, 4 * kblocks, started);
    umma_commit(smem_u32(&done[1]));
  }
  __syncwarp();
  // ---- the decayed scores: a thread a token and 32 keys
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, row = (warp & 3) * 32 + lane, part = warp >> 2, c0 = part * 32;
  const uint32_t lanes = tmem + ((uint32_t)((warp & 3) * 32) << 16);
  bool ok = mbar_wait_warp(smem_u32(&done[0]), 0, &abort_flag, status);
  ok = ok && mbar_wait_warp(smem_u32(&done[1]), 0, &abort_flag, status);      // (the queries may be overwritten)
  tc_fence_after();
  if (ok) {
    uint32_t r[32];
    tmem_load32(lanes + SCORE_COL + c0, r);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      float x[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int back = row - (c0 + 8 * w + e);
        x[e] = back >= 0 ? __uint_as_float(r[8 * w + e]) * fast_exp2(l2d * (float)back) : 0.f;
      }
      put_terms(x, ph, pl, operand_offset(row, c0 / 8 + w, BLOCK_BYTES));
    }
  }
  operands_ready();
  if (threadIdx.x == 0 && ok) {
    const Operand v = mn_major(smem_u32(vs), BLOCK_BYTES);
    const int steps = (n + 15) / 16;
    bool started = false;
    multiply(tmem + INNER_COL, k_major(smem_u32(ph)), v, idesc_v, steps, started);
    multiply(tmem + INNER_COL, k_major(smem_u32(pl)), v, idesc_v, steps, started);
    umma_commit(smem_u32(&done[2]));
  }
  __syncwarp();
  // ---- carried part times decay^(token + 1), plus the inner part: a thread a token and 32 value columns
  const bool mine = c0 < 64 * vblocks;
  float o[32];
  {
    uint32_t r[32];
    const float by = exp2f(l2d * (float)(row + 1));
    if (ok && mine) {
      tmem_load32(lanes + CARRIED_COL + c0, r);
#pragma unroll
      for (int j = 0; j < 32; ++j) o[j] = __uint_as_float(r[j]) * by;
    }
    ok = ok && mbar_wait_warp(smem_u32(&done[2]), 0, &abort_flag, status);
    tc_fence_after();
    if (ok && mine) {
      tmem_load32(lanes + INNER_COL + c0, r);
#pragma unroll
      for (int j = 0; j < 32; ++j) o[j] += __uint_as_float(r[j]);
    }
  }
  if (fin.y != nullptr) {
    // (one value tile: the block holds the whole head, columns beyond dv are zero)
    float* squares = reinterpret_cast<float*>(smem);     // [4][CHUNK], in the place of the decayed scores, which have been read
    float ss = 0.f;
    if (ok && mine) {
#pragma unroll
      for (int j = 0; j < 32; ++j) ss += o[j] * o[j];
    }
    squares[part * CHUNK + row] = ss;
    __syncthreads();
    const float inv = 1.f / sqrtf((squares[row] + squares[CHUNK + row] + squares[2 * CHUNK + row] + squares[3 * CHUNK + row]) / (float)dv + fin.eps);
    if (ok && mine && row < n) {
      const int64_t at = (start + row) * p.stride + p.off_g + (int64_t)h * dv + c0;
      bf16* dst = fin.y + ((start + row) * c.heads + h) * dv + c0;
      const bool words = dv % 8 == 0 && p.stride % 8 == 0 && p.off_g % 8 == 0;
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        if (words) {
          if (c0 + 8 * w < dv) {
            float g[8];
            unpack8(*reinterpret_cast<const uint4*>(proj + at + 8 * w), g);
            uint32_t v[4];
#pragma unroll
            for (int e = 0; e < 4; ++e)
              v[e] = pack_bf16(o[8 * w + 2 * e] * inv * quick_gate(g[2 * e], fin.gate_silu), o[8 * w + 2 * e + 1] * inv * quick_gate(g[2 * e + 1], fin.gate_silu));
            *reinterpret_cast<uint4*>(dst + 8 * w) = make_uint4(v[0], v[1], v[2], v[3]);
          }
        } else {
#pragma unroll
          for (int e = 0; e < 8; ++e)
            if (c0 + 8 * w + e < dv) dst[8 * w + e] = __float2bfloat16_rn(o[8 * w + e] * inv * quick_gate(to_f32(proj[at + 8 * w + e]), fin.gate_silu));
        }
      }
    }
  } else if (ok && mine && row < n) {
    float* dst = out + (start + row) * c.heads * dv + (int64_t)h * dv + v0 + c0;
    if (dv % 4 == 0) {
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (v0 + c0 + 4 * j < dv) reinterpret_cast<float4*>(dst)[j] = make_float4(o[4 * j], o[4 * j + 1], o[4 * j + 2], o[4 * j + 3]);
    } else {
#pragma unroll
      for (int j = 0; j < 32; ++j)
        if (v0 + c0 + j < dv) dst[j] = o[j];
    }
  }
  tensor_leave(tmem, OUT_TMEM, &abort_flag);
}

size_t state_smem(int dv) { return 1024 + (size_t)(4 + blocks_of(dv < VT ? dv : VT)) * BLOCK_BYTES; }
size_t out_smem(int dk, int dv, bool lo) {
  const size_t kb = blocks_of(dk), vb = blocks_of(dv < VT ? dv : VT), rows = (lo ? 4 : 2) * kb;
  return 1024 + ((rows > 4 ? rows : 4) + vb + vb * kb) * BLOCK_BYTES;      // (a term of the state: vb * kb blocks of 64 rows)
}

// ------------------------------------------------------------------ norm and gate
// V neighbouring gates of token t from column off_g + i on, summed and rounded like `column`.
template <typename T, int V>
__device__ __forceinline__ void load_gates(const Projection& p, int64_t t, int i, int silu, float (&g)[V]) {
  const int64_t at = t * p.stride + p.off_g + i;
  if (V == 1) {
    g[0] = gate_value(column<T>(p, t, p.off_g + i), silu);
    return;
  }
  float4 v;
  if (p.splits == 0 && sizeof(T) == 2) {
    const uint2 raw = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p.data) + at);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v = make_float4(a.x, a.y, b.x, b.y);
  } else {
    const float* src = reinterpret_cast<const float*>(p.data) + at;
    v = *reinterpret_cast<const float4*>(src);
    for (int s = 1; s < p.splits; ++s) {
      const float4 u = *reinterpret_cast<const float4*>(src + s * p.plane);
      v.x += u.x; v.y += u.y; v.z += u.z; v.w += u.w;
    }
    v = make_float4(rounded_to<T>(v.x), rounded_to<T>(v.y), rounded_to<T>(v.z), rounded_to<T>(v.w));
  }
  g[0] = gate_value(v.x, silu);
  g[V > 1 ? 1 : 0] = gate_value(v.y, silu);
  g[V > 2 ? 2 : 0] = gate_value(v.z, silu);
  g[V > 3 ? 3 : 0] = gate_value(v.w, silu);
}
template <int V>
__device__ __forceinline__ void load_row(const float* p, float (&x)[V]) {
  if (V == 4) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    x[0] = v.x; x[V > 1 ? 1 : 0] = v.y; x[V > 2 ? 2 : 0] = v.z; x[V > 3 ? 3 : 0] = v.w;
  } else {
    x[0] = p[0];
  }
}
template <int V> __device__ __forceinline__ void store_row(float* p, const float (&x)[V]) {
  if (V == 4) *reinterpret_cast<float4*>(p) = make_float4(x[0], x[V > 1 ? 1 : 0], x[V > 2 ? 2 : 0], x[V > 3 ? 3 : 0]);
  else p[0] = x[0];
}
template <int V> __device__ __forceinline__ void store_row(bf16* p, const float (&x)[V]) {
  if (V == 4) *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(x[0], x[V > 1 ? 1 : 0]), pack_bf16(x[V > 2 ? 2 : 0], x[V > 3 ? 3 : 0]));
  else p[0] = __float2bfloat16_rn(x[0]);
}

// One root mean square over the whole row (all heads together), times a weight [width]. A block a token; V elements a
// thread at a time.
template <typename T, int V>
__global__ void __launch_bounds__(1024)
decay_out_joint_kernel(const float* __restrict__ o, const Projection p, int width, const void* __restrict__ w, int w_f32, float eps,
                       int gate_silu, T* __restrict__ y) {
  __shared__ float scratch[32];
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  const int words = width / V, step = blockDim.x;
  const float* row = o + t * width;
  float ss = 0.f;
  for (int n = threadIdx.x; n < words; n += step) {
    float x[V];
    load_row<V>(row + n * V, x);
#pragma unroll
    for (int e = 0; e < V; ++e) ss += x[e] * x[e];
  }
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
  for (int n = threadIdx.x; n < words; n += step) {
    float x[V], g[V];
    load_row<V>(row + n * V, x);
    load_gates<T, V>(p, t, n * V, gate_silu, g);
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = x[e] * inv * load_flex(w, w_f32, n * V + e) * g[e];
    store_row<V>(y + t * width + n * V, x);
  }
}

// Every head by its own root mean square, no weight. A warp a head.
template <typename T, int V>
__global__ void __launch_bounds__(256)
decay_out_heads_kernel(const float* __restrict__ o, const Projection p, int heads, int dv, float eps, int gate_silu, T* __restrict__ y) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t t = blockIdx.x;
  const int lane = threadIdx.x & 31, h = blockIdx.y * 8 + (threadIdx.x >> 5);
  if (h >= heads) return;
  const int words = dv / V;
  const float* row = o + (t * heads + h) * dv;
  float ss = 0.f;
  for (int n = lane; n < words; n += 32) {
    float x[V];
    load_row<V>(row + n * V, x);
#pragma unroll
    for (int e = 0; e < V; ++e) ss += x[e] * x[e];
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)dv + eps);
  for (int n = lane; n < words; n += 32) {
    float x[V], g[V];
    load_row<V>(row + n * V, x);
    load_gates<T, V>(p, t, h * dv + n * V, gate_silu, g);
#pragma unroll
    for (int e = 0; e < V; ++e) x[e] = x[e] * inv * g[e];
    store_row<V>(y + (t * heads + h) * dv + n * V, x);
  }
}

template <typename T, int V>
void launch_decay_out(const float* o, const Projection& p, int tokens, int heads, int dv, int joint, const void* w, int w_f32, float eps,
                      int gate_silu, void* y, cudaStream_t stream) {
  if (!joint) {
    vosti_launch(decay_out_heads_kernel<T, V>, dim3(tokens, (heads + 7) / 8), dim3(256), 0, stream, o, p, heads, dv, eps, gate_silu, (T*)y);
    return;
  }
  const int width = heads * dv, wanted = (width / V + 31) / 32 * 32;
  const int threads = tokens > 64 || wanted < 256 ? 256 : wanted > 1024 ? 1024 : wanted;      // few rows: a thread a word
  vosti_launch(decay_out_joint_kernel<T, V>, dim3(tokens), dim3(threads), 0, stream, o, p, width, w, w_f32, eps, gate_silu, (T*)y);
}

template <typename T, int V>
void launch_scan(const Projection& p, const Recurrence& c, float* out, int requests, int max_len, cudaStream_t stream) {
  const dim3 grid((c.dv + SCAN_LANES * V - 1) / (SCAN_LANES * V), c.heads, requests);
  const size_t smem = (size_t)2 * SCAN_TOKENS * c.rot_half * sizeof(float);
  if (c.dk <= 64) vosti_launch(decay_scan_kernel<T, V, 2>, grid, dim3(SCAN_THREADS), smem, stream, p, c, out, max_len);
  else if (c.dk <= 128) vosti_launch(decay_scan_kernel<T, V, 4>, grid, dim3(SCAN_THREADS), smem, stream, p, c, out, max_len);
  else vosti_launch(decay_scan_kernel<T, V, 8>, grid, dim3(SCAN_THREADS), smem, stream, p, c, out, max_len);
}
}  // namespace

#define VOSTI_DECAY_CHECKS(name)                                                                                                       \
  VOSTI_REQUIRE(heads > 0 && dk > 0 && dk <= MAX_DK && dv > 0 && requests >= 0 && splits >= 0, name ": bad sizes heads=%d dk=%d dv=%d", heads, dk, dv); \
  VOSTI_REQUIRE(heads <= 65535 && requests <= 65535, name ": too many heads or requests for one launch");                              \
  VOSTI_REQUIRE(state_stride >= (int64_t)heads * dk * dv && state_stride % 4 == 0, name ": the state slots are too small");            \
  VOSTI_REQUIRE(rot_half >= 0 && 2 * rot_half <= dk && (rot_half == 0 || (freq != nullptr && positions != nullptr)), name ": the rotation takes at most the whole head"); \
  VOSTI_REQUIRE(!(silu && rot_half > 0), name ": SiLU or a rotation, not both")

// proj: the serving type [tokens, stride] (splits 0) or float32 [splits, tokens, stride]. Requests with more than max_len
// tokens are left out (0: none is). out: float32 [tokens, heads * dv].
VOSTI_API int vosti_decay_scan(const void* proj, int splits, int64_t stride, int tokens, int off_q, int off_k, int off_v, int heads, int dk,
                               int dv, int silu, const float* decay, float key_scale, const float* freq, int rot_half,
                               const int* positions, float* state, int64_t state_stride, const int* cu_q, const int* state_slots,
                               int num_slots, int requests, int max_len, float* out, int is_f32, cudaStream_t stream) {
  VOSTI_DECAY_CHECKS("decay_scan");
  if (tokens == 0 || requests == 0) return VOSTI_OK;
  const Projection p = {proj, splits, stride, (int64_t)tokens * stride, off_q, off_k, off_v, 0};
  const Recurrence c = {heads, dk, dv, silu, decay, nullptr, key_scale, freq, rot_half, positions, state, state_stride, cu_q, state_slots, num_slots};
  if (is_f32) {
    if (dv % 4 == 0) launch_scan<float, 4>(p, c, out, requests, max_len, stream);
    else launch_scan<float, 1>(p, c, out, requests, max_len, stream);
  } else {
    if (dv % 4 == 0) launch_scan<bf16, 4>(p, c, out, requests, max_len, stream);
    else launch_scan<bf16, 1>(p, c, out, requests, max_len, stream);
  }
  VOSTI_LAUNCH_CHECK();
}

// Tokens of a chunk, and whether the chunk kernels take heads of this width.
VOSTI_API int vosti_decay_chunk() { return CHUNK; }
VOSTI_API int vosti_decay_chunk_fits(int dk) { return dk > 0 && dk <= CHUNK_MAX_DK; }

// out float32 pairs [tokens, half]: cosine and sine of positions[t] * freq[i].
VOSTI_API int vosti_rotation_table(const float* freq, int half, const int* positions, int tokens, void* out, cudaStream_t stream) {
  VOSTI_REQUIRE(half > 0 && tokens >= 0 && freq != nullptr && positions != nullptr && out != nullptr, "rotation_table: bad arguments");
  if (tokens == 0) return VOSTI_OK;
  const int64_t n = (int64_t)tokens * half;
  const int blocks = (int)((n + 255) / 256 < 148 * 8 ? (n + 255) / 256 : 148 * 8);
  vosti_launch(rotation_table_kernel, dim3(blocks), dim3(256), 0, stream, freq, half, positions, n, (float2*)out);
  VOSTI_LAUNCH_CHECK();
}

// The long portions of a step: proj bfloat16 [tokens, stride]; chunk_request / chunk_first int32 [chunks] (see Chunks),
// long_requests / long_chunk0 int32 [longs]; turns the rotation table of the step's tokens, or null;
// states float32 scratch [chunks, heads, dk, dv]. With y (bfloat16 [tokens, heads * dv]; dv <= 128) every head's read-out is
// divided by its root mean square, gated by the columns from off_g on and written there; else out receives the read-outs.
VOSTI_API int vosti_decay_chunks(const void* proj, int64_t stride, int tokens, int off_q, int off_k, int off_v, int heads, int dk, int dv,
                                 int silu, const float* log2_decay, float key_scale, const float* freq, const void* turns, int rot_half,
                                 const int* positions, float* state, int64_t state_stride, const int* cu_q, const int* state_slots,
                                 int num_slots, const int* chunk_request, const int* chunk_first, int chunks, const int* long_requests,
                                 const int* long_chunk0, int requests, float* states, float* out, int off_g, float eps, int gate_silu,
                                 void* y, unsigned* status, cudaStream_t stream) {
  const int splits = 0;
  VOSTI_DECAY_CHECKS("decay_chunks");
  VOSTI_REQUIRE(dk <= CHUNK_MAX_DK, "decay_chunks: heads of %d (at most %d)", dk, CHUNK_MAX_DK);
  VOSTI_REQUIRE(rot_half == 0 || turns != nullptr, "decay_chunks: the rotation table is missing");
  VOSTI_REQUIRE(y != nullptr ? dv <= VT : out != nullptr, "decay_chunks: nowhere to write, or a head too wide to be normed at once");
  VOSTI_REQUIRE(((reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(states) | reinterpret_cast<uintptr_t>(turns) |
                  reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(y)) & 15) == 0,
                "decay_chunks: operands must be 16-byte aligned");
  if (tokens == 0 || chunks == 0) return VOSTI_OK;
  const Projection p = {proj, 0, stride, 0, off_q, off_k, off_v, off_g};
  const Recurrence c = {heads, dk, dv, silu, nullptr, log2_decay, key_scale, freq, rot_half, positions, state, state_stride, cu_q, state_slots, num_slots};
  const Chunks k = {chunk_request, chunk_first, (const float2*)turns, states};
  const HeadOut fin = {(bf16*)y, eps, gate_silu};
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(decay_chunk_state_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)state_smem(VT));
    cudaFuncSetAttribute(decay_chunk_state_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)state_smem(VT));
    cudaFuncSetAttribute(decay_chunk_out_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)out_smem(CHUNK_MAX_DK, VT, true));
    cudaFuncSetAttribute(decay_chunk_out_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)out_smem(CHUNK_MAX_DK, VT, false));
    configured = true;
  }
  const dim3 grid(chunks, heads, (dv + VT - 1) / VT);
  if (rot_half > 0) vosti_launch(decay_chunk_state_kernel<true>, grid, dim3(CHUNK_THREADS), state_smem(dv), stream, p, c, k, status);
  else vosti_launch(decay_chunk_state_kernel<false>, grid, dim3(CHUNK_THREADS), state_smem(dv), stream, p, c, k, status);
  const int64_t size = (int64_t)dk * dv;
  if (size % 4 == 0)
    vosti_launch(decay_chunk_scan_kernel<4>, dim3((unsigned)((size / 4 + 255) / 256), heads, requests), dim3(256), 0, stream, c, long_requests, long_chunk0, states);
  else
    vosti_launch(decay_chunk_scan_kernel<1>, dim3((unsigned)((size + 255) / 256), heads, requests), dim3(256), 0, stream, c, long_requests, long_chunk0, states);
  if (rot_half > 0) vosti_launch(decay_chunk_out_kernel<true>, grid, dim3(CHUNK_THREADS), out_smem(dk, dv, true), stream, p, c, k, out, fin, status);
  else vosti_launch(decay_chunk_out_kernel<false>, grid, dim3(CHUNK_THREADS), out_smem(dk, dv, false), stream, p, c, k, out, fin, status);
  VOSTI_LAUNCH_CHECK();
}

// o float32 [tokens, heads * dv]; the gate: columns off_g .. off_g + heads * dv - 1 of proj. joint: w [heads * dv].
VOSTI_API int vosti_decay_out(const float* o, const void* proj, int splits, int64_t stride, int off_g, int tokens, int heads, int dv,
                              int joint, const void* w, int w_f32, float eps, int gate_silu, void* y, int is_f32, cudaStream_t stream) {
  VOSTI_REQUIRE(tokens >= 0 && heads > 0 && dv > 0 && splits >= 0, "decay_out: bad sizes");
  VOSTI_REQUIRE(!joint || w != nullptr, "decay_out: the joint norm's weight is missing");
  if (tokens == 0) return VOSTI_OK;
  const Projection p = {proj, splits, stride, (int64_t)tokens * stride, 0, 0, 0, off_g};
  const bool words = dv % 4 == 0 && stride % 4 == 0 && off_g % 4 == 0 &&
                     ((reinterpret_cast<uintptr_t>(o) | reinterpret_cast<uintptr_t>(proj) | reinterpret_cast<uintptr_t>(y)) & 15) == 0;
#define VOSTI_OUT_ARGS o, p, tokens, heads, dv, joint, w, w_f32, eps, gate_silu, y, stream
  if (is_f32) {
    if (words) launch_decay_out<float, 4>(VOSTI_OUT_ARGS);
    else launch_decay_out<float, 1>(VOSTI_OUT_ARGS);
  } else {
    if (words) launch_decay_out<bf16, 4>(VOSTI_OUT_ARGS);
    else launch_decay_out<bf16, 1>(VOSTI_OUT_ARGS);
  }
#undef VOSTI_OUT_ARGS
  VOSTI_LAUNCH_CHECK();
}
