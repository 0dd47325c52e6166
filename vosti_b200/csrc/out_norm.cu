// The sublayer boundary of blocks that norm a sublayer's output only, over a float32 residual stream:
// one kernel closes a sublayer and opens the next one,
//
//   y  = the sublayer's output (see below)
//   x <- x + scale * y / sqrt(mean(y^2) + eps) * (offset + w)      scale a learned vector, or none
//
// and writes the stream (float32) and its rounding to the serving type, which the next sublayer
// reads. y is one of
//   * a row of a product: float32 or bfloat16, or float32 unsummed K splits added in split order,
//     plus an optional bias;
//   * a token's rows among rows sorted by expert: sum over picks of weight[t, k] * row[where[t, k]],
//     picks in order, each with its splits (weights absent: all `share`);
//   * the mean of two side-by-side branches' rows, each first divided by its own root mean square
//     (branch_eps) and multiplied by a weight of its own.
// y lies in shared memory between the passes; what the last pass reads besides (stream, norm weight,
// scale) is requested ahead, before the reductions.
#include "common.cuh"

namespace {

__device__ __forceinline__ float4 flex4(const void* p, int is_f32, int64_t i) {
  if (is_f32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
  const uint2 raw = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p) + i);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void put4(bf16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 raw;
  raw.x = *reinterpret_cast<const unsigned*>(&lo);
  raw.y = *reinterpret_cast<const unsigned*>(&hi);
  *reinterpret_cast<uint2*>(p) = raw;
}
__device__ __forceinline__ float dot4(float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }

constexpr int MAX_TERMS = 2;
struct OutNorm {
  const void* y[MAX_TERMS];          // [rows, width]; splits > 1: float32 [splits, rows, width], `plane` apart
  int y_f32[MAX_TERMS], splits[MAX_TERMS];
  int64_t plane[MAX_TERMS];
  int terms;                         // 1, or 2 branches
  const void* bias;                  // [width] or null (one term)
  int bias_f32;
  const int* where;                  // [rows, picks] rows of y, or null (one term)
  const float* pick_weights;         // [rows, picks], or null: `share`
  int picks, y_rows;
  float share;
  const void* branch_w[MAX_TERMS];
  int branch_f32;
  float branch_eps;
  const float* stream;
  float* stream_out;
  const void* w;                     // [width]
  int w_f32;
  float offset, eps;
  const void* scale;                 // [width] or null
  int scale_f32;
  int width;
};

// Elements i .. i + 3 of row `row` of term b, its splits added in split order, eight loads in flight.
__device__ __forceinline__ float4 term4(const OutNorm& a, int b, int64_t row, int i) {
  const int64_t at = row * a.width + i;
  if (a.splits[b] == 1) return flex4(a.y[b], a.y_f32[b], at);
  const float* p = reinterpret_cast<const float*>(a.y[b]) + at;
  float4 v = *reinterpret_cast<const float4*>(p);
  int s = 1;
  for (; s + 8 <= a.splits[b]; s += 8) {
    float4 u[8];
#pragma unroll
    for (int k = 0; k < 8; ++k) u[k] = *reinterpret_cast<const float4*>(p + (s + k) * a.plane[b]);
#pragma unroll
    for (int k = 0; k < 8; ++k) { v.x += u[k].x; v.y += u[k].y; v.z += u[k].z; v.w += u[k].w; }
  }
  for (; s + 3 <= a.splits[b]; s += 3) {
    float4 u[3];
#pragma unroll
    for (int k = 0; k < 3; ++k) u[k] = *reinterpret_cast<const float4*>(p + (s + k) * a.plane[b]);
#pragma unroll
    for (int k = 0; k < 3; ++k) { v.x += u[k].x; v.y += u[k].y; v.z += u[k].z; v.w += u[k].w; }
  }
  for (; s < a.splits[b]; ++s) {
    const float4 u = *reinterpret_cast<const float4*>(p + s * a.plane[b]);
    v.x += u.x; v.y += u.y; v.z += u.z; v.w += u.w;
  }
  return v;
}
__device__ __forceinline__ float term1(const OutNorm& a, int b, int64_t row, int i) {
  const int64_t at = row * a.width + i;
  float v = load_flex(a.y[b], a.y_f32[b], at);
  for (int s = 1; s < a.splits[b]; ++s) v += reinterpret_cast<const float*>(a.y[b])[s * a.plane[b] + at];
  return v;
}

// V: elements a thread takes at a time (4, or 1 where the width is no multiple of 4).
template <typename TO, int V>
__global__ void __launch_bounds__(1024)
out_norm_stream_kernel(const OutNorm a, TO* __restrict__ out, unsigned* status) {
  extern __shared__ __align__(16) float rows_smem[];          // [terms][width]
  __shared__ float scratch[32];
  pdl_wait();
  pdl_launch_dependents();
  const int width = a.width, first = threadIdx.x * V, step = blockDim.x * V;
  const int64_t r = blockIdx.x, base = r * width;
  // the last pass's operands for this thread's first elements (all of them, when the row is no wider than the block)
  float4 ahead_x = make_float4(0.f, 0.f, 0.f, 0.f), ahead_w = ahead_x, ahead_s = make_float4(1.f, 1.f, 1.f, 1.f);
  if (V == 4 && first < width) {
    ahead_x = *reinterpret_cast<const float4*>(a.stream + base + first);
    ahead_w = flex4(a.w, a.w_f32, first);
    if (a.scale != nullptr) ahead_s = flex4(a.scale, a.scale_f32, first);
  }
  float ss[MAX_TERMS] = {0.f, 0.f};
#pragma unroll
  for (int b = 0; b < MAX_TERMS; ++b) {
    if (b >= a.terms) break;
    float* row = rows_smem + b * width;
    for (int i = first; i < width; i += step) {
      if (V == 4) {
        float4 y;
        if (a.where == nullptr) {
          y = term4(a, b, r, i);
        } else {
          y = make_float4(0.f, 0.f, 0.f, 0.f);
          for (int k = 0; k < a.picks; ++k) {
            int from = a.where[r * a.picks + k];
            if (from < 0 || from >= a.y_rows) { raise_fault(status, VOSTI_FAULT_ROW_RANGE); from = 0; }
            const float c = a.pick_weights != nullptr ? a.pick_weights[r * a.picks + k] : a.share;
            const float4 v = term4(a, b, from, i);
            y.x = fmaf(c, v.x, y.x); y.y = fmaf(c, v.y, y.y); y.z = fmaf(c, v.z, y.z); y.w = fmaf(c, v.w, y.w);
          }
        }
        if (a.bias != nullptr) {
          const float4 v = flex4(a.bias, a.bias_f32, i);
          y.x += v.x; y.y += v.y; y.z += v.z; y.w += v.w;
        }
        *reinterpret_cast<float4*>(row + i) = y;
        ss[b] += dot4(y);
      } else {
        float y = 0.f;
        if (a.where == nullptr) {
          y = term1(a, b, r, i);
        } else {
          for (int k = 0; k < a.picks; ++k) {
            int from = a.where[r * a.picks + k];
            if (from < 0 || from >= a.y_rows) { raise_fault(status, VOSTI_FAULT_ROW_RANGE); from = 0; }
            y = fmaf(a.pick_weights != nullptr ? a.pick_weights[r * a.picks + k] : a.share, term1(a, b, from, i), y);
          }
        }
        if (a.bias != nullptr) y += load_flex(a.bias, a.bias_f32, i);
        row[i] = y;
        ss[b] += y * y;
      }
    }
  }
  float total = block_sum(ss[0], scratch);
  if (a.terms == 2) {
    // the branches' mean; a thread reads what it wrote itself
    const float inv0 = 1.f / sqrtf(total / (float)width + a.branch_eps);
    const float inv1 = 1.f / sqrtf(block_sum(ss[1], scratch) / (float)width + a.branch_eps);
    float sum = 0.f;
    for (int i = first; i < width; i += step) {
      if (V == 4) {
        const float4 w0 = flex4(a.branch_w[0], a.branch_f32, i), w1 = flex4(a.branch_w[1], a.branch_f32, i);
        float4 y = *reinterpret_cast<const float4*>(rows_smem + i);
        const float4 z = *reinterpret_cast<const float4*>(rows_smem + width + i);
        y = make_float4(0.5f * (y.x * inv0 * w0.x + z.x * inv1 * w1.x), 0.5f * (y.y * inv0 * w0.y + z.y * inv1 * w1.y),
                        0.5f * (y.z * inv0 * w0.z + z.z * inv1 * w1.z), 0.5f * (y.w * inv0 * w0.w + z.w * inv1 * w1.w));
        *reinterpret_cast<float4*>(rows_smem + i) = y;
        sum += dot4(y);
      } else {
        const float y = 0.5f * (rows_smem[i] * inv0 * load_flex(a.branch_w[0], a.branch_f32, i) +
                                rows_smem[width + i] * inv1 * load_flex(a.branch_w[1], a.branch_f32, i));
        rows_smem[i] = y;
        sum += y * y;
      }
    }
    total = block_sum(sum, scratch);
  }
  const float inv = 1.f / sqrtf(total / (float)width + a.eps);
  for (int i = first; i < width; i += step) {
    if (V == 4) {
      const float4 y = *reinterpret_cast<const float4*>(rows_smem + i);
      float4 x = ahead_x, w = ahead_w, s = ahead_s;
      if (i != first) {
        x = *reinterpret_cast<const float4*>(a.stream + base + i);
        w = flex4(a.w, a.w_f32, i);
        if (a.scale != nullptr) s = flex4(a.scale, a.scale_f32, i);
      }
      x.x = fmaf(s.x, y.x * inv * (a.offset + w.x), x.x);
      x.y = fmaf(s.y, y.y * inv * (a.offset + w.y), x.y);
      x.z = fmaf(s.z, y.z * inv * (a.offset + w.z), x.z);
      x.w = fmaf(s.w, y.w * inv * (a.offset + w.w), x.w);
      *reinterpret_cast<float4*>(a.stream_out + base + i) = x;
      if (out != nullptr) put4(out + base + i, x);
    } else {
      const float s = a.scale != nullptr ? load_flex(a.scale, a.scale_f32, i) : 1.f;
      const float x = fmaf(s, rows_smem[i] * inv * (a.offset + load_flex(a.w, a.w_f32, i)), a.stream[base + i]);
      a.stream_out[base + i] = x;
      if (out != nullptr) out[base + i] = from_f32<TO>(x);
    }
  }
}

constexpr size_t MAX_ROW_BYTES = 200 * 1024;

template <typename TO, int V>
cudaError_t launch_out_norm(const OutNorm& a, void* out, int rows, int threads, size_t smem, unsigned* status, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(out_norm_stream_kernel<TO, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MAX_ROW_BYTES);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  return vosti_launch(out_norm_stream_kernel<TO, V>, dim3(rows), dim3(threads), smem, stream, a, (TO*)out, status);
}
}  // namespace

// Widest row the boundary kernel takes with one term or with two branches.
VOSTI_API int vosti_out_norm_max_width(int terms) { return (int)(MAX_ROW_BYTES / sizeof(float) / (terms > 1 ? 2 : 1)); }

// See the file's head. ys, y_f32, splits: `terms` entries; a term's splits lie rows * width floats apart (y_rows * width
// with `where`). out: the stream's rounding [rows, width] in bfloat16, or null; stream_out may be the stream.
VOSTI_API int vosti_out_norm_stream(const void* const* ys, const int* y_f32, const int* splits, int terms, const void* bias, int bias_f32,
                                    const int* where, const float* pick_weights, int picks, int y_rows, float share,
                                    const void* const* branch_w, int branch_f32, float branch_eps, const float* stream, float* stream_out,
                                    const void* w, int w_f32, float offset, float eps, const void* scale, int scale_f32, void* out,
                                    int rows, int width, unsigned* status, cudaStream_t stream_id) {
  VOSTI_REQUIRE(rows >= 0 && width > 0 && (terms == 1 || terms == 2), "out_norm_stream: bad sizes rows=%d width=%d terms=%d", rows, width, terms);
  VOSTI_REQUIRE(stream != nullptr && stream_out != nullptr && w != nullptr, "out_norm_stream: a stream and a weight are needed");
  VOSTI_REQUIRE(terms == 1 || (bias == nullptr && where == nullptr && branch_w != nullptr), "out_norm_stream: branches take no bias and no picks");
  VOSTI_REQUIRE(where == nullptr || (picks > 0 && y_rows > 0), "out_norm_stream: bad picks");
  const size_t smem = (size_t)terms * width * sizeof(float);
  VOSTI_REQUIRE(smem <= MAX_ROW_BYTES, "out_norm_stream: a row of %d elements does not fit shared memory", width);
  if (rows == 0) return VOSTI_OK;
  OutNorm a = {};
  for (int b = 0; b < terms; ++b) {
    VOSTI_REQUIRE(ys[b] != nullptr && splits[b] >= 1 && (splits[b] == 1 || y_f32[b]), "out_norm_stream: unsummed splits are float32");
    a.y[b] = ys[b];
    a.y_f32[b] = y_f32[b];
    a.splits[b] = splits[b];
    a.plane[b] = (int64_t)(where != nullptr ? y_rows : rows) * width;
    if (terms == 2) a.branch_w[b] = branch_w[b];
  }
  a.terms = terms;
  a.bias = bias; a.bias_f32 = bias_f32;
  a.where = where; a.pick_weights = pick_weights; a.picks = picks; a.y_rows = y_rows; a.share = share;
  a.branch_f32 = branch_f32; a.branch_eps = branch_eps;
  a.stream = stream; a.stream_out = stream_out;
  a.w = w; a.w_f32 = w_f32; a.offset = offset; a.eps = eps;
  a.scale = scale; a.scale_f32 = scale_f32;
  a.width = width;
  // few rows: a thread a 16-byte word, so that a row's loads are all in flight at once; many: four words, and small
  // blocks, of which an SM holds more (measured at widths of 2,048 and 4,096)
  const int wanted = (width / (rows <= 64 ? 4 : 16) + 31) / 32 * 32, most = rows <= 64 ? 1024 : 256;
  const int threads = wanted > most ? most : wanted < 128 ? 128 : wanted;
  cudaError_t e;
  if (width % 4 == 0) e = launch_out_norm<bf16, 4>(a, out, rows, threads, smem, status, stream_id);
  else e = launch_out_norm<bf16, 1>(a, out, rows, threads, smem, status, stream_id);
  if (e != cudaSuccess) { vosti_set_error("%s", cudaGetErrorString(e)); return (int)e; }
  VOSTI_LAUNCH_CHECK();
}
