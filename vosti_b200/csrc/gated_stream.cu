// A pre-norm sublayer boundary whose sublayers join the float32 stream through gates: one kernel
// closes the sublayer before it and opens the next one,
//
//   x  = stream + mult * sigmoid(z + zb) * y          y: the sublayer's output, z: the gate's product
//   h  = x / sqrt(mean(x^2) + eps) * (offset + w)     w a vector, or one number `gain`
//   u  = h + conv(h)                                  (optional) the next mixer's causal convolution
//
// y may also be spread over several rows: token t's output is share * the sum of the rows where[t, 0 ..
// picks - 1] of y (experts' outputs sorted by expert), picks in order, each with its splits.
//
// x goes back to the stream in float32, h (rounded to the serving type) is what the next gate and
// feed-forward read, u what the next mixer reads. y and z may be a product's unsummed K splits
// (float32 [splits, rows, width]), added in split order. With `rows` the kernel works on the rows
// that list names (the last norm before the output head: only wanted rows are made).
//
// The convolution joins in when every request of the step brings one token (row r is request r):
// then the inputs before the token are all in the request's state slot, tail [taps - 1, width]
// (oldest first), and a thread that owns a channel reads the tail and moves it on. Steps with
// longer portions run scan_conv afterwards; both add the taps oldest first with the same
// multiply-add chain, so a token's u does not depend on which of them ran.
#include "common.cuh"

namespace {

__device__ __forceinline__ float4 load_flex4(const void* p, int is_f32, int64_t i) {
  if (is_f32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
  const uint2 raw = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p) + i);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}
// four values rounded to the output type: stored, and handed back as what was stored
__device__ __forceinline__ float4 store_rounded(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; return v; }
__device__ __forceinline__ float4 store_rounded(bf16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 raw;
  raw.x = *reinterpret_cast<const unsigned*>(&lo);
  raw.y = *reinterpret_cast<const unsigned*>(&hi);
  *reinterpret_cast<uint2*>(p) = raw;
  const float2 a = __bfloat1622float2(lo), b = __bfloat1622float2(hi);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ float logistic(float v) { return 1.f / (1.f + expf(-v)); }

// Sum of the splits of four neighbouring floats, in split order, eight splits' loads in flight together.
__device__ __forceinline__ float4 sum_splits4(const float* p, int splits, int64_t plane) {
  float4 a = *reinterpret_cast<const float4*>(p);
  int s = 1;
  for (; s + 8 <= splits; s += 8) {
    float4 b[8];
#pragma unroll
    for (int u = 0; u < 8; ++u) b[u] = *reinterpret_cast<const float4*>(p + (s + u) * plane);
#pragma unroll
    for (int u = 0; u < 8; ++u) { a.x += b[u].x; a.y += b[u].y; a.z += b[u].z; a.w += b[u].w; }
  }
  for (; s + 2 <= splits; s += 2) {
    const float4 b = *reinterpret_cast<const float4*>(p + s * plane), c = *reinterpret_cast<const float4*>(p + (s + 1) * plane);
    a.x = (a.x + b.x) + c.x; a.y = (a.y + b.y) + c.y; a.z = (a.z + b.z) + c.z; a.w = (a.w + b.w) + c.w;
  }
  for (; s < splits; ++s) {
    const float4 b = *reinterpret_cast<const float4*>(p + s * plane);
    a.x += b.x; a.y += b.y; a.z += b.z; a.w += b.w;
  }
  return a;
}

struct GatedBoundary {
  const float* stream;         // [source rows, width]
  const void* y;               // null: nothing to add
  int y_f32, y_splits;
  const int* where;            // [source rows, picks]: y's rows of every row; null: row by row
  int picks;
  float share;
  int64_t y_plane;             // one split of y
  const float* z;              // null: no gate
  int z_splits;
  const void* zb;              // the gate's bias, or null
  int zb_f32;
  float mult;
  int64_t plane;               // source rows * width: one split of z
  const int* rows;             // the rows to make, or null: all
  int source_rows;
  float* stream_out;           // may be the stream; null: not wanted
  const void* weight;          // [width], or null: `gain` for every element
  int w_f32;
  float offset, gain, eps;
  const float* conv_w;         // float32 [taps, width], oldest tap first; null: no convolution
  int taps;
  float* state;                // [slots, state_stride]; the tail starts at tail_offset
  int64_t state_stride, tail_offset;
  const int* state_slots;
  int num_slots;
  int width, cached;           // cached: the row fits the launch's shared memory
};

template <typename TO>
__global__ void __launch_bounds__(1024)
gated_rms_stream_kernel(const GatedBoundary a, TO* __restrict__ out, TO* __restrict__ conv_out, unsigned* status) {
  extern __shared__ __align__(16) float row_smem[];
  __shared__ float scratch[32];
  pdl_wait();
  pdl_launch_dependents();
  const int width = a.width;
  int source = blockIdx.x;
  if (a.rows != nullptr) {
    source = a.rows[blockIdx.x];
    if (source < 0 || source >= a.source_rows) {
      if (threadIdx.x == 0) raise_fault(status, VOSTI_FAULT_ROW_RANGE);
      source = 0;
    }
  }
  const int64_t from = (int64_t)source * width, to = (int64_t)blockIdx.x * width;
  const bool vec = width % 4 == 0;
  auto sum4 = [&](int i) {
    float4 x = *reinterpret_cast<const float4*>(a.stream + from + i);
    if (a.y == nullptr) return x;
    auto row4 = [&](int64_t base) {
      return a.y_splits > 1 ? sum_splits4(reinterpret_cast<const float*>(a.y) + base + i, a.y_splits, a.y_plane)
                            : load_flex4(a.y, a.y_f32, base + i);
    };
    float4 y;
    if (a.where == nullptr) {
      y = row4(from);
    } else {
      y = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int k = 0; k < a.picks; ++k) {
        const float4 v = row4((int64_t)a.where[(int64_t)source * a.picks + k] * width);
        y.x = fmaf(a.share, v.x, y.x); y.y = fmaf(a.share, v.y, y.y); y.z = fmaf(a.share, v.z, y.z); y.w = fmaf(a.share, v.w, y.w);
      }
    }
    if (a.z != nullptr) {
      float4 g = sum_splits4(a.z + from + i, a.z_splits, a.plane);
      if (a.zb != nullptr) {
        const float4 b = load_flex4(a.zb, a.zb_f32, i);
        g.x += b.x; g.y += b.y; g.z += b.z; g.w += b.w;
      }
      y.x *= logistic(g.x); y.y *= logistic(g.y); y.z *= logistic(g.z); y.w *= logistic(g.w);
    }
    x.x = fmaf(a.mult, y.x, x.x); x.y = fmaf(a.mult, y.y, x.y); x.z = fmaf(a.mult, y.z, x.z); x.w = fmaf(a.mult, y.w, x.w);
    return x;
  };
  auto sum1 = [&](int i) {
    float x = a.stream[from + i];
    if (a.y == nullptr) return x;
    auto row1 = [&](int64_t base) {
      float v = load_flex(a.y, a.y_f32, base + i);
      for (int s = 1; s < a.y_splits; ++s) v += reinterpret_cast<const float*>(a.y)[s * a.y_plane + base + i];
      return v;
    };
    float y = 0.f;
    if (a.where == nullptr) y = row1(from);
    else
      for (int k = 0; k < a.picks; ++k) y = fmaf(a.share, row1((int64_t)a.where[(int64_t)source * a.picks + k] * width), y);
    if (a.z != nullptr) {
      float g = a.z[from + i];
      for (int s = 1; s < a.z_splits; ++s) g += a.z[s * a.plane + from + i];
      if (a.zb != nullptr) g += load_flex(a.zb, a.zb_f32, i);
      y *= logistic(g);
    }
    return fmaf(a.mult, y, x);
  };
  // pass 1: the sum (kept in shared memory where it fits, else read back from the stream it was stored to,
  // by the thread that wrote it, or formed again) and its squares
  float ss = 0.f;
  if (vec) {
    for (int i = threadIdx.x * 4; i < width; i += blockDim.x * 4) {
      const float4 x = sum4(i);
      if (a.cached) *reinterpret_cast<float4*>(row_smem + i) = x;
      if (a.stream_out != nullptr) *reinterpret_cast<float4*>(a.stream_out + to + i) = x;
      ss += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
    }
  } else {
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
      const float x = sum1(i);
      if (a.cached) row_smem[i] = x;
      if (a.stream_out != nullptr) a.stream_out[to + i] = x;
      ss += x * x;
    }
  }
  if (out == nullptr) return;
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + a.eps);
  float* tail = nullptr;
  if (conv_out != nullptr && a.taps > 1) {
    const int slot = a.state_slots[blockIdx.x];
    if (slot >= 0 && slot < a.num_slots) tail = a.state + (int64_t)slot * a.state_stride + a.tail_offset;
    else if (threadIdx.x == 0) raise_fault(status, VOSTI_FAULT_SLOT_RANGE);
  }
  // pass 2: the norm, and the convolution of the row with its request's tail
  if (vec) {
    for (int i = threadIdx.x * 4; i < width; i += blockDim.x * 4) {
      float4 x = a.cached ? *reinterpret_cast<const float4*>(row_smem + i)
                          : a.stream_out != nullptr ? *reinterpret_cast<const float4*>(a.stream_out + to + i) : sum4(i);
      float4 w = make_float4(a.gain, a.gain, a.gain, a.gain);
      if (a.weight != nullptr) {
        const float4 v = load_flex4(a.weight, a.w_f32, i);
        w = make_float4(a.offset + v.x, a.offset + v.y, a.offset + v.z, a.offset + v.w);
      }
      const float4 h = store_rounded(out + to + i, make_float4(x.x * inv * w.x, x.y * inv * w.y, x.z * inv * w.z, x.w * inv * w.w));
      if (conv_out == nullptr) continue;
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int j = 0; j < a.taps; ++j) {
        const float4 k = *reinterpret_cast<const float4*>(a.conv_w + (int64_t)j * width + i);
        float4 v = h;
        if (j < a.taps - 1) {
          v = make_float4(0.f, 0.f, 0.f, 0.f);
          if (tail != nullptr) {
            v = *reinterpret_cast<const float4*>(tail + (int64_t)j * width + i);
            if (j > 0) *reinterpret_cast<float4*>(tail + (int64_t)(j - 1) * width + i) = v;
          }
        }
        acc.x = fmaf(k.x, v.x, acc.x); acc.y = fmaf(k.y, v.y, acc.y); acc.z = fmaf(k.z, v.z, acc.z); acc.w = fmaf(k.w, v.w, acc.w);
      }
      if (tail != nullptr) *reinterpret_cast<float4*>(tail + (int64_t)(a.taps - 2) * width + i) = h;
      store_rounded(conv_out + to + i, make_float4(h.x + acc.x, h.y + acc.y, h.z + acc.z, h.w + acc.w));
    }
    return;
  }
  for (int i = threadIdx.x; i < width; i += blockDim.x) {
    const float x = a.cached ? row_smem[i] : a.stream_out != nullptr ? a.stream_out[to + i] : sum1(i);
    const TO rounded = from_f32<TO>(x * inv * (a.weight != nullptr ? a.offset + load_flex(a.weight, a.w_f32, i) : a.gain));
    out[to + i] = rounded;
    if (conv_out == nullptr) continue;
    const float h = to_f32(rounded);
    float acc = 0.f;
    for (int j = 0; j < a.taps; ++j) {
      float v = h;
      if (j < a.taps - 1) {
        v = tail != nullptr ? tail[(int64_t)j * width + i] : 0.f;
        if (tail != nullptr && j > 0) tail[(int64_t)(j - 1) * width + i] = v;
      }
      acc = fmaf(a.conv_w[(int64_t)j * width + i], v, acc);
    }
    if (tail != nullptr) tail[(int64_t)(a.taps - 2) * width + i] = h;
    conv_out[to + i] = from_f32<TO>(h + acc);
  }
}

}  // namespace

// stream float32 [source_rows, width]; y (or null) float32 or bfloat16 [source_rows, width], or with y_splits
// > 1 float32 [y_splits, source_rows, width]; with `where` (int32 [source_rows, picks], every entry a row of y)
// y has y_rows rows and a row's output is share * the sum of those; z (or null) float32 likewise; zb [width] (or null); `rows`
// int32 [count] (or null: count = source_rows); stream_out float32 [count, width] (or null; not with
// `rows`); out, conv_out [count, width] in the output type (conv_out null: no convolution; it needs
// count = the step's requests, one row each). Without `weight` every element is multiplied by `gain`.
VOSTI_API int vosti_gated_rms_stream(const float* stream, const void* y, int y_f32, int y_splits, const int* where, int picks,
                                     float share, int y_rows, const float* z, int z_splits,
                                     const void* zb, int zb_f32, float mult, const int* rows, int count, int source_rows,
                                     float* stream_out, const void* weight, int w_f32, float offset, float gain, float eps,
                                     const float* conv_w, int taps, float* state, int64_t state_stride, int64_t tail_offset,
                                     const int* state_slots, int num_slots, void* out, void* conv_out, int out_f32, int width,
                                     unsigned* status, cudaStream_t stream_id) {
  VOSTI_REQUIRE(count >= 0 && source_rows >= 0 && width > 0, "gated_rms_stream: bad sizes rows=%d width=%d", count, width);
  VOSTI_REQUIRE(stream != nullptr && (out != nullptr || stream_out != nullptr), "gated_rms_stream: a stream and somewhere to write are needed");
  VOSTI_REQUIRE(y_splits >= 1 && (y_splits == 1 || y_f32) && z_splits >= 1, "gated_rms_stream: unsummed splits are float32");
  VOSTI_REQUIRE(where == nullptr || (y != nullptr && picks >= 1 && y_rows >= 1), "gated_rms_stream: picked rows need their number");
  VOSTI_REQUIRE(z == nullptr || y != nullptr, "gated_rms_stream: a gate without something to gate");
  VOSTI_REQUIRE(rows == nullptr ? count == source_rows : stream_out == nullptr, "gated_rms_stream: the stream is stored for all rows or for none");
  VOSTI_REQUIRE(conv_out == nullptr || (out != nullptr && conv_w != nullptr && taps >= 1 &&
                                        (taps == 1 || (state != nullptr && state_slots != nullptr))),
                "gated_rms_stream: the convolution needs its taps and, for more than one, the state slots");
  if (count == 0) return VOSTI_OK;
  GatedBoundary a = {};
  a.stream = stream; a.y = y; a.y_f32 = y_f32; a.y_splits = y_splits; a.where = where; a.picks = picks; a.share = share;
  a.y_plane = (int64_t)(where != nullptr ? y_rows : source_rows) * width; a.z = z; a.z_splits = z_splits; a.zb = zb; a.zb_f32 = zb_f32;
  a.mult = mult; a.plane = (int64_t)source_rows * width; a.rows = rows; a.source_rows = source_rows; a.stream_out = stream_out;
  a.weight = weight; a.w_f32 = w_f32; a.offset = offset; a.gain = gain; a.eps = eps; a.conv_w = conv_w; a.taps = taps; a.state = state;
  a.state_stride = state_stride; a.tail_offset = tail_offset; a.state_slots = state_slots; a.num_slots = num_slots; a.width = width;
  a.cached = width <= 12288;                                // 48 KB of shared memory hold the row
  const size_t smem = a.cached ? (size_t)width * sizeof(float) : 0;
  // few rows: a thread a 16-byte word, so that a row's loads are all in flight at once
  int threads = 256;
  if (count <= 64 && width % 4 == 0) threads = width / 4 >= 1024 ? 1024 : (width / 4 + 31) / 32 * 32 > 256 ? (width / 4 + 31) / 32 * 32 : 256;
  if (out_f32)
    vosti_launch(gated_rms_stream_kernel<float>, dim3(count), dim3(threads), smem, stream_id, a, (float*)out, (float*)conv_out, status);
  else
    vosti_launch(gated_rms_stream_kernel<bf16>, dim3(count), dim3(threads), smem, stream_id, a, (bf16*)out, (bf16*)conv_out, status);
  VOSTI_LAUNCH_CHECK();
}
