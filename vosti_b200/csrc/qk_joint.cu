// After a q | k | further projection whose queries and keys are normed over their whole projection
// (all heads at once) and whose values are the keys themselves:
//
//   q' = q + bq,  k' = k + bk
//   queries  <- q' / sqrt(mean(q'^2) + eps) * wq        (the mean over all heads' elements)
//   key slot <- k' / sqrt(mean(k'^2) + eps) * wk        value slot <- k'
//
// everything in float32, rounded once. The projection is float32 or the serving type, or float32
// unsummed K splits, added in split order; columns after k (a gate per head) are summed into a
// tensor of their own. One block per token and side: blockIdx.y 0 makes the queries, 1 keys, values
// and the further columns. A side's row lies in shared memory between the two passes.
#include "common.cuh"

namespace {

struct QkJoint {
  const void* proj;          // [tokens, stride]; splits > 1: float32 [splits, tokens, stride], `plane` apart
  int proj_f32, splits;
  int64_t stride, plane;
  const float* bias;         // [wq + wk] or null
  const void* q_norm;        // [wq]
  const void* k_norm;        // [wk]
  int norm_f32;
  float eps;
  const int* slot_mapping;
  int64_t num_slots;
  int page_size, wq, wk, dk, nkv, extra_width;
  float* extra;              // [tokens, extra_width] or null
};

__device__ __forceinline__ float4 quad(const void* p, int is_f32, int64_t i) {
  if (is_f32) return *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(p) + i);
  const uint2 raw = *reinterpret_cast<const uint2*>(reinterpret_cast<const bf16*>(p) + i);
  const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
  const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
  return make_float4(lo.x, lo.y, hi.x, hi.y);
}
__device__ __forceinline__ void put_quad(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put_quad(bf16* p, float4 v) {
  const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
  uint2 raw;
  raw.x = *reinterpret_cast<const unsigned*>(&lo);
  raw.y = *reinterpret_cast<const unsigned*>(&hi);
  *reinterpret_cast<uint2*>(p) = raw;
}

template <typename T, int V>
__global__ void __launch_bounds__(1024)
qk_joint_kernel(const QkJoint a, T* __restrict__ q_out, T* __restrict__ k_cache, T* __restrict__ v_cache, unsigned* status) {
  extern __shared__ __align__(16) float side_row[];
  __shared__ float scratch[32];
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x;
  const bool keys = blockIdx.y == 1;
  const int64_t row = (int64_t)t * a.stride;
  auto sum1 = [&](int64_t col) {
    float x = load_flex(a.proj, a.proj_f32, row + col);
    for (int s = 1; s < a.splits; ++s) x += reinterpret_cast<const float*>(a.proj)[s * a.plane + row + col];
    return x;
  };
  if (keys && a.extra != nullptr)
    for (int i = threadIdx.x; i < a.extra_width; i += blockDim.x) a.extra[(int64_t)t * a.extra_width + i] = sum1(a.wq + a.wk + i);
  bool store = true;
  int64_t page = 0, offset = 0;
  if (keys) {
    if (k_cache == nullptr) return;
    const int64_t slot = a.slot_mapping[t];
    if (slot < 0 || slot >= a.num_slots) {
      if (threadIdx.x == 0) raise_fault(status, VOSTI_FAULT_SLOT_RANGE);
      store = false;
    } else {
      page = slot / a.page_size;
      offset = slot % a.page_size;
    }
  }
  const int width = keys ? a.wk : a.wq, col0 = keys ? a.wq : 0;
  const void* norm = keys ? a.k_norm : a.q_norm;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {
    if (V == 4) {
      float4 x = quad(a.proj, a.proj_f32, row + col0 + i);
      for (int s = 1; s < a.splits; ++s) {
        const float4 y = *reinterpret_cast<const float4*>(reinterpret_cast<const float*>(a.proj) + s * a.plane + row + col0 + i);
        x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
      }
      if (a.bias != nullptr) {
        const float4 y = *reinterpret_cast<const float4*>(a.bias + col0 + i);
        x.x += y.x; x.y += y.y; x.z += y.z; x.w += y.w;
      }
      *reinterpret_cast<float4*>(side_row + i) = x;
      ss += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
    } else {
      float x = sum1(col0 + i);
      if (a.bias != nullptr) x += a.bias[col0 + i];
      side_row[i] = x;
      ss += x * x;
    }
  }
  const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + a.eps);
  if (!store) return;
  for (int i = threadIdx.x * V; i < width; i += blockDim.x * V) {      // (a thread reads what it wrote itself)
    T* dst = q_out + (int64_t)t * a.wq + i;
    T* val = nullptr;
    if (keys) {
      const int g = i / a.dk, c = i - g * a.dk;
      const int64_t at = ((page * a.nkv + g) * a.page_size + offset) * a.dk + c;
      dst = k_cache + at;
      val = v_cache + at;
    }
    if (V == 4) {
      const float4 x = *reinterpret_cast<const float4*>(side_row + i), w = quad(norm, a.norm_f32, i);
      put_quad(dst, make_float4(x.x * inv * w.x, x.y * inv * w.y, x.z * inv * w.z, x.w * inv * w.w));
      if (keys) put_quad(val, x);
    } else {
      const float x = side_row[i];
      *dst = from_f32<T>(x * inv * load_flex(norm, a.norm_f32, i));
      if (keys) *val = from_f32<T>(x);
    }
  }
}

constexpr size_t MAX_SIDE_BYTES = 200 * 1024;

template <typename T, int V>
cudaError_t launch_qk_joint(const QkJoint& a, void* q_out, void* k_cache, void* v_cache, int tokens, int threads, size_t smem,
                            unsigned* status, cudaStream_t stream) {
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(qk_joint_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MAX_SIDE_BYTES);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  return vosti_launch(qk_joint_kernel<T, V>, dim3(tokens, 2), dim3(threads), smem, stream, a, (T*)q_out, (T*)k_cache, (T*)v_cache, status);
}
}  // namespace

// proj [tokens, >= (nq + nkv) * dk + extra_width], rows `stride` elements apart; q_out [tokens, nq * dk]; caches
// [pages, nkv, page_size, dk], or null (queries and further columns only); extra float32 [tokens, extra_width] or null.
VOSTI_API int vosti_qk_joint(const void* proj, int proj_f32, int splits, int64_t stride, const float* bias, const void* q_norm,
                             const void* k_norm, int norm_f32, float eps, void* q_out, void* k_cache, void* v_cache,
                             const int* slot_mapping, int64_t num_slots, int page_size, int tokens, int nq, int nkv, int dk,
                             float* extra, int extra_width, int is_f32, unsigned* status, cudaStream_t stream) {
  VOSTI_REQUIRE(tokens >= 0 && nq > 0 && nkv > 0 && dk > 0, "qk_joint: bad sizes");
  VOSTI_REQUIRE(splits >= 1 && (splits == 1 || proj_f32), "qk_joint: unsummed splits are float32");
  VOSTI_REQUIRE(stride >= (int64_t)(nq + nkv) * dk + (extra != nullptr ? extra_width : 0), "qk_joint: the projection's rows are too narrow");
  VOSTI_REQUIRE(k_cache == nullptr || (v_cache != nullptr && slot_mapping != nullptr && page_size > 0), "qk_joint: a cache needs slots");
  VOSTI_REQUIRE(q_norm != nullptr && k_norm != nullptr, "qk_joint: the norms' weights are missing");
  const int wide = (nq > nkv ? nq : nkv) * dk;
  const size_t smem = (size_t)wide * sizeof(float);
  VOSTI_REQUIRE(smem <= MAX_SIDE_BYTES, "qk_joint: a projection of %d columns does not fit shared memory", wide);
  if (tokens == 0) return VOSTI_OK;
  QkJoint a = {};
  a.proj = proj; a.proj_f32 = proj_f32; a.splits = splits; a.stride = stride; a.plane = (int64_t)tokens * stride;
  a.bias = bias; a.q_norm = q_norm; a.k_norm = k_norm; a.norm_f32 = norm_f32; a.eps = eps;
  a.slot_mapping = slot_mapping; a.num_slots = num_slots; a.page_size = page_size;
  a.wq = nq * dk; a.wk = nkv * dk; a.dk = dk; a.nkv = nkv; a.extra = extra; a.extra_width = extra != nullptr ? extra_width : 0;
  const bool words = dk % 4 == 0 && stride % 4 == 0 && (reinterpret_cast<uintptr_t>(proj) & 15) == 0 &&
                     (bias == nullptr || (reinterpret_cast<uintptr_t>(bias) & 15) == 0) && (reinterpret_cast<uintptr_t>(q_norm) & 15) == 0 &&
                     (reinterpret_cast<uintptr_t>(k_norm) & 15) == 0;
  // few tokens: a thread a 16-byte word; many: small blocks, of which an SM holds more
  const int wanted = (wide / 4 + 31) / 32 * 32, most = tokens <= 64 ? 1024 : 128;
  const int threads = wanted > most ? most : wanted < 128 ? 128 : wanted;
  cudaError_t e;
#define VOSTI_JOINT_ARGS a, q_out, k_cache, v_cache, tokens, threads, smem, status, stream
  if (is_f32) e = words ? launch_qk_joint<float, 4>(VOSTI_JOINT_ARGS) : launch_qk_joint<float, 1>(VOSTI_JOINT_ARGS);
  else e = words ? launch_qk_joint<bf16, 4>(VOSTI_JOINT_ARGS) : launch_qk_joint<bf16, 1>(VOSTI_JOINT_ARGS);
#undef VOSTI_JOINT_ARGS
  if (e != cudaSuccess) { vosti_set_error("%s", cudaGetErrorString(e)); return (int)e; }
  VOSTI_LAUNCH_CHECK();
}
