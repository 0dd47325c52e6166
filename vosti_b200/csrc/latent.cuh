// What the latent attention's CUDA-core and tensor-core files share.
#pragma once
#include "common.cuh"

// 1 / denominator of a softmax whose sum is l at the reference maximum m (base-2 units), after one more
// logit `sink_l2` (-inf: none) has joined it; relative to m, so that sums taken at m can be multiplied by it.
__device__ __forceinline__ float sink_inverse(float m, float l, float sink_l2) {
  if (sink_l2 == -INFINITY) return l > 0.f ? 1.f / l : 0.f;
  if (m == -INFINITY) return 0.f;
  const float top = fmaxf(m, sink_l2);
  const float down = exp2f(m - top);
  return down / (l * down + exp2f(sink_l2 - top));
}

// The output gate of a per-head product: one factor a head, or sigmoid of one number an element, or none.
struct HeadGate {
  const float* per_head;       // [tokens, heads], or null
  const void* per_element;     // [tokens, heads * out] before the sigmoid, rows `row` elements apart, or null
  int element_f32;
  int64_t row;
  int pairs;                   // two neighbouring elements of per_element (bfloat16) are one aligned word
  __device__ __forceinline__ float2 at_pair(int t, int h, int o, int heads, int out) const {
    if (per_element == nullptr || !pairs) return make_float2(at(t, h, o, heads, out), at(t, h, o + 1, heads, out));
    const __nv_bfloat162 raw = *reinterpret_cast<const __nv_bfloat162*>(reinterpret_cast<const bf16*>(per_element) +
                                                                        (int64_t)t * row + (int64_t)h * out + o);
    const float2 z = __bfloat1622float2(raw);
    return make_float2(__fdividef(1.f, 1.f + __expf(-z.x)), __fdividef(1.f, 1.f + __expf(-z.y)));
  }
  __device__ __forceinline__ float at(int t, int h, int o, int heads, int out) const {
    if (per_head != nullptr) return per_head[(int64_t)t * heads + h];
    if (per_element != nullptr) return 1.f / (1.f + expf(-load_flex(per_element, element_f32, (int64_t)t * row + (int64_t)h * out + o)));
    return 1.f;
  }
};
