// The end of a softmax whose denominator may hold a sink: a key without a value.
#pragma once
#include "common.cuh"

// What a row's weighted values are multiplied by at the end: they and `l` = sum exp(s - m) were formed relative to the
// row's maximum m.  Without a sink 1 / l (0 where nothing is seen).  With one, exp(sink[h]) joins the sum; relative to
// max(m, sink[h]) nothing overflows, however far apart the two are.
__device__ __forceinline__ float softmax_sink_factor(float m, float l, const float* sink, int h) {
  if (sink == nullptr) return l > 0.f ? 1.0f / l : 0.f;
  if (m == -INFINITY) return 0.f;
  const float s = sink[h], top = fmaxf(m, s), f = expf(m - top);
  return f / (l * f + expf(s - top));
}
