// What a softmax attention may have besides a scale and a window: a cap on the scores, a sink per head, first positions
// that stay visible, values of another size than the keys, and longer output rows. The attention kernels take it as an
// argument that their plain instantiations ignore (OPTIONS = false) and that others read (OPTIONS = true).
#pragma once
#include "wide_kv.cuh"

struct ScoreOptions {
  const float* sinks;  // [heads] or null
  float cap;           // 0: scores as they are
  int keep;            // the sequence's first `keep` positions are seen at any distance
  int value_dim;
  int out_stride;      // elements of an output row
};

constexpr float SCORE_LOG2E = 1.4426950408889634f;

// A score in units of log2 e, s = q . k: scale s, or cap tanh(scale s / cap). For |scale s / cap| <= SMALL the tanh is
// x (1 + x^2 P(x^2)) with P fitted to tanh for the smallest largest relative error on that interval (1.2e-7, a float32's
// rounding): multiply-adds only, where the general form needs an exponential and a reciprocal per score.
struct ScoreCap {
  float in, scale_log2, at, twice, small_up_to;
  static constexpr float SMALL = 0.625f;
  __device__ __forceinline__ ScoreCap(float scale, float cap) {
    scale_log2 = scale * SCORE_LOG2E;
    in = cap > 0.f ? scale / cap : 0.f;
    at = cap * SCORE_LOG2E;
    twice = -2.0f * cap * SCORE_LOG2E;
    small_up_to = cap > 0.f ? SMALL * cap / scale : INFINITY;
  }
  __device__ __forceinline__ float small(float s) const {
    float x = s * in, t = x * x;
    float p = fmaf(t, fmaf(t, fmaf(t, 0.01519537f, -0.0519479f), 0.13308175f), -0.33332341f);
    float y = s * scale_log2;
    return fmaf(y * t, p, y);
  }
  __device__ __forceinline__ float any(float s) const {  // cap - 2 cap / (e^(2x) + 1)
    if (in == 0.f) return s * scale_log2;
    float e = fast_exp2(s * in * (2.0f * SCORE_LOG2E)), r;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(e + 1.0f));
    return fmaf(twice, r, at);
  }
};

// The last step of a softmax's sum under a sink: with the running maximum m (log2 units) and sum l, the factor that the
// running weighted sum of values is multiplied by.
__device__ __forceinline__ float sink_factor(float m, float l, const float* sinks, int head) {
  if (sinks == nullptr) return 1.0f / l;
  float sink = sinks[head] * SCORE_LOG2E, top = fmaxf(m, sink);
  float f = fast_exp2(m - top);
  return f / fmaf(l, f, fast_exp2(sink - top));
}
