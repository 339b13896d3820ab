// What a softmax attention may have besides a scale and a window: a cap on the scores, a sink per head, first positions
// that stay visible, chunks, values of another size than the keys, a factor of
// the output, and longer output rows. The attention kernels take it as an
// argument that their plain instantiations ignore (OPTIONS = false) and that others read (OPTIONS = true).
#pragma once
#include "wide_kv.cuh"

struct ScoreOptions {
  const float* sinks;  // [heads] or null
  float cap;           // 0: scores as they are
  int keep;            // the sequence's first `keep` positions are seen at any distance
  int value_dim;
  int out_stride;      // elements of an output row
  int chunk;           // 0, or: a token sees the positions of its own chunk of this many only
  float out_scale;     // what the outputs are multiplied by before they are rounded
};

constexpr float SCORE_LOG2E = 1.4426950408889634f;

// A score in units of log2 e, s = q . k: scale s, or cap tanh(scale s / cap). For |scale s / cap| <= SMALL the tanh is
// x (1 + x^2 P(x^2)) with P fitted to tanh for the smallest largest relative error on that interval (1.2e-7, a float32's
// rounding): multiply-adds only, two scores an instruction, where the general form needs an exponential and a reciprocal
// per score. Without a cap the same form has P = 0.
struct ScoreCap {
  float in, c[5], at, twice, small_up_to;
  static constexpr float SMALL = 0.625f;
  __device__ __forceinline__ ScoreCap(float scale, float cap) {
    const bool capped = cap > 0.f;
    in = capped ? scale / cap : 1.0f;
    at = cap * SCORE_LOG2E;
    twice = -2.0f * at;
    small_up_to = capped ? SMALL * cap / scale : INFINITY;
    c[0] = capped ? at : scale * SCORE_LOG2E;
    c[1] = -0.33332341f * at;
    c[2] = 0.13308175f * at;
    c[3] = -0.0519479f * at;
    c[4] = 0.01519537f * at;
  }
  // two scores that are small, and `add` added to both
  __device__ __forceinline__ float2 small2(float2 s, float2 add) const {
    auto both = [](float v) { return make_float2(v, v); };
    float2 x = __fmul2_rn(s, both(in)), t = __fmul2_rn(x, x);
    float2 r = __ffma2_rn(t, __ffma2_rn(t, __ffma2_rn(t, __ffma2_rn(t, both(c[4]), both(c[3])), both(c[2])), both(c[1])),
                          both(c[0]));
    return __ffma2_rn(x, r, add);
  }
  __device__ __forceinline__ float any(float s) const {
    if (fabsf(s) <= small_up_to) {
      float x = s * in, t = x * x;
      return x * fmaf(t, fmaf(t, fmaf(t, fmaf(t, c[4], c[3]), c[2]), c[1]), c[0]);
    }
    return large(s);
  }
  __device__ __forceinline__ float large(float s) const {  // cap - 2 cap / (e^(2x) + 1); at any size of x
    float e = fast_exp2(s * in * (2.0f * SCORE_LOG2E)), r;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(e + 1.0f));
    return fmaf(twice, r, at);
  }
};

// The last step of a softmax's sum under a sink: with the running maximum m (log2 units) and sum l, the factor that the
// running weighted sum of values is multiplied by (the output's own factor in it).
__device__ __forceinline__ float sink_factor(float m, float l, const ScoreOptions& options, int head) {
  if (options.sinks == nullptr) return options.out_scale / l;
  float sink = options.sinks[head] * SCORE_LOG2E, top = fmaxf(m, sink);
  float f = fast_exp2(m - top);
  return f * options.out_scale / fmaf(l, f, fast_exp2(sink - top));
}
