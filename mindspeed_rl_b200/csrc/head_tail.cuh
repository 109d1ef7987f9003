// What the epilogues of soft-max attention may add to a head's result: exp(sink[h]) in the soft-max sum, and
// sigmoid(gate[t, h]) as a factor.  And the soft cap of scores.
#pragma once
#include "dtype_utils.cuh"

namespace msrl {

template <typename T>
struct HeadTail {
  const T* gate;             // [tokens, gate_ld] logits, or null
  long long gate_ld;
  const float* sink;         // [heads], or null

  __device__ __forceinline__ float gated(long long t, int h) const {
    return gate != nullptr ? sigmoid_f(ldf(gate + t * gate_ld + h)) : 1.f;
  }
  // Factor on sum_j exp(s_j - m) v_j whose weights add up to l; nothing visible: 0.
  __device__ __forceinline__ float scale(long long t, int h, float m, float l) const {
    if (!(l > 0.f)) return 0.f;
    if (sink == nullptr) return gated(t, h) / l;
    const float d = sink[h] - m;                           // far above m: the whole quotient scaled by exp(-d)
    return d > 60.f ? gated(t, h) * expf(-d) / (l * expf(-d) + 1.f) : gated(t, h) / (l + expf(d));
  }
  // the same with m in the exp2 domain
  __device__ __forceinline__ float scale2(long long t, int h, float m, float l) const {
    return scale(t, h, m * 0.6931471805599453f, l);
  }
};

// cap * tanh(x / cap)
__device__ __forceinline__ float softcapped(float x, float cap) { return cap * tanhf(x / cap); }

// The same for tensor-core kernels, in the exp2 domain (v = x log2(e)), with tanh(y) = 1 - 2 / (exp(2 y) + 1): two
// approximate function units per score, an error of a few ulp of the cap.
struct SoftCap2 {
  float rate, cap2;          // 2 / cap, cap * log2(e)
  __device__ __forceinline__ explicit SoftCap2(float cap) : rate(2.f / cap), cap2(cap * 1.4426950408889634f) {}
  __device__ __forceinline__ float operator()(float v) const {
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(v * rate));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(e + 1.f));
    return fmaf(-2.f * cap2, r, cap2);
  }
};

}  // namespace msrl
