// Element-wise recurrence whose gate and candidate do not depend on the state, in fp32:
//
//   z = sigmoid(z_proj + z_bias),  u = x_proj + x_bias,  c = u + 1/2 for u >= 0, else sigmoid(u)
//   S <- (1 - z) S + z c;          y = S * silu(g_proj) * scale
//
// over state slots [slots, width]; S is zero before a sequence's first token.  Prompts are cut into segments of SEG tokens:
// the factor and the sum that every segment leaves (all segments in parallel), a pass over the segments, and the outputs of
// every segment from the state before it.  One thread owns V channels.
#include "dtype_utils.cuh"

namespace msrl {
namespace gru {

constexpr int SEG = 64;                  // tokens of a segment
constexpr int AHEAD = 8, SEGS_AHEAD = 32;     // tokens, segments whose rows are loaded together

template <typename T>
struct Args {
  const T *z, *x, *g;                    // sections of rows [tokens, ld]
  long long ld;
  const float *z_bias, *x_bias;          // [width]
  float* state;                          // [slots, width]
  const int* cu;                         // null: one token per sequence, `start` holds positions
  const int* start;
  const long long* slots;
  float scale;
  T* y;                                  // [tokens, y_ld]; columns [width, padded) become zero
  long long y_ld;
  int width, padded;
  float *keep, *sum;                     // [segments, width]: factor and sum, then (in sum) the state before the segment
};

__device__ __forceinline__ long long seg_id(int t0, int b, int j) { return t0 / SEG + b + j; }

// bf16 rows do not need the last bits of the exponential and the division
template <typename T>
__device__ __forceinline__ void step_of(float zp, float xp, float zb, float xb, float& keep, float& add) {
  zp += zb;
  const float u = xp + xb, a = fabsf(zp);
  float e, inv;
  if constexpr (sizeof(T) == 2) {
    e = __expf(-a);
    inv = __fdividef(1.f, 1.f + e);
  } else {
    e = expf(-a);
    inv = 1.f / (1.f + e);
  }
  const float small = e * inv, z = zp >= 0.f ? inv : small;
  keep = zp >= 0.f ? small : 1.f - small;
  add = z * (u >= 0.f ? u + 0.5f : sigmoid_t<T>(u));
}

// V entries as they are stored
template <typename T, int V>
struct alignas(V * sizeof(T)) Packed {
  T v[V];
};
// OUT: outputs from the state before the segment; otherwise the segment's factor and sum.  WHOLE: one segment holds the
// sequence, its state comes from the slot and goes back.  grid (channels / (128 V), segments, B)
template <typename T, int V, bool OUT, bool WHOLE>
__global__ void __launch_bounds__(128) scan_kernel(const Args<T> p) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * V, j = blockIdx.y, b = blockIdx.z;
  const int s0 = p.cu != nullptr ? p.cu[b] : b, end = p.cu != nullptr ? p.cu[b + 1] : b + 1, t0 = s0 + j * SEG;
  const int len = min(end - t0, SEG);
  if (len <= 0 || c >= p.padded) return;
  if (c >= p.width) {                    // padding of the output row
    if (OUT) {
      const float zero[4] = {0.f, 0.f, 0.f, 0.f};
      for (int i = 0; i < len; ++i) stv<V>(p.y + (long long)(t0 + i) * p.y_ld + c, zero);
    }
    return;
  }
  const long long slot = p.slots[b], at = WHOLE ? 0 : seg_id(s0, b, j) * p.width + c;
  float S[4] = {0.f, 0.f, 0.f, 0.f}, A[4] = {1.f, 1.f, 1.f, 1.f}, zb[4], xb[4];
  ldv<V>(p.z_bias + c, zb);
  ldv<V>(p.x_bias + c, xb);
  if (OUT) {
    if (!WHOLE) ldv<V>(p.sum + at, S);
    else if (p.start[b] > 0 && slot >= 0) ldv<V>(p.state + slot * p.width + c, S);
  }
  using R = Packed<T, V>;
  struct Rows {
    R z[AHEAD], x[AHEAD], g[AHEAD];
  } now, next;
  const T *zp = p.z + (long long)t0 * p.ld + c, *xp = p.x + (long long)t0 * p.ld + c, *gp = p.g + (long long)t0 * p.ld + c;
  auto fetch = [&](Rows& rows, int i0) {
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (i0 + i < len) {
        const long long at = (i0 + i) * p.ld;
        rows.z[i] = *reinterpret_cast<const R*>(zp + at);
        rows.x[i] = *reinterpret_cast<const R*>(xp + at);
        if (OUT) rows.g[i] = *reinterpret_cast<const R*>(gp + at);
      }
    }
  };
  fetch(now, 0);
  for (int i0 = 0; i0 < len; i0 += AHEAD) {
    fetch(next, i0 + AHEAD);
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (i0 + i < len) {
        float z[4], x[4], g[4], y[4];
        ldv<V>(reinterpret_cast<const T*>(&now.z[i]), z);
        ldv<V>(reinterpret_cast<const T*>(&now.x[i]), x);
        if (OUT) ldv<V>(reinterpret_cast<const T*>(&now.g[i]), g);
#pragma unroll
        for (int e = 0; e < V; ++e) {
          float keep, add;
          step_of<T>(z[e], x[e], zb[e], xb[e], keep, add);
          S[e] = keep * S[e] + add;
          if (OUT) y[e] = S[e] * g[e] * sigmoid_t<T>(g[e]) * p.scale;
          else A[e] *= keep;
        }
        if (OUT) stv<V>(p.y + (long long)(t0 + i0 + i) * p.y_ld + c, y);
      }
    }
    now = next;
  }
  if (!OUT) {
    stv<V>(p.keep + at, A);
    stv<V>(p.sum + at, S);
  } else if (WHOLE && slot >= 0) {
    stv<V>(p.state + slot * p.width + c, S);
  }
}

// grid (channels / 128, B): segment after segment
template <typename T>
__global__ void __launch_bounds__(128) carry_kernel(const Args<T> p) {
  const int c = blockIdx.x * 128 + threadIdx.x, b = blockIdx.y;
  const int t0 = p.cu[b], len = p.cu[b + 1] - t0, n = (len + SEG - 1) / SEG;
  if (len <= 0 || c >= p.width) return;
  const long long slot = p.slots[b], at = seg_id(t0, b, 0) * p.width + c;
  float s = p.start[b] > 0 && slot >= 0 ? p.state[slot * p.width + c] : 0.f;
  for (int j0 = 0; j0 < n; j0 += SEGS_AHEAD) {
    float keep[SEGS_AHEAD], sum[SEGS_AHEAD];
#pragma unroll
    for (int i = 0; i < SEGS_AHEAD; ++i) {
      if (j0 + i < n) {
        keep[i] = p.keep[at + (long long)(j0 + i) * p.width];
        sum[i] = p.sum[at + (long long)(j0 + i) * p.width];
      }
    }
#pragma unroll
    for (int i = 0; i < SEGS_AHEAD; ++i) {
      if (j0 + i < n) {
        p.sum[at + (long long)(j0 + i) * p.width] = s;
        s = keep[i] * s + sum[i];
      }
    }
  }
  if (slot >= 0) p.state[slot * p.width + c] = s;
}

template <typename T, int V>
int launch(const Args<T>& p, int most, int batch, cudaStream_t st) {
  const dim3 grid((unsigned)((p.padded + 128 * V - 1) / (128 * V)), (unsigned)most, (unsigned)batch);
  if (most == 1) {
    scan_kernel<T, V, true, true><<<grid, 128, 0, st>>>(p);
    return (int)cudaGetLastError();
  }
  scan_kernel<T, V, false, false><<<grid, 128, 0, st>>>(p);
  carry_kernel<T><<<dim3((unsigned)((p.width + 127) / 128), (unsigned)batch), 128, 0, st>>>(p);
  scan_kernel<T, V, true, false><<<grid, 128, 0, st>>>(p);
  return (int)cudaGetLastError();
}

}  // namespace gru
}  // namespace msrl

using namespace msrl;

// floats
MSRL_API long long msrl_min_gru_scratch(int width, int tokens, int batch, int max_q) {
  return max_q > gru::SEG ? 2LL * ((long long)tokens / gru::SEG + batch) * width + 8 : 4;
}

// z, x, g: first columns of the sections of rows [tokens, ld].  cu == null: one token per sequence
MSRL_API int msrl_min_gru(const void* z, const void* x, const void* g, long long ld, const float* z_bias, const float* x_bias,
                          float* state, const int* cu, const int* start, const long long* slots, float scale, void* y,
                          long long y_ld, int width, int padded, int tokens, int batch, int max_q, float* scratch, int is_f32,
                          cudaStream_t st) {
  if (batch == 0 || tokens == 0) return 0;
  if (batch > 65535) return (int)cudaErrorNotSupported;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const long long n = ((long long)tokens / gru::SEG + batch) * width;
    const gru::Args<T> p{(const T*)z, (const T*)x, (const T*)g, ld, z_bias, x_bias, state, cu, start, slots, scale, (T*)y, y_ld,
                         width, padded, scratch, scratch + (n + 3) / 4 * 4};
    const int most = cu == nullptr ? 1 : (max_q + gru::SEG - 1) / gru::SEG;
    auto at2 = [](const void* q) { return (reinterpret_cast<uintptr_t>(q) & (2 * sizeof(T) - 1)) == 0; };
    const bool v2 = width % 2 == 0 && padded % 2 == 0 && ld % 2 == 0 && y_ld % 2 == 0 && at2(z) && at2(x) && at2(g) && at2(y);
    return v2 ? gru::launch<T, 2>(p, most, batch, st) : gru::launch<T, 1>(p, most, batch, st);
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}
