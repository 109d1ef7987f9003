// Short causal convolutions over time, one filter per channel, on rows of a projection.
//
// The last `taps` inputs of a sequence live in a ring of its state slot (entry p % taps holds position p).  With `taps`
// entries, one more than the next token needs, the entry a step writes is never one that the same step reads.
// Positions before the sequence's start count as zero, so a slot needs no clearing when it is used again.
#pragma once
#include "dtype_utils.cuh"

namespace msrl {

template <typename T>
struct ConvIn {
  const T* proj;             // [tokens, ld]
  long long ld;
  const float* conv;         // [channels, taps], last tap = current token
  int taps, channels;
  T* ring;                   // [slots, taps, channels]
};

// The convolution of one channel: `col` is its column in proj, `ch` its ring / weight row, `i` the token's index inside
// this portion (row t of proj), `pos` its position in the sequence.  TAPS > 0 fixes the number of taps so that all loads
// are in flight together.
template <int TAPS, typename T>
__device__ __forceinline__ float conv_one(const ConvIn<T>& p, long long t, int i, int pos, long long slot, int col, int ch) {
  const int taps = TAPS > 0 ? TAPS : p.taps;
  const T* ring = p.ring + slot * taps * p.channels + ch;
  float s = 0.f;
  if constexpr (TAPS > 0) {
    float x[TAPS], w[TAPS];
    const int at = pos % TAPS;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const int back = TAPS - 1 - j;
      const int entry = at - back < 0 ? at - back + TAPS : at - back;
      x[j] = 0.f;
      if (pos - back >= 0)
        x[j] = ldf(i - back >= 0 ? p.proj + (t - back) * p.ld + col : ring + (long long)entry * p.channels);
      w[j] = p.conv[(long long)ch * TAPS + j];
    }
#pragma unroll
    for (int j = 0; j < TAPS; ++j) s += x[j] * w[j];
  } else {
    for (int j = 0; j < taps; ++j) {
      const int back = taps - 1 - j;
      if (pos - back < 0) continue;
      s += ldf(i - back >= 0 ? p.proj + (t - back) * p.ld + col : ring + (long long)((pos - back) % taps) * p.channels) *
           p.conv[(long long)ch * taps + j];
    }
  }
  return s;
}

// Four neighbouring channels over consecutive tokens, the window in registers.
template <int TAPS, typename T>
struct ConvWindow {
  float w[TAPS][4], x[TAPS][4];
  __device__ __forceinline__ void weights(const float* conv, int ch) {
    // the 4 x TAPS weights lie side by side: ch is a multiple of 4
    float f[TAPS][4];
#pragma unroll
    for (int i = 0; i < TAPS; ++i) ldf4(conv + (long long)ch * TAPS + i * 4, f[i]);
#pragma unroll
    for (int c = 0; c < 4; ++c)
#pragma unroll
      for (int j = 0; j < TAPS; ++j) w[j][c] = f[(c * TAPS + j) / 4][(c * TAPS + j) % 4];
  }
  // window entries before token t (index i of its portion, position pos); x[TAPS - 1] is the token's own
  __device__ __forceinline__ void fill(const ConvIn<T>& p, long long t, int i, int pos, long long slot, int col, int ch) {
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j) {
      const int back = TAPS - 1 - j;            // shifted once more before use: entry j + 1 holds position pos - back
#pragma unroll
      for (int c = 0; c < 4; ++c) x[j + 1][c] = 0.f;
      if (pos - back >= 0) {
        if (i - back >= 0) ldf4(p.proj + (t - back) * p.ld + col, x[j + 1]);
        else ldf4(p.ring + (slot * TAPS + (pos - back) % TAPS) * p.channels + ch, x[j + 1]);
      }
    }
  }
  // U >= TAPS - 1 tokens at once: nothing is shifted in between
  template <int U>
  __device__ __forceinline__ void steps(float (&in)[U][4]) {
    static_assert(U >= TAPS - 1, "the window must lie inside the tokens");
    float last[TAPS > 1 ? TAPS - 1 : 1][4];
#pragma unroll
    for (int c = 0; c < 4; ++c) {
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j) last[j][c] = in[U - (TAPS - 1) + j][c];
#pragma unroll
      for (int n = U - 1; n >= 0; --n) {                 // from the last on: a token's input is still there for later ones
        float s = 0.f;
#pragma unroll
        for (int j = 0; j < TAPS; ++j) s += w[j][c] * (n + j < TAPS - 1 ? x[n + j + 1][c] : in[n + j < TAPS - 1 ? 0 : n + j - (TAPS - 1)][c]);
        in[n][c] = s;
      }
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j) x[j + 1][c] = last[j][c];
    }
  }
  __device__ __forceinline__ void step(const float (&in)[4], float (&y)[4]) {
#pragma unroll
    for (int c = 0; c < 4; ++c) {
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j) x[j][c] = x[j + 1][c];
      x[TAPS - 1][c] = in[c];
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) s += x[j][c] * w[j][c];
      y[c] = s;
    }
  }
};

// The last inputs of every portion, after all of its convolutions: channels [0, n0) lie from column c0 on, the next n1
// from c1 on, the rest from c2 on.
template <typename T>
__global__ void conv_ring_kernel(const ConvIn<T> p, int n0, int n1, int c0, int c1, int c2, const int* cu, const int* start_pos,
                                 const long long* slots) {
  const int b = blockIdx.y, len = cu[b + 1] - cu[b];
  const int ch = blockIdx.x * blockDim.x + threadIdx.x;
  if (ch >= p.channels) return;
  const int col = ch < n0 ? c0 + ch : ch < n0 + n1 ? c1 + ch - n0 : c2 + ch - n0 - n1;
  for (int i = max(0, len - p.taps); i < len; ++i) {
    const int pos = start_pos[b] + i;
    p.ring[(slots[b] * p.taps + pos % p.taps) * p.channels + ch] = p.proj[(cu[b] + i) * p.ld + col];
  }
}

}  // namespace msrl
