// Arguments shared by the kernels of matrix_memory.cu and matrix_memory_tcgen05.cu.
#pragma once
#include "dtype_utils.cuh"

namespace msrl {
namespace mem {

template <typename T>
struct Args {
  const T* proj;                         // [tokens, ld]: q | k | v | gate sections at the given columns
  long long ld;
  const float* z;                        // [tokens, z_ld]: input gate logits [H] | forget gate logits [H]
  long long z_ld;
  int H, dim, vdim, rms_dim, q_col, k_col, v_col, g_col;
  int silu;                              // the output gate: silu, else sigmoid
  float scale, cap, floor, eps;
  const float* bias;                     // [2 H]
  const float* decay;                    // [2 H]: a constant decay per head and its logarithm, or null.  With it there are no
                                         // gates (i = 0, so m stays zero) and no denominator; z, bias, nrm and peak are unused
  const float* norm;                     // [H * vdim]
  float *memory, *nrm, *peak;
  const int* cu;
  const int* start;                      // position of a portion's first token
  const long long* slots;
  T* y;                                  // [tokens, H * vdim]
};

template <typename T>
__device__ __forceinline__ void log_gates(const Args<T>& p, long long t, int h, float& i, float& f) {
  if (p.decay != nullptr) {
    i = 0.f;
    f = p.decay[p.H + h];
    return;
  }
  const float* z = p.z + t * p.z_ld + h;
  i = p.cap * tanhf((z[0] + p.bias[h]) / p.cap);
  const float x = p.cap * tanhf((z[p.H] + p.bias[p.H + h]) / p.cap);
  f = fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}

template <typename T>
__device__ __forceinline__ float out_gate(const Args<T>& p, float g, float s) { return p.silu ? g * s : s; }   // s = sigmoid(g)

template <typename T>
Args<T> make_args(const void* proj, long long ld, const float* z, long long z_ld, const int* ints, const float* floats,
                  const float* bias, const float* decay, const float* norm, float* memory, float* nrm, float* peak,
                  const int* cu, const int* start, const long long* slots, void* y) {
  return Args<T>{(const T*)proj, ld, z, z_ld, ints[0], ints[1], ints[2], ints[3], ints[4], ints[5], ints[6], ints[7],
                 ints[8], floats[0], floats[1], floats[2], floats[3], bias, decay, norm, memory, nrm, peak, cu, start, slots, (T*)y};
}

// bf16 prompts in chunks of C tokens
constexpr int C = 128;

struct Chunks {
  float* state;                          // [chunks, H, dim * vdim + dim]: U and its n part, then the state before the chunk
  float *top, *sum, *before;             // [chunks, H]: max a, sum of f, m before the chunk
  float *a, *run, *b;                    // [H, tokens]: a, running max of a, sum of f inside the chunk
  float* o;                              // [tokens, H * vdim] when a head does not fit one block's columns
  int tokens;
};

__device__ __forceinline__ long long chunk_id(int t0, int b, int j) { return t0 / C + b + j; }

}  // namespace mem
}  // namespace msrl
