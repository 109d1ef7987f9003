// Arguments shared by the kernels of wkv.cu and wkv_chunk.cu.
#pragma once
#include "dtype_utils.cuh"

namespace msrl {
namespace wkv {

template <typename T>
struct Args {
  const T *r, *k, *v, *g;                // [tokens, H * dim]
  const float* w;                        // decays, [tokens, H * dim]
  const float *u, *norm;                 // [H * dim]
  float* state;                          // [slots, H, dim, dim]
  const int* cu;
  const int* start;
  const long long* slots;
  T* y;                                  // [tokens, H * dim]
  int H, dim;
  float eps;
  int L;                                 // tokens of a segment
  float* seg;                            // [segments, H, dim, dim]: added states, then the states before the segments
  float* seg_w;                          // [segments, H, dim]: products of decays
  float* o;                              // [tokens, H * dim] where a head's columns are spread over blocks, else null
};

__device__ __forceinline__ long long seg_id(int t0, int b, int j, int L) { return t0 / L + b + j; }

constexpr int TT = 16;                   // tokens per tile

enum { WHOLE = 0, ADDED = 1, FROM_SEGMENT = 2 };

// wkv_chunk.cu: the same for bf16 rows with dim a multiple of 8 up to 128, sixteen tokens at a time on the tensor cores
int launch_chunked(const Args<__nv_bfloat16>& p, int mode, int segments, int batch, cudaStream_t st);
// decays of bf16 weights on the tensor cores: an even number of channels, rank up to 128
int launch_decay(const float* a, const __nv_bfloat16* w2, const float* w0, float* w, int tokens, int rank, int channels,
                 cudaStream_t st);

}  // namespace wkv
}  // namespace msrl
