// Between the fused q | k | v projection and grouped-head attention, one block per token, everything in fp32:
//
//   q, k <- RMS norm over the whole projection (all heads at once) * weight, then rotation of the first `rot` entries
//           of every head, entry i with entry i + rot / 2
//   v    <- (1 - mix) v + mix v_first, v_first = the values of another layer for the same token (optional)
//
// Results go back into the projection row (where prompt attention and the decode query read them) and, for k and v, to
// the token's cache rows.  Heads are padded (qp, vp); pad entries are zero on the way in and stay zero.
#include "dtype_utils.cuh"

namespace msrl {

template <typename T>
struct QkvArgs {
  T* proj;
  long long ld;
  int H, G, dim, vdim, qp, vp, q_col, k_col, v_col, rot, table_rows, first_vdim, first_vp;
  const float *q_norm, *k_norm;
  float eps;
  const float* table;                    // [table_rows, rot]: cos | sin
  const int* positions;
  const long long* slots;                // cache row per token, < 0: not cached
  T *k_cache, *v_cache;                  // [rows, G, qp], [rows, G, vp]
  const T* first;                        // or null
  long long first_ld;
  const float* mix;
};

// V entries at a time; every size and column is a multiple of V (rot of 2 V)
template <typename T, int V>
__global__ void __launch_bounds__(256) qkv_prep_kernel(const QkvArgs<T> p) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  T* row = p.proj + t * p.ld;
  const int nq = p.H * p.qp, nk = p.G * p.qp, nv = p.G * p.vp;
  float qq = 0.f, kk = 0.f;
  for (int c = threadIdx.x * V; c < nq; c += 256 * V) {
    float x[4];
    ldv<V>(row + p.q_col + c, x);
#pragma unroll
    for (int i = 0; i < V; ++i) qq += x[i] * x[i];
  }
  for (int c = threadIdx.x * V; c < nk; c += 256 * V) {
    float x[4];
    ldv<V>(row + p.k_col + c, x);
#pragma unroll
    for (int i = 0; i < V; ++i) kk += x[i] * x[i];
  }
  const long long slot = p.slots[t];
  // values do not wait for the norms
  T* vc = slot >= 0 ? p.v_cache + slot * nv : nullptr;
  const float lam = p.first != nullptr ? *p.mix : 0.f;
  for (int c = threadIdx.x * V; c < nv; c += 256 * V) {
    float x[4];
    ldv<V>(row + p.v_col + c, x);
    if (p.first != nullptr) {
      float f[4] = {0.f, 0.f, 0.f, 0.f};
      const int h = c / p.vp, d = c - h * p.vp;
      const T* fr = p.first + t * p.first_ld;
      if (p.first_vp == p.vp && p.first_vdim == p.vdim) {
        ldv<V>(fr + c, f);
      } else {
#pragma unroll
        for (int i = 0; i < V; ++i) {
          if (d + i < p.vdim) {
            const int e = h * p.vdim + d + i;
            f[i] = ldf(fr + e / p.first_vdim * p.first_vp + e % p.first_vdim);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < V; ++i) x[i] = (1.f - lam) * x[i] + lam * f[i];
      stv<V>(row + p.v_col + c, x);
    }
    if (vc != nullptr) stv<V>(vc + c, x);
  }
  const float rq = 1.f / sqrtf(block_sum(qq, red) / (float)(p.H * p.dim) + p.eps);
  const float rk = 1.f / sqrtf(block_sum(kk, red) / (float)(p.G * p.dim) + p.eps);
  const float* cs = p.table + (long long)min(max(p.positions[t], 0), p.table_rows - 1) * p.rot;
  const int half = p.rot / 2;
  T* kc = slot >= 0 ? p.k_cache + slot * nk : nullptr;
  // a head is `half` rotated pairs and qp - rot entries that pass: units of V pairs, then units of V entries
  const int pair_units = half / V, units = pair_units + (p.qp - p.rot) / V;
  for (int i = threadIdx.x; i < (p.H + p.G) * units; i += 256) {
    int h = i / units;
    const int u = i - h * units;
    const bool is_k = h >= p.H;
    if (is_k) h -= p.H;
    const int base = h * p.qp, d = u < pair_units ? u * V : p.rot + (u - pair_units) * V;
    T* x = row + (is_k ? p.k_col : p.q_col) + base;
    T* out = is_k && kc != nullptr ? kc + base : nullptr;
    const float* w = (is_k ? p.k_norm : p.q_norm) + base;
    const float r = is_k ? rk : rq;
    float a[4], wa[4];
    ldv<V>(x + d, a);
    ldv<V>(w + d, wa);
#pragma unroll
    for (int j = 0; j < V; ++j) a[j] *= r * wa[j];
    if (u < pair_units) {
      float b[4], wb[4], c[4], s[4], y[4];
      ldv<V>(x + d + half, b);
      ldv<V>(w + d + half, wb);
      ldv<V>(cs + d, c);
      ldv<V>(cs + half + d, s);
#pragma unroll
      for (int j = 0; j < V; ++j) {
        b[j] *= r * wb[j];
        y[j] = a[j] * c[j] - b[j] * s[j];
        b[j] = b[j] * c[j] + a[j] * s[j];
        a[j] = y[j];
      }
      stv<V>(x + d + half, b);
      if (out != nullptr) stv<V>(out + d + half, b);
    }
    stv<V>(x + d, a);
    if (out != nullptr) stv<V>(out + d, a);
  }
}

}  // namespace msrl

using namespace msrl;

// ints: H, G, dim, vdim, qp, vp, q_col, k_col, v_col, rot, table rows, vdim and vp of `first`
MSRL_API int msrl_qkv_prep(void* proj, long long ld, const int* ints, const float* q_norm, const float* k_norm, float eps,
                           const float* table, const int* positions, const long long* slots, void* k_cache, void* v_cache,
                           const void* first, long long first_ld, const float* mix, int tokens, int is_f32,
                           cudaStream_t st) {
  if (tokens == 0) return 0;
  if (ints[9] % 2 != 0 || ints[9] > ints[2] || (first != nullptr && mix == nullptr)) return (int)cudaErrorInvalidValue;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    QkvArgs<T> p{(T*)proj, ld, ints[0], ints[1], ints[2], ints[3], ints[4], ints[5], ints[6], ints[7], ints[8], ints[9],
                 ints[10], ints[11], ints[12], q_norm, k_norm, eps, table, positions, slots, (T*)k_cache, (T*)v_cache,
                 (const T*)first, first_ld, mix};
    const bool v4 = ld % 4 == 0 && p.qp % 4 == 0 && p.vp % 4 == 0 && p.q_col % 4 == 0 && p.k_col % 4 == 0 &&
                    p.v_col % 4 == 0 && p.rot % 8 == 0 && first_ld % 4 == 0 &&
                    (reinterpret_cast<uintptr_t>(first) & 15) == 0;
    if (v4) qkv_prep_kernel<T, 4><<<(unsigned)tokens, 256, 0, st>>>(p);
    else qkv_prep_kernel<T, 1><<<(unsigned)tokens, 256, 0, st>>>(p);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}
