// Between the fused q | k | v projection and grouped-head attention, one block per token, everything in fp32:
//
//   q, k <- RMS norm over the whole projection (all heads at once) * weight, then rotation of the first `rot` entries
//           of every head, entry i with entry i + rot / 2
//   v    <- (1 - mix) v + mix v_first, v_first = the values of another layer for the same token (optional)
//
// Results go back into the projection row (where prompt attention and the decode query read them) and, for k and v, to
// the token's cache rows.  Heads are padded (qp, vp); pad entries are zero on the way in and stay zero.
//
// `turned_prep` is the form without norms of q and k whose values are normed per head (RMS, no weight) and turned by the
// token's position over all their entries, entry m with m + vdim / 2; `turn_back` turns attention outputs back by the
// query's position, scales them and stores them as columns of a wider row.
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

template <typename T>
struct TurnArgs {
  T* proj;
  long long ld;
  int H, G, dim, vdim, qp, vp, q_col, k_col, v_col, rot, table_rows;
  float eps;
  const float* table;                    // [table_rows, rot]: cos | sin for queries and keys
  const float* vtable;                   // [table_rows, vdim]: the same for values
  const int* positions;
  const long long* slots;                // cache row per token, < 0: not cached
  T *k_cache, *v_cache;                  // [rows, G, qp], [rows, G, vp]
};

// V entries at a time of pairs (d, d + half) of x, turned by the angle of (c, s); sign turns back
template <int V>
__device__ __forceinline__ void turn_pairs(float (&a)[4], float (&b)[4], const float* cs, int half, int d, float sign, float mult) {
  float c[4], s[4];
  ldv<V>(cs + d, c);
  ldv<V>(cs + half + d, s);
#pragma unroll
  for (int j = 0; j < V; ++j) {
    const float y = (a[j] * c[j] - sign * b[j] * s[j]) * mult;
    b[j] = (b[j] * c[j] + sign * a[j] * s[j]) * mult;
    a[j] = y;
  }
}

// One block per token: a warp per value head first (norm and rotation), then units of q and k spread over the threads.
template <typename T, int V>
__global__ void __launch_bounds__(256) turned_prep_kernel(const TurnArgs<T> p) {
  const long long t = blockIdx.x;
  T* row = p.proj + t * p.ld;
  const long long slot = p.slots[t];
  const long long at = min(max(p.positions[t], 0), p.table_rows - 1);
  const float* cs = p.table + at * p.rot;
  const float* vcs = p.vtable + at * p.vdim;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int vhalf = p.vdim / 2, half = p.rot / 2;
  for (int g = warp; g < p.G; g += 8) {
    T* x = row + p.v_col + g * p.vp;
    T* out = slot >= 0 ? p.v_cache + (slot * p.G + g) * p.vp : nullptr;
    float ss = 0.f;
    for (int c = lane * V; c < p.vdim; c += 32 * V) {
      float f[4];
      ldv<V>(x + c, f);
#pragma unroll
      for (int i = 0; i < V; ++i) ss += f[i] * f[i];
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
    for (int d = lane * V; d < vhalf; d += 32 * V) {
      float a[4], b[4];
      ldv<V>(x + d, a);
      ldv<V>(x + d + vhalf, b);
      turn_pairs<V>(a, b, vcs, vhalf, d, 1.f, inv);
      stv<V>(x + d, a);
      stv<V>(x + d + vhalf, b);
      if (out != nullptr) {
        stv<V>(out + d, a);
        stv<V>(out + d + vhalf, b);
      }
    }
    if (out != nullptr)
      for (int d = p.vdim + lane; d < p.vp; d += 32) stf(out + d, 0.f);
  }
  // rotated pairs of queries and keys; what a key passes unchanged only goes to the cache
  const int units = half / V;
  for (int i = threadIdx.x; i < (p.H + p.G) * units; i += 256) {
    int h = i / units;
    const int d = (i - h * units) * V;
    const bool is_k = h >= p.H;
    if (is_k) h -= p.H;
    T* x = row + (is_k ? p.k_col : p.q_col) + h * p.qp;
    float a[4], b[4];
    ldv<V>(x + d, a);
    ldv<V>(x + d + half, b);
    turn_pairs<V>(a, b, cs, half, d, 1.f, 1.f);
    stv<V>(x + d, a);
    stv<V>(x + d + half, b);
    if (is_k && slot >= 0) {
      T* out = p.k_cache + (slot * p.G + h) * p.qp;
      stv<V>(out + d, a);
      stv<V>(out + d + half, b);
    }
  }
  if (slot < 0) return;
  const int pass = (p.qp - p.rot) / V;
  for (int i = threadIdx.x; i < p.G * pass; i += 256) {
    const int h = i / pass, d = p.rot + (i - h * pass) * V;
    float a[4];
    ldv<V>(row + p.k_col + h * p.qp + d, a);
    stv<V>(p.k_cache + (slot * p.G + h) * p.qp + d, a);
  }
}

// attn [tokens, H, vp] -> out [tokens, ld] (H * vp columns); one block per token
template <typename T, int V>
__global__ void __launch_bounds__(256)
turn_back_kernel(const T* attn, T* out, long long ld, int H, int vdim, int vp, const float* table, int table_rows,
                 const int* positions, float scale) {
  const long long t = blockIdx.x;
  const float* cs = table + (long long)min(max(positions[t], 0), table_rows - 1) * vdim;
  const T* in = attn + t * H * vp;
  T* o = out + t * ld;
  const int half = vdim / 2, pairs = half / V;
  for (int i = threadIdx.x; i < H * pairs; i += 256) {
    const int h = i / pairs, d = (i - h * pairs) * V;
    float a[4], b[4];
    ldv<V>(in + h * vp + d, a);
    ldv<V>(in + h * vp + d + half, b);
    turn_pairs<V>(a, b, cs, half, d, -1.f, scale);
    stv<V>(o + h * vp + d, a);
    stv<V>(o + h * vp + d + half, b);
  }
  const int pad = vp - vdim;
  for (int i = threadIdx.x; i < H * pad; i += 256) stf(o + i / pad * vp + vdim + i % pad, 0.f);
}

}  // namespace msrl

using namespace msrl;

// ints: H, G, dim, vdim, qp, vp, q_col, k_col, v_col, rot, table rows
MSRL_API int msrl_turned_prep(void* proj, long long ld, const int* ints, float eps, const float* table, const float* vtable,
                              const int* positions, const long long* slots, void* k_cache, void* v_cache, int tokens,
                              int is_f32, cudaStream_t st) {
  if (tokens == 0) return 0;
  if (ints[9] % 2 != 0 || ints[9] > ints[2] || ints[3] % 2 != 0) return (int)cudaErrorInvalidValue;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const TurnArgs<T> p{(T*)proj, ld, ints[0], ints[1], ints[2], ints[3], ints[4], ints[5], ints[6], ints[7], ints[8], ints[9],
                        ints[10], eps, table, vtable, positions, slots, (T*)k_cache, (T*)v_cache};
    const bool v4 = ld % 4 == 0 && p.qp % 4 == 0 && p.vp % 4 == 0 && p.q_col % 4 == 0 && p.k_col % 4 == 0 &&
                    p.v_col % 4 == 0 && p.rot % 8 == 0 && p.vdim % 8 == 0;
    if (v4) turned_prep_kernel<T, 4><<<(unsigned)tokens, 256, 0, st>>>(p);
    else turned_prep_kernel<T, 1><<<(unsigned)tokens, 256, 0, st>>>(p);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

MSRL_API int msrl_turn_back(const void* attn, void* out, long long ld, int H, int vdim, int vp, const float* table,
                            int table_rows, const int* positions, float scale, int tokens, int is_f32, cudaStream_t st) {
  if (tokens == 0) return 0;
  if (vdim % 2 != 0) return (int)cudaErrorInvalidValue;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const bool v4 = vdim % 8 == 0 && vp % 4 == 0 && ld % 4 == 0 && (reinterpret_cast<uintptr_t>(out) & 15) == 0;
    if (v4) turn_back_kernel<T, 4><<<(unsigned)tokens, 256, 0, st>>>((const T*)attn, (T*)out, ld, H, vdim, vp, table, table_rows,
                                                                     positions, scale);
    else turn_back_kernel<T, 1><<<(unsigned)tokens, 256, 0, st>>>((const T*)attn, (T*)out, ld, H, vdim, vp, table, table_rows,
                                                                  positions, scale);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

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
