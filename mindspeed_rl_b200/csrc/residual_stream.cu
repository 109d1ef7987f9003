// Kernels around an fp32 residual stream (bf16 or fp32 activations, selected by `is_f32`).
//
//   embed_norm        resid[t] = scale * table[id[t]];                        y[t] = norm(resid[t])
//   add_norm          resid[t] += delta[t] + delta2[t];                       y[t] = norm(resid[t])
//   moe_combine_norm  resid[t] += w * sum_j e[pos(t, j)] + sig(h[t].sg) * sh[t] + delta2[t];  y[t] = norm(resid[t])
//
// norm(x) = x / sqrt(mean(x^2) + eps) * (offset + weight), all in fp32, with x less its mean when `centered` (the
// squares are then summed in a pass of their own over the kept row); y is stored in the activation type.  One block
// per row; the row stays in registers between the sum and the norm (longer rows than the register budget re-read the
// residual they just wrote).  A null `y` skips the norm; without a norm weight y is the residual itself.
//
//   post_add          d = delta[t], or sum_j w[t, j] * e[pos(t, j)] + sh[t] where a negative pos stands for the residual's
//                     row; resid[t] += mult * d / sqrt(mean(d^2) + eps) * weight;  y[t] = resid[t] or a norm of it.
//                     Between the add and y: resid[t] += again[t] + step (what a pass of a loop adds before it runs)
//   post_embed        the same with d = table[id[t]] and a residual that starts at zero; `first` keeps it as it was before
//                     `step`
//   side_gate         g[t] = gelu_tanh(g[t]) * rows[id[t]], or for few tokens with the product in it: g[t] = x[t] gate^T
//   soft_cap          x = cap * tanh(x / cap)
//
//   glu               act(gate) * up of rows [gate | up]: silu, tanh-gelu, or the clamped swish with (up + 1)
#include "dtype_utils.cuh"

namespace msrl {

constexpr int RS_THREADS = 256;

enum { SRC_EMBED = 0, SRC_DELTA = 1, SRC_MOE = 2 };

template <typename T>
struct RowArgs {
  float* resid;
  const float* norm_w;
  T* y;
  int W;
  float eps, offset;
  int centered;
  const T* delta2;                        // SRC_DELTA, SRC_MOE: one more term, or null
  // SRC_EMBED
  const long long* ids;
  const T* table;
  float scale;
  // SRC_DELTA
  const T* delta;
  // SRC_MOE
  const T* e;
  const int* pos;
  int top;
  float expert_w;
  const T* h;
  const T* sg;
  const T* shared;
};

// FULL: with the options `centered` and `delta2`
template <typename T, int V, int NPT, int SRC, bool FULL>
__global__ void __launch_bounds__(RS_THREADS) row_norm_kernel(const RowArgs<T> p) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const int W = p.W;
  float* res = p.resid + t * W;
  const T* tab = nullptr;
  if constexpr (SRC == SRC_EMBED) tab = p.table + p.ids[t] * W;
  float sig = 0.f;
  if constexpr (SRC == SRC_MOE) {
    if (p.shared != nullptr) {
      sig = 1.f;
      if (p.sg != nullptr) {
        float s = 0.f;
        for (int c = threadIdx.x * V; c < W; c += RS_THREADS * V) {
          float a[4], b[4];
          ldv<V>(p.h + t * W + c, a);
          ldv<V>(p.sg + c, b);
#pragma unroll
          for (int i = 0; i < V; ++i) s += a[i] * b[i];
        }
        sig = sigmoid_f(block_sum(s, red));
      }
    }
  }
  auto value = [&](int c, float (&f)[4]) {
    if constexpr (SRC == SRC_EMBED) {
      ldv<V>(tab + c, f);
#pragma unroll
      for (int i = 0; i < V; ++i) f[i] *= p.scale;
    } else if constexpr (SRC == SRC_DELTA) {
      float d[4];
      ldv<V>(res + c, f);
      ldv<V>(p.delta + t * W + c, d);
#pragma unroll
      for (int i = 0; i < V; ++i) f[i] += d[i];
      if (FULL && p.delta2 != nullptr) {
        ldv<V>(p.delta2 + t * W + c, d);
#pragma unroll
        for (int i = 0; i < V; ++i) f[i] += d[i];
      }
    } else {
      float d[4], acc[4] = {0.f, 0.f, 0.f, 0.f};
      for (int j = 0; j < p.top; ++j) {
        ldv<V>(p.e + (long long)p.pos[t * p.top + j] * W + c, d);
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] += d[i];
      }
      ldv<V>(res + c, f);
#pragma unroll
      for (int i = 0; i < V; ++i) acc[i] *= p.expert_w;
      if (p.shared != nullptr) {
        ldv<V>(p.shared + t * W + c, d);
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] += sig * d[i];
      }
      if (FULL && p.delta2 != nullptr) {
        ldv<V>(p.delta2 + t * W + c, d);
#pragma unroll
        for (int i = 0; i < V; ++i) acc[i] += d[i];
      }
#pragma unroll
      for (int i = 0; i < V; ++i) f[i] += acc[i];
    }
  };
  float keep[NPT][4];
  float ss = 0.f, sum = 0.f;
#pragma unroll
  for (int k = 0; k < NPT; ++k) {
    const int c = (k * RS_THREADS + threadIdx.x) * V;
    if (c < W) {
      value(c, keep[k]);
      stv<V>(res + c, keep[k]);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        ss += keep[k][i] * keep[k][i];
        if (FULL) sum += keep[k][i];
      }
    }
  }
  for (int c = (NPT * RS_THREADS + threadIdx.x) * V; c < W; c += RS_THREADS * V) {
    float f[4];
    value(c, f);
    stv<V>(res + c, f);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      ss += f[i] * f[i];
      if (FULL) sum += f[i];
    }
  }
  if (p.y == nullptr) return;
  T* y = p.y + t * W;
  if (SRC == SRC_EMBED && p.norm_w == nullptr) {
#pragma unroll
    for (int k = 0; k < NPT; ++k) {
      const int c = (k * RS_THREADS + threadIdx.x) * V;
      if (c < W) stv<V>(y + c, keep[k]);
    }
    for (int c = (NPT * RS_THREADS + threadIdx.x) * V; c < W; c += RS_THREADS * V) {
      float f[4];
      ldv<V>(res + c, f);
      stv<V>(y + c, f);
    }
    return;
  }
  float mean = 0.f;
  if (FULL && p.centered) {
    mean = block_sum(sum, red) / (float)W;
    ss = 0.f;
#pragma unroll
    for (int k = 0; k < NPT; ++k) {
      if ((k * RS_THREADS + threadIdx.x) * V < W) {
#pragma unroll
        for (int i = 0; i < V; ++i) {
          keep[k][i] -= mean;
          ss += keep[k][i] * keep[k][i];
        }
      }
    }
    for (int c = (NPT * RS_THREADS + threadIdx.x) * V; c < W; c += RS_THREADS * V) {
      float f[4];
      ldv<V>(res + c, f);
#pragma unroll
      for (int i = 0; i < V; ++i) ss += (f[i] - mean) * (f[i] - mean);
    }
  }
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)W + p.eps);
#pragma unroll
  for (int k = 0; k < NPT; ++k) {
    const int c = (k * RS_THREADS + threadIdx.x) * V;
    if (c < W) {
      float w[4];
      ldv<V>(p.norm_w + c, w);
#pragma unroll
      for (int i = 0; i < V; ++i) w[i] = keep[k][i] * r * (p.offset + w[i]);
      stv<V>(y + c, w);
    }
  }
  for (int c = (NPT * RS_THREADS + threadIdx.x) * V; c < W; c += RS_THREADS * V) {
    float f[4], w[4];
    ldv<V>(res + c, f);
    ldv<V>(p.norm_w + c, w);
#pragma unroll
    for (int i = 0; i < V; ++i) w[i] = (f[i] - mean) * r * (p.offset + w[i]);
    stv<V>(y + c, w);
  }
}

template <typename T, int SRC, bool FULL>
int launch_rows(const RowArgs<T>& p, long long rows, cudaStream_t st) {
  if (p.W % 4 == 0) {
    const int units = (p.W / 4 + RS_THREADS - 1) / RS_THREADS;
    if (units <= 1) row_norm_kernel<T, 4, 1, SRC, FULL><<<(unsigned)rows, RS_THREADS, 0, st>>>(p);
    else if (units <= 2) row_norm_kernel<T, 4, 2, SRC, FULL><<<(unsigned)rows, RS_THREADS, 0, st>>>(p);
    else if (units <= 4) row_norm_kernel<T, 4, 4, SRC, FULL><<<(unsigned)rows, RS_THREADS, 0, st>>>(p);
    else row_norm_kernel<T, 4, 8, SRC, FULL><<<(unsigned)rows, RS_THREADS, 0, st>>>(p);
  } else {
    row_norm_kernel<T, 1, 4, SRC, FULL><<<(unsigned)rows, RS_THREADS, 0, st>>>(p);
  }
  return (int)cudaGetLastError();
}

template <typename T, int SRC>
int launch_row_norm(const RowArgs<T>& p, long long rows, cudaStream_t st) {
  if (rows == 0) return 0;
  return p.centered || p.delta2 != nullptr ? launch_rows<T, SRC, true>(p, rows, st) : launch_rows<T, SRC, false>(p, rows, st);
}

enum { POST_ROWS = 0, POST_MOE = 1, POST_EMBED = 2 };

template <typename T>
struct PostArgs {
  const T* delta;                         // the sublayer's rows, or null:
  const T* e;                             // expert rows,
  const int* pos;                         // [rows, top]
  const float* weights;                   // [rows, top]
  int top;
  const T* shared;                        // one more term, or null
  float* resid;
  const float* norm_w;
  float eps, mult;
  const float* after_w;                   // norm of the sum, or null
  float after_eps;
  T* y;
  int W;
  const float* again;                     // ENTRY: [rows, W] and
  const float* step;                      // [W] that the sum gets before its norm, or null
  const long long* ids;                   // POST_EMBED
  const T* table;
  float* first;                           // [rows, W] or null
};

// adds the normed values to the residual (and, with ENTRY, what a pass adds); the sum stays in `a`
template <typename T, int V, bool ENTRY>
__device__ __forceinline__ void post_sum(const PostArgs<T>& p, long long t, int c, float inv, const float (&b)[4], float (&a)[4],
                                         float& sum) {
  const long long at = t * p.W + c;
  float w[4];
  ldv<V>(p.norm_w + c, w);
#pragma unroll
  for (int i = 0; i < V; ++i) a[i] += b[i] * inv * w[i];
  if constexpr (ENTRY) {
    if (p.first != nullptr) stv<V>(p.first + at, a);
    if (p.again != nullptr) {
      ldv<V>(p.again + at, w);
#pragma unroll
      for (int i = 0; i < V; ++i) a[i] += w[i];
    }
    if (p.step != nullptr) {
      ldv<V>(p.step + c, w);
#pragma unroll
      for (int i = 0; i < V; ++i) a[i] += w[i];
    }
  }
#pragma unroll
  for (int i = 0; i < V; ++i) sum += a[i] * a[i];
  stv<V>(p.resid + at, a);
  if (p.after_w == nullptr) stv<V>(p.y + at, a);
}

template <typename T, int V>
__device__ __forceinline__ void post_after(const PostArgs<T>& p, long long t, int c, float q, const float (&a)[4]) {
  float w[4];
  ldv<V>(p.after_w + c, w);
#pragma unroll
  for (int i = 0; i < V; ++i) w[i] *= a[i] * q;
  stv<V>(p.y + t * p.W + c, w);
}

// One block per row.  Rows up to NPT * 256 * V entries stay in registers; what is longer is computed again.
template <typename T, int V, int NPT, int SRC, bool ENTRY>
__global__ void __launch_bounds__(RS_THREADS) post_add_kernel(const PostArgs<T> p) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  const int W = p.W;
  float* res = p.resid + t * W;
  const T* rows = nullptr;
  if constexpr (SRC == POST_ROWS) rows = p.delta + t * W;
  if constexpr (SRC == POST_EMBED) rows = p.table + p.ids[t] * W;
  auto value = [&](int c, float (&r)[4], float (&d)[4]) {     // the residual's entries and the sublayer's
    if constexpr (SRC == POST_EMBED) {
#pragma unroll
      for (int i = 0; i < V; ++i) r[i] = 0.f;
    } else {
      ldv<V>(res + c, r);
    }
    if constexpr (SRC != POST_MOE) {
      ldv<V>(rows + c, d);
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) d[i] = 0.f;
      for (int j = 0; j < p.top; ++j) {
        const int at = p.pos[t * p.top + j];
        const float w = p.weights[t * p.top + j];
        float f[4];
        if (at >= 0) ldv<V>(p.e + (long long)at * W + c, f);
#pragma unroll
        for (int i = 0; i < V; ++i) d[i] += w * (at >= 0 ? f[i] : r[i]);
      }
      if (p.shared != nullptr) {
        float f[4];
        ldv<V>(p.shared + t * W + c, f);
#pragma unroll
        for (int i = 0; i < V; ++i) d[i] += f[i];
      }
    }
  };
  float r[NPT][4], d[NPT][4], ss = 0.f;
#pragma unroll
  for (int k = 0; k < NPT; ++k) {
    const int c = (k * RS_THREADS + threadIdx.x) * V;
    if (c < W) {
      value(c, r[k], d[k]);
#pragma unroll
      for (int i = 0; i < V; ++i) ss += d[k][i] * d[k][i];
    }
  }
  const int rest = (NPT * RS_THREADS + threadIdx.x) * V;
  for (int c = rest; c < W; c += RS_THREADS * V) {
    float a[4], b[4];
    value(c, a, b);
#pragma unroll
    for (int i = 0; i < V; ++i) ss += b[i] * b[i];
  }
  const float inv = p.mult / sqrtf(block_sum(ss, red) / (float)W + p.eps);
  float sum = 0.f;
#pragma unroll
  for (int k = 0; k < NPT; ++k) {
    const int c = (k * RS_THREADS + threadIdx.x) * V;
    if (c < W) post_sum<T, V, ENTRY>(p, t, c, inv, d[k], r[k], sum);
  }
  for (int c = rest; c < W; c += RS_THREADS * V) {
    float a[4], b[4];
    value(c, a, b);
    post_sum<T, V, ENTRY>(p, t, c, inv, b, a, sum);
  }
  if (p.after_w == nullptr) return;
  const float q = 1.f / sqrtf(block_sum(sum, red) / (float)W + p.after_eps);
#pragma unroll
  for (int k = 0; k < NPT; ++k) {
    const int c = (k * RS_THREADS + threadIdx.x) * V;
    if (c < W) post_after<T, V>(p, t, c, q, r[k]);
  }
  for (int c = rest; c < W; c += RS_THREADS * V) {
    float a[4];
    ldv<V>(res + c, a);
    post_after<T, V>(p, t, c, q, a);
  }
}

template <typename T, int SRC, bool ENTRY>
int launch_post_rows(const PostArgs<T>& p, long long rows, cudaStream_t st) {
  const unsigned g = (unsigned)rows;
  if (p.W % 4 != 0) {
    post_add_kernel<T, 1, 4, SRC, ENTRY><<<g, RS_THREADS, 0, st>>>(p);
  } else {
    const int units = (p.W / 4 + RS_THREADS - 1) / RS_THREADS;
    if (units <= 1) post_add_kernel<T, 4, 1, SRC, ENTRY><<<g, RS_THREADS, 0, st>>>(p);
    else if (units <= 2) post_add_kernel<T, 4, 2, SRC, ENTRY><<<g, RS_THREADS, 0, st>>>(p);
    else if (units <= 4) post_add_kernel<T, 4, 4, SRC, ENTRY><<<g, RS_THREADS, 0, st>>>(p);
    else post_add_kernel<T, 4, 8, SRC, ENTRY><<<g, RS_THREADS, 0, st>>>(p);
  }
  return (int)cudaGetLastError();
}

template <typename T, int SRC>
int launch_post(const PostArgs<T>& p, long long rows, cudaStream_t st) {
  if constexpr (SRC == POST_EMBED) return launch_post_rows<T, SRC, true>(p, rows, st);
  else return p.again != nullptr || p.step != nullptr ? launch_post_rows<T, SRC, true>(p, rows, st)
                                                      : launch_post_rows<T, SRC, false>(p, rows, st);
}

template <typename T>
__device__ __forceinline__ float gelu_tanh_t(float g) {
  const float k = 2.f * 0.7978845608028654f;             // 0.5 (1 + tanh(z)) = sigmoid(2 z), z = sqrt(2 / pi) (...)
  return g * sigmoid_t<T>(k * (g + 0.044715f * g * g * g));
}

// One warp per token and gate output: few tokens leave a matrix product nothing to share.  grid (padded dim / 8, tokens)
template <typename T, int V>
__global__ void __launch_bounds__(256)
side_gate_product_kernel(const T* x, const T* gate, T* g, long long g_ld, const T* rows, const long long* ids, long long ld, int col,
                         int dim, int W) {
  const long long t = blockIdx.y;
  const int j = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (j >= g_ld) return;
  float acc = 0.f;
  if (j < dim) {
    const T *a = x + t * W, *b = gate + (long long)j * W;
#pragma unroll 8
    for (int c = lane * V; c < W; c += 32 * V) {
      float f[4], h[4];
      ldv<V>(a + c, f);
      ldv<V>(b + c, h);
#pragma unroll
      for (int i = 0; i < V; ++i) acc += f[i] * h[i];
    }
  }
  acc = warp_sum(acc);
  if (lane == 0) stf(g + t * g_ld + j, j < dim ? gelu_tanh_t<T>(acc) * ldf(rows + ids[t] * ld + col + j) : 0.f);
}

// entries past `dim` of a padded row become zero
template <typename T>
__global__ void __launch_bounds__(256)
side_gate_kernel(T* g, long long g_ld, const T* rows, const long long* ids, long long ld, int col, int dim, long long n) {
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= n) return;
  const long long t = i / g_ld;
  const int j = (int)(i - t * g_ld);
  stf(g + i, j < dim ? gelu_tanh_t<T>(ldf(g + i)) * ldf(rows + ids[t] * ld + col + j) : 0.f);
}

template <typename T, int V>
__global__ void __launch_bounds__(256) soft_cap_kernel(T* x, long long n, float cap) {
  const long long i = ((long long)blockIdx.x * 256 + threadIdx.x) * V;
  if (i >= n) return;
  float f[4];
  ldv<V>(x + i, f);
#pragma unroll
  for (int k = 0; k < V; ++k)          // bf16 results: tanh z = 1 - 2 / (e^2z + 1) without the last bits
    f[k] = sizeof(T) == 2 ? cap - __fdividef(2.f * cap, __expf(2.f * f[k] / cap) + 1.f) : cap * tanhf(f[k] / cap);
  stv<V>(x + i, f);
}

enum { GLU_SILU = 0, GLU_GELU_TANH = 1, GLU_CLAMPED_SWISH = 2 };

template <int KIND, typename T>
__device__ __forceinline__ float glu_one(float g, float u, float limit, float alpha) {
  if constexpr (KIND == GLU_SILU) {
    return g * sigmoid_t<T>(g) * u;
  } else if constexpr (KIND == GLU_GELU_TANH) {
    return gelu_tanh_t<T>(g) * u;
  } else {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * sigmoid_t<T>(alpha * g) * (u + 1.f);
  }
}

// x [rows, 2F] -> y [rows, F]; rows of a 128-row tile whose tile_expert is negative are skipped, and inside a
// tile the pad rows past the expert's count
template <typename T, int V, int KIND>
__global__ void __launch_bounds__(256)
glu_kernel(const T* x, T* y, int F, float limit, float alpha, const int* tile_expert, const int* counts,
           const int* offsets) {
  const long long r = blockIdx.x;
  if (tile_expert != nullptr) {
    const int e = tile_expert[r / 128];
    if (e < 0 || r - offsets[e] >= counts[e]) return;
  }
  // two vectors a thread, both loads in flight
  float g[2][4], u[2][4];
  const int c0 = (blockIdx.y * 512 + threadIdx.x) * V;
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int c = c0 + k * 256 * V;
    if (c < F) {
      ldv<V>(x + r * 2 * F + c, g[k]);
      ldv<V>(x + r * 2 * F + F + c, u[k]);
    }
  }
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int c = c0 + k * 256 * V;
    if (c < F) {
#pragma unroll
      for (int i = 0; i < V; ++i) g[k][i] = glu_one<KIND, T>(g[k][i], u[k][i], limit, alpha);
      stv<V>(y + r * F + c, g[k]);
    }
  }
}

template <typename T, int V>
int launch_glu(const T* x, T* y, long long rows, int F, int kind, float limit, float alpha, const int* tile_expert,
               const int* counts, const int* offsets, cudaStream_t st) {
  const dim3 grid((unsigned)rows, (unsigned)((F / V + 511) / 512));
  if (kind == GLU_SILU)
    glu_kernel<T, V, GLU_SILU><<<grid, 256, 0, st>>>(x, y, F, limit, alpha, tile_expert, counts, offsets);
  else if (kind == GLU_GELU_TANH)
    glu_kernel<T, V, GLU_GELU_TANH><<<grid, 256, 0, st>>>(x, y, F, limit, alpha, tile_expert, counts, offsets);
  else
    glu_kernel<T, V, GLU_CLAMPED_SWISH><<<grid, 256, 0, st>>>(x, y, F, limit, alpha, tile_expert, counts, offsets);
  return (int)cudaGetLastError();
}

}  // namespace msrl

using namespace msrl;

template <typename T>
static RowArgs<T> base_args(float* resid, const float* norm_w, void* y, int W, float eps, float offset,
                            int centered) {
  RowArgs<T> p{};
  p.resid = resid;
  p.norm_w = norm_w;
  p.y = (T*)y;
  p.W = W;
  p.eps = eps;
  p.offset = offset;
  p.centered = centered;
  return p;
}

MSRL_API int msrl_embed_norm(const long long* ids, const void* table, float scale, float* resid, const float* norm_w,
                             void* y, long long rows, int W, float eps, float offset, int centered, int is_f32,
                             cudaStream_t st) {
  auto run = [&](auto tag) {
    using T = decltype(tag);
    RowArgs<T> p = base_args<T>(resid, norm_w, y, W, eps, offset, centered);
    p.ids = ids;
    p.table = (const T*)table;
    p.scale = scale;
    return launch_row_norm<T, SRC_EMBED>(p, rows, st);
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

MSRL_API int msrl_add_norm(const void* delta, const void* delta2, float* resid, const float* norm_w, void* y,
                           long long rows, int W, float eps, float offset, int centered, int is_f32, cudaStream_t st) {
  auto run = [&](auto tag) {
    using T = decltype(tag);
    RowArgs<T> p = base_args<T>(resid, norm_w, y, W, eps, offset, centered);
    p.delta = (const T*)delta;
    p.delta2 = (const T*)delta2;
    return launch_row_norm<T, SRC_DELTA>(p, rows, st);
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

MSRL_API int msrl_moe_combine_norm(const void* e, const int* pos, int top, float expert_w, const void* h,
                                   const void* sg, const void* shared, const void* delta, float* resid,
                                   const float* norm_w, void* y, long long rows, int W, float eps, float offset,
                                   int centered, int is_f32, cudaStream_t st) {
  auto run = [&](auto tag) {
    using T = decltype(tag);
    RowArgs<T> p = base_args<T>(resid, norm_w, y, W, eps, offset, centered);
    p.e = (const T*)e;
    p.pos = pos;
    p.top = top;
    p.expert_w = expert_w;
    p.h = (const T*)h;
    p.sg = (const T*)sg;
    p.shared = (const T*)shared;
    p.delta2 = (const T*)delta;
    return launch_row_norm<T, SRC_MOE>(p, rows, st);
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

template <typename T>
static PostArgs<T> post_args(float* resid, const float* norm_w, float eps, float mult, const float* after_w, float after_eps,
                             const float* again, const float* step, void* y, int W) {
  PostArgs<T> p{};
  p.resid = resid;
  p.norm_w = norm_w;
  p.eps = eps;
  p.mult = mult;
  p.after_w = after_w;
  p.after_eps = after_eps;
  p.again = again;
  p.step = step;
  p.y = (T*)y;
  p.W = W;
  return p;
}

MSRL_API int msrl_post_add(const void* delta, const void* e, const int* pos, const float* weights, int top, const void* shared,
                           float* resid, const float* norm_w, float eps, float mult, const float* after_w, float after_eps,
                           const float* again, const float* step, void* y, long long rows, int W, int is_f32,
                           cudaStream_t st) {
  if (rows == 0) return 0;
  if (delta == nullptr && (e == nullptr || pos == nullptr || weights == nullptr)) return (int)cudaErrorInvalidValue;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    PostArgs<T> p = post_args<T>(resid, norm_w, eps, mult, after_w, after_eps, again, step, y, W);
    p.delta = (const T*)delta;
    p.e = (const T*)e;
    p.pos = pos;
    p.weights = weights;
    p.top = top;
    p.shared = (const T*)shared;
    return delta == nullptr ? launch_post<T, POST_MOE>(p, rows, st) : launch_post<T, POST_ROWS>(p, rows, st);
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

MSRL_API int msrl_post_embed(const long long* ids, const void* table, float* resid, float* first, const float* norm_w, float eps,
                             float mult, const float* after_w, float after_eps, const float* step, void* y, long long rows,
                             int W, int is_f32, cudaStream_t st) {
  if (rows == 0) return 0;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    PostArgs<T> p = post_args<T>(resid, norm_w, eps, mult, after_w, after_eps, nullptr, step, y, W);
    p.ids = ids;
    p.table = (const T*)table;
    p.first = first;
    return launch_post<T, POST_EMBED>(p, rows, st);
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

// x [rows, W] -> g [rows, g_ld] with gate [>= dim, W]
MSRL_API int msrl_side_gate_product(const void* x, const void* gate, void* g, long long g_ld, const void* table,
                                    const long long* ids, long long ld, int col, int dim, long long rows, int W, int is_f32,
                                    cudaStream_t st) {
  if (rows == 0) return 0;
  if (rows > 65535) return (int)cudaErrorNotSupported;
  const dim3 grid((unsigned)((g_ld + 7) / 8), (unsigned)rows);
  auto run = [&](auto tag) {
    using T = decltype(tag);
    auto* kernel = W % 4 == 0 ? side_gate_product_kernel<T, 4> : side_gate_product_kernel<T, 1>;
    kernel<<<grid, 256, 0, st>>>((const T*)x, (const T*)gate, (T*)g, g_ld, (const T*)table, ids, ld, col, dim, W);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

MSRL_API int msrl_side_gate(void* g, long long g_ld, const void* table, const long long* ids, long long ld, int col, int dim,
                            long long rows, int is_f32, cudaStream_t st) {
  const long long n = rows * g_ld;
  if (n == 0) return 0;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    side_gate_kernel<T><<<(unsigned)((n + 255) / 256), 256, 0, st>>>((T*)g, g_ld, (const T*)table, ids, ld, col, dim, n);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

MSRL_API int msrl_soft_cap(void* x, long long n, float cap, int is_f32, cudaStream_t st) {
  if (n == 0) return 0;
  if (!(cap > 0.f)) return (int)cudaErrorInvalidValue;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    if (n % 4 == 0) soft_cap_kernel<T, 4><<<(unsigned)((n / 4 + 255) / 256), 256, 0, st>>>((T*)x, n, cap);
    else soft_cap_kernel<T, 1><<<(unsigned)((n + 255) / 256), 256, 0, st>>>((T*)x, n, cap);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

MSRL_API int msrl_glu_fwd(const void* x, void* y, long long rows, int F, int kind, float limit, float alpha,
                          const int* tile_expert, const int* counts, const int* offsets, int is_f32,
                          cudaStream_t st) {
  if (rows == 0 || F == 0) return 0;
  if (kind < 0 || kind > 2) return (int)cudaErrorInvalidValue;
  const bool v4 = F % 4 == 0;
  if (is_f32)
    return v4 ? launch_glu<float, 4>((const float*)x, (float*)y, rows, F, kind, limit, alpha, tile_expert, counts, offsets, st)
              : launch_glu<float, 1>((const float*)x, (float*)y, rows, F, kind, limit, alpha, tile_expert, counts, offsets, st);
  return v4 ? launch_glu<__nv_bfloat16, 4>((const __nv_bfloat16*)x, (__nv_bfloat16*)y, rows, F, kind, limit, alpha, tile_expert, counts, offsets, st)
            : launch_glu<__nv_bfloat16, 1>((const __nv_bfloat16*)x, (__nv_bfloat16*)y, rows, F, kind, limit, alpha, tile_expert, counts, offsets, st);
}
