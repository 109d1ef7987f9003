// Soft-max attention on the CUDA cores: any head sizes, fp32 arithmetic, bf16 or fp32 storage.  Serves what the
// tensor-core kernels do not: true 32-bit products and unusual head sizes.
//
//   attn_simt     packed sequences, causal (bottom-right aligned), grouped heads, optional window
//   decode_simt   one query per sequence over paged keys and values, optional window or chunk
//
// Both take a soft cap on the scores, a sink and a gate per head (head_tail.cuh).
#include "head_tail.cuh"

namespace msrl {

// ---- soft-max attention of packed sequences on the CUDA cores ------------------------------------------
template <typename T>
struct SimtArgs {
  const T *q, *k, *v;
  long long q_ld, k_ld, v_ld;
  int q_stride, k_stride, v_stride;      // head strides
  int dq, dv;
  int rep, window;                       // query heads per key head; keys a query sees (0: all)
  const int *cu_q, *cu_k;
  float scale, softcap;                  // softcap 0: not capped
  HeadTail<T> tail;
  T* out;                                // [tokens, H * o_stride]
  long long o_ld;
  int o_stride;
};

constexpr int SB = 32;                   // query rows and keys per tile

template <typename T, int ACC>
__global__ void __launch_bounds__(256) attn_simt_kernel(const SimtArgs<T> p) {
  extern __shared__ float smf[];
  const int ldq = p.dq + 1;
  float* sQ = smf;
  float* sK = sQ + SB * ldq;
  float* sV = sK + SB * ldq;
  float* sP = sV + SB * p.dv;            // [SB][SB + 1]
  const int h = blockIdx.y, b = blockIdx.z;
  const int q0 = p.cu_q[b], qlen = p.cu_q[b + 1] - q0, k0 = p.cu_k[b], klen = p.cu_k[b + 1] - k0;
  const int m0 = blockIdx.x * SB;
  if (m0 >= qlen) return;
  const int off = klen - qlen;           // bottom-right aligned causal mask
  const int row = threadIdx.x >> 3, part = threadIdx.x & 7;
  for (int i = threadIdx.x; i < SB * p.dq; i += 256) {
    const int r = i / p.dq, d = i % p.dq;
    sQ[r * ldq + d] = m0 + r < qlen ? ldf(p.q + (long long)(q0 + m0 + r) * p.q_ld + h * p.q_stride + d) : 0.f;
  }
  float acc[ACC];
#pragma unroll
  for (int i = 0; i < ACC; ++i) acc[i] = 0.f;
  float m_run = -INFINITY, l_run = 0.f;
  const int kmax = min(klen, m0 + SB + off), hk = h / p.rep;
  const int window = p.window > 0 ? p.window : klen + 1;
  for (int kb = max(m0 + off - window + 1, 0) / SB * SB; kb < kmax; kb += SB) {
    __syncthreads();
    for (int i = threadIdx.x; i < SB * p.dq; i += 256) {
      const int r = i / p.dq, d = i % p.dq;
      sK[r * ldq + d] = kb + r < klen ? ldf(p.k + (long long)(k0 + kb + r) * p.k_ld + hk * p.k_stride + d) : 0.f;
    }
    for (int i = threadIdx.x; i < SB * p.dv; i += 256) {
      const int r = i / p.dv, d = i % p.dv;
      sV[r * p.dv + d] = kb + r < klen ? ldf(p.v + (long long)(k0 + kb + r) * p.v_ld + hk * p.v_stride + d) : 0.f;
    }
    __syncthreads();
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    for (int d = 0; d < p.dq; ++d) {
      const float x = sQ[row * ldq + d];
#pragma unroll
      for (int j = 0; j < 4; ++j) s[j] += x * sK[(part + 8 * j) * ldq + d];
    }
    float mx = -INFINITY;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int key = kb + part + 8 * j;
      const int back = m0 + row + off - key;
      s[j] *= p.scale;
      if (p.softcap > 0.f) s[j] = softcapped(s[j], p.softcap);
      s[j] = key < klen && back >= 0 && back < window ? s[j] : -INFINITY;
      mx = fmaxf(mx, s[j]);
    }
#pragma unroll
    for (int x = 4; x > 0; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
    const float m_new = fmaxf(m_run, mx);
    const float m_use = m_new == -INFINITY ? 0.f : m_new;
    const float corr = expf(m_run - m_use);
    float sum = 0.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      s[j] = expf(s[j] - m_use);
      sum += s[j];
      sP[row * (SB + 1) + part + 8 * j] = s[j];
    }
#pragma unroll
    for (int x = 4; x > 0; x >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, x);
    l_run = l_run * corr + sum;
    m_run = m_new;
    __syncwarp();                        // a row's eight threads share a warp
#pragma unroll
    for (int i = 0; i < ACC; ++i) {
      const int c = part + 8 * i;
      if (c < p.dv) {
        float a = acc[i] * corr;
        for (int j = 0; j < SB; ++j) a += sP[row * (SB + 1) + j] * sV[j * p.dv + c];
        acc[i] = a;
      }
    }
  }
  if (m0 + row < qlen) {
    const float inv = p.tail.scale(q0 + m0 + row, h, m_run, l_run);
#pragma unroll
    for (int i = 0; i < ACC; ++i) {
      const int c = part + 8 * i;
      if (c < p.dv) stf(p.out + (long long)(q0 + m0 + row) * p.o_ld + h * p.o_stride + c, acc[i] * inv);
    }
  }
}

// ---- decode ------------------------------------------------------------------------------------------------
template <typename T>
struct PagedSimtArgs {
  const T* q;                            // one token per sequence, row stride q_ld, head stride qp
  long long q_ld;
  const T *k, *v;                        // [blocks, block_size, G, qp] and [.., vp]
  const int *block_tables, *context_lens;
  T* out;                                // [B, H * vp]
  int H, G, qp, vp, block_size, max_blocks, window, q_stride, chunk;      // chunk > 0: keys of the query's chunk
  float scale, softcap;
  HeadTail<T> tail;
};

constexpr int PS_ACC = 4;                // value columns per thread: vp <= 512

template <typename T>
__global__ void __launch_bounds__(128) paged_decode_simt_kernel(const PagedSimtArgs<T> p) {
  extern __shared__ float sQ[];
  __shared__ float sS[32];
  __shared__ long long sRow[32];
  const int h = blockIdx.x, b = blockIdx.y, hk = h / (p.H / p.G);
  const int n = p.context_lens[b];
  const int first = p.chunk > 0 ? max(n - 1, 0) / p.chunk * p.chunk : p.window > 0 ? max(n - p.window, 0) : 0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int c = threadIdx.x; c < p.qp; c += 128) sQ[c] = ldf(p.q + (long long)b * p.q_ld + h * p.q_stride + c);
  const int* bt = p.block_tables + (long long)b * p.max_blocks;
  float acc[PS_ACC] = {0.f, 0.f, 0.f, 0.f};
  float m_run = -INFINITY, l_run = 0.f;
  for (int kb = first; kb < n; kb += 32) {
    __syncthreads();
    for (int j = warp; j < 32; j += 4) {
      const int key = kb + j;
      float s = -INFINITY;
      long long row = 0;
      if (key < n) {
        row = ((long long)bt[key / p.block_size] * p.block_size + key % p.block_size) * p.G + hk;
        s = 0.f;
        for (int c = lane; c < p.qp; c += 32) s += sQ[c] * ldf(p.k + row * p.qp + c);
        s = warp_sum(s) * p.scale;
        if (p.softcap > 0.f) s = softcapped(s, p.softcap);
      }
      if (lane == 0) {
        sS[j] = s;
        sRow[j] = row;
      }
    }
    __syncthreads();
    float m_new = m_run;
    for (int j = 0; j < 32; ++j) m_new = fmaxf(m_new, sS[j]);
    const float corr = expf(m_run - m_new);
    l_run *= corr;
    m_run = m_new;
#pragma unroll
    for (int i = 0; i < PS_ACC; ++i) acc[i] *= corr;
    const int keys = min(32, n - kb);
    for (int j = 0; j < keys; ++j) {
      const float pj = expf(sS[j] - m_new);
      l_run += pj;
#pragma unroll
      for (int i = 0; i < PS_ACC; ++i) {
        const int c = threadIdx.x + 128 * i;
        if (c < p.vp) acc[i] += pj * ldf(p.v + sRow[j] * p.vp + c);
      }
    }
  }
  const float inv = p.tail.scale(b, h, m_run, l_run);
#pragma unroll
  for (int i = 0; i < PS_ACC; ++i) {
    const int c = threadIdx.x + 128 * i;
    if (c < p.vp) stf(p.out + ((long long)b * p.H + h) * p.vp + c, acc[i] * inv);
  }
}

}  // namespace msrl

using namespace msrl;

// lds: q, k, v, out row strides; ints: q, k, v, out head strides, dq, dv, query heads per key head, window (0: all)
MSRL_API int msrl_attn_simt(const void* q, const void* k, const void* v, void* out, const long long* lds,
                            const int* ints, const int* cu_q, const int* cu_k, int batch, int max_q, int H, float scale,
                            float softcap, const void* gate, long long gate_ld, const float* sink, int is_f32,
                            cudaStream_t st) {
  if (batch == 0 || max_q == 0) return 0;
  const int dq = ints[4], dv = ints[5];
  if (dv > 512 || batch > 65535 || H > 65535) return (int)cudaErrorNotSupported;
  const size_t smem = sizeof(float) * (2 * (size_t)SB * (dq + 1) + (size_t)SB * dv + SB * (SB + 1));
  if (smem > 227 * 1024) return (int)cudaErrorNotSupported;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    SimtArgs<T> p{(const T*)q, (const T*)k, (const T*)v, lds[0], lds[1], lds[2], ints[0], ints[1], ints[2],
                  dq, dv, ints[6], ints[7], cu_q, cu_k, scale, softcap, {(const T*)gate, gate_ld, sink}, (T*)out, lds[3], ints[3]};
    const dim3 grid((unsigned)((max_q + SB - 1) / SB), (unsigned)H, (unsigned)batch);
    auto go = [&](auto kernel) {
      cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
      kernel<<<grid, 256, smem, st>>>(p);
      return (int)cudaGetLastError();
    };
    if (dv <= 64) return go(attn_simt_kernel<T, 8>);
    if (dv <= 128) return go(attn_simt_kernel<T, 16>);
    if (dv <= 256) return go(attn_simt_kernel<T, 32>);
    return go(attn_simt_kernel<T, 64>);
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

// ints: H, G, qp, vp, block size, block-table width, window (0: all), query head stride, chunk (0: none)
MSRL_API int msrl_paged_decode_simt(const void* q, long long q_ld, const void* k, const void* v, const int* block_tables,
                                    const int* context_lens, void* out, const int* ints, int batch, float scale, float softcap,
                                    const void* gate, long long gate_ld, const float* sink, int is_f32, cudaStream_t st) {
  if (batch == 0) return 0;
  if (ints[3] > 128 * PS_ACC || ints[2] > 8192 || batch > 65535) return (int)cudaErrorNotSupported;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    PagedSimtArgs<T> p{(const T*)q, q_ld, (const T*)k, (const T*)v, block_tables, context_lens, (T*)out, ints[0], ints[1],
                       ints[2], ints[3], ints[4], ints[5], ints[6], ints[7], ints[8], scale, softcap, {(const T*)gate, gate_ld, sink}};
    paged_decode_simt_kernel<T><<<dim3((unsigned)p.H, (unsigned)batch), 128, p.qp * sizeof(float), st>>>(p);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}
