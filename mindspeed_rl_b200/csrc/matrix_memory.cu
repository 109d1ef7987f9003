// Matrix memory with exponential gates, for prompts (prefill portions) and single-token decode steps.
//
// Per head, state S [dim, vdim], n [dim] and a running maximum m, all fp32 and zero before a sequence's first token:
//
//   i = cap tanh((z_i + b_i) / cap),  f = log sigmoid(cap tanh((z_f + b_f) / cap))
//   m' = max(f + m, i);  S' = e^(f + m - m') S + e^(i - m') k v^T;  n' likewise with k alone
//   o = S'^T q / (max(|n' . q|, e^-m') + floor)            (q carries `scale`)
//   y = o / rms(o) * norm * sigmoid(gate)
//
// or, with a constant decay per head in place of the gates (linear attention),  S' = decay S + k v^T,  o = S'^T q.  The output
// gate is a sigmoid or a silu.
//
// What a sequence carries lives in a state slot (memory [slots, H, dim, vdim], norm [slots, H, dim], peak [slots, H]); the
// first token of a sequence ignores what the slot holds.
//
//   decode    one kernel: state read and written once, coalesced; a cluster of blocks shares a head's value columns
//             and exchanges the sums of squares through distributed shared memory
//   scan      prompts token by token, any sizes, fp32 arithmetic throughout, followed by `finish` (norm and gate)
//   chunked   bf16 prompts in chunks of 128 tokens, all chunks in parallel.  With b_t the sum of f from the chunk's start,
//             a_t = i_t - b_t and M_t = max(m before the chunk, a_s for s <= t), m_t = b_t + M_t and the weight of token s
//             in S_t is e^(a_s - M_t), that of the state before the chunk e^(m - M_t):
//               chunk_state   U = sum_s e^(a_s - max a) k_s v_s^T of every chunk
//               carry         running state over the chunks, element by element; leaves the state before every chunk
//               chunk_out     (Q K^T with the weights) V + (Q S) with the weights, denominators, norm and gate
//             chunk_state and chunk_out are in matrix_memory_tcgen05.cu.
#include <cooperative_groups.h>

#include "matrix_memory.cuh"

namespace msrl {
namespace mem {

namespace cg = cooperative_groups;

// ---- decode -----------------------------------------------------------------------------------------------
constexpr int DB = 8, DC = 4;            // state rows of a thread in flight, output columns of a thread (of 256 DC)

// grid (cluster = column slices, H, B); `positions` stands in for `start`
template <typename T>
__global__ void __launch_bounds__(256) decode_kernel(const Args<T> p) {
  extern __shared__ float sm[];
  __shared__ float red[32];
  __shared__ float4 part[256];
  __shared__ float slice_ss;
  const cg::cluster_group cluster = cg::this_cluster();
  const int h = blockIdx.y, b = blockIdx.z;
  const int width = p.vdim / gridDim.x, c0 = blockIdx.x * width;
  const long long slot = p.slots[b];
  T* y = p.y + (long long)b * p.H * p.vdim + h * p.vdim + c0;
  if (slot < 0) {                        // the same for the whole cluster
    for (int c = threadIdx.x; c < width; c += 256) stf(y + c, 0.f);
    return;
  }
  const bool fresh = p.start[b] == 0;
  float* sq = sm;
  float* sk = sm + p.dim;
  const T* row = p.proj + b * p.ld;
  const bool plain = p.decay != nullptr;
  float* nr = p.nrm + (slot * p.H + h) * p.dim;
  float m = 0.f, keep = 0.f, take = 1.f;
  if (plain) {
    if (!fresh) keep = p.decay[h];
  } else {
    float gi, gf;
    log_gates(p, b, h, gi, gf);
    const float m0 = fresh ? 0.f : p.peak[slot * p.H + h];
    m = fmaxf(gf + m0, gi);
    if (!fresh) keep = expf(gf + m0 - m);
    take = expf(gi - m);
  }
  float nq = 0.f;
  for (int d = threadIdx.x; d < p.dim; d += 256) {
    const float q = ldf(row + p.q_col + h * p.dim + d) * p.scale, k = take * ldf(row + p.k_col + h * p.dim + d);
    sq[d] = q;
    sk[d] = k;
    if (!plain) nq += q * (fresh ? k : keep * nr[d] + k);
  }
  float den = 1.f;
  if (plain) __syncthreads();            // sq, sk
  else den = fmaxf(fabsf(block_sum(nq, red)), expf(-m)) + p.floor;
  const int quads = width / 4, lanes = 256 / quads;
  const int cq = threadIdx.x % quads, rl = threadIdx.x / quads;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  if (rl < lanes) {
    float v[4];
    ldf4(row + p.v_col + h * p.vdim + c0 + cq * 4, v);
    float* S = p.memory + (slot * p.H + h) * p.dim * p.vdim + c0 + cq * 4;
    for (int r0 = rl; r0 < p.dim; r0 += lanes * DB) {
      float4 s[DB];
#pragma unroll
      for (int i = 0; i < DB; ++i) {
        const int r = r0 + i * lanes;
        s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (!fresh && r < p.dim) s[i] = *reinterpret_cast<const float4*>(S + (long long)r * p.vdim);
      }
#pragma unroll
      for (int i = 0; i < DB; ++i) {
        const int r = r0 + i * lanes;
        if (r < p.dim) {
          const float k = sk[r], q = sq[r];
          s[i].x = keep * s[i].x + k * v[0];
          s[i].y = keep * s[i].y + k * v[1];
          s[i].z = keep * s[i].z + k * v[2];
          s[i].w = keep * s[i].w + k * v[3];
          *reinterpret_cast<float4*>(S + (long long)r * p.vdim) = s[i];
          o.x += q * s[i].x;
          o.y += q * s[i].y;
          o.z += q * s[i].z;
          o.w += q * s[i].w;
        }
      }
    }
  }
  part[threadIdx.x] = o;
  __syncthreads();
  float val[DC], ss = 0.f;
#pragma unroll
  for (int i = 0; i < DC; ++i) {
    const int c = threadIdx.x + i * 256;
    val[i] = 0.f;
    if (c < width) {
      const float* f = reinterpret_cast<const float*>(part);
      for (int l = 0; l < lanes; ++l) val[i] += f[l * width + c];
      val[i] /= den;
    }
    ss += val[i] * val[i];
  }
  ss = block_sum(ss, red);
  if (gridDim.x > 1) {
    if (threadIdx.x == 0) slice_ss = ss;
    cluster.sync();
    ss = 0.f;
    for (unsigned r = 0; r < gridDim.x; ++r) ss += *cluster.map_shared_rank(&slice_ss, r);
    cluster.sync();                      // no block leaves while its sum is read; all have read n and m
  } else {
    __syncthreads();
  }
  if (blockIdx.x == 0 && !plain) {
    for (int d = threadIdx.x; d < p.dim; d += 256) nr[d] = fresh ? sk[d] : keep * nr[d] + sk[d];
    if (threadIdx.x == 0) p.peak[slot * p.H + h] = m;
  }
  const float inv = 1.f / sqrtf(ss / (float)p.rms_dim + p.eps);
#pragma unroll
  for (int i = 0; i < DC; ++i) {
    const int x = threadIdx.x + i * 256, c = h * p.vdim + c0 + x;
    if (x < width) {
      const float g = ldf(row + p.g_col + c);
      stf(y + x, val[i] * inv * p.norm[c] * out_gate(p, g, sigmoid_f(g)));
    }
  }
}

// ---- prompts, token by token --------------------------------------------------------------------------------
constexpr int ST = 16, SC = 32;          // tokens per tile, value columns per block

// NR state rows per thread: eight lanes share a column; dim <= 8 NR
template <typename T, int NR>
__global__ void __launch_bounds__(256) scan_kernel(const Args<T> p, float* o) {
  extern __shared__ float sm[];
  __shared__ float sv[ST][SC], sg[ST][3];                         // gates: keep, take, m
  float* sq = sm;
  float* sk = sm + ST * p.dim;
  const int c0 = blockIdx.x * SC, h = blockIdx.y, b = blockIdx.z;
  const int t0 = p.cu[b], len = p.cu[b + 1] - t0;
  if (len <= 0) return;
  const int lane8 = threadIdx.x & 7, col = threadIdx.x >> 3, c = c0 + col;
  const long long slot = p.slots[b];
  const bool old = p.start[b] > 0 && slot >= 0, plain = p.decay != nullptr;
  float S[NR], n[NR], m = old && !plain ? p.peak[slot * p.H + h] : 0.f;
  float* Sg = p.memory + (slot * p.H + h) * p.dim * p.vdim;
  float* ng = p.nrm + (slot * p.H + h) * p.dim;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = lane8 + 8 * i;
    const bool in = old && r < p.dim;
    S[i] = in && c < p.vdim ? Sg[(long long)r * p.vdim + c] : 0.f;
    n[i] = in && !plain ? ng[r] : 0.f;
  }
  for (int base = 0; base < len; base += ST) {
    const int nt = min(ST, len - base);
    __syncthreads();
    for (int x = threadIdx.x; x < nt * p.dim; x += 256) {
      const int s = x / p.dim, d = x % p.dim;
      const T* row = p.proj + (long long)(t0 + base + s) * p.ld + h * p.dim + d;
      sq[x] = ldf(row + p.q_col) * p.scale;
      sk[x] = ldf(row + p.k_col);
    }
    for (int x = threadIdx.x; x < nt * SC; x += 256) {
      const int s = x / SC, d = c0 + x % SC;
      sv[s][x % SC] = d < p.vdim ? ldf(p.proj + (long long)(t0 + base + s) * p.ld + p.v_col + h * p.vdim + d) : 0.f;
    }
    if (threadIdx.x < nt) log_gates(p, t0 + base + threadIdx.x, h, sg[threadIdx.x][1], sg[threadIdx.x][0]);
    __syncthreads();
    for (int s = 0; s < nt; ++s) {
      float keep = 0.f, take = 1.f;
      if (plain) {
        keep = p.decay[h];
      } else {
        const float gi = sg[s][1], gf = sg[s][0], top = fmaxf(gf + m, gi);
        keep = expf(gf + m - top);
        take = expf(gi - top);
        m = top;
      }
      const float v = sv[s][col] * take;
      float acc = 0.f, nq = 0.f;
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int r = lane8 + 8 * i;
        if (r < p.dim) {
          const float k = sk[s * p.dim + r], q = sq[s * p.dim + r];
          S[i] = keep * S[i] + k * v;
          n[i] = keep * n[i] + k * take;
          acc += S[i] * q;
          nq += n[i] * q;
        }
      }
#pragma unroll
      for (int x = 4; x > 0; x >>= 1) {
        acc += __shfl_xor_sync(0xffffffffu, acc, x);
        nq += __shfl_xor_sync(0xffffffffu, nq, x);
      }
      if (lane8 == 0 && c < p.vdim)
        o[((long long)(t0 + base + s) * p.H + h) * p.vdim + c] = plain ? acc : acc / (fmaxf(fabsf(nq), expf(-m)) + p.floor);
    }
  }
  if (slot < 0) return;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = lane8 + 8 * i;
    if (r < p.dim) {
      if (c < p.vdim) Sg[(long long)r * p.vdim + c] = S[i];
    }
  }
}

// n and m of the token-by-token form: every block of a head computes them, so a kernel of its own stores them once all
// blocks have read the old ones.  One block per (head, sequence).
template <typename T>
__global__ void __launch_bounds__(256) scan_norm_kernel(const Args<T> p) {
  __shared__ float sg[ST][3];
  const int h = blockIdx.x, b = blockIdx.y;
  const int t0 = p.cu[b], len = p.cu[b + 1] - t0;
  const long long slot = p.slots[b];
  if (len <= 0 || slot < 0) return;
  const bool old = p.start[b] > 0;
  float m = old ? p.peak[slot * p.H + h] : 0.f;
  float* ng = p.nrm + (slot * p.H + h) * p.dim;
  float n[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < 2; ++i)
    if (old && threadIdx.x + 256 * i < p.dim) n[i] = ng[threadIdx.x + 256 * i];
  for (int base = 0; base < len; base += ST) {
    const int nt = min(ST, len - base);
    __syncthreads();
    if (threadIdx.x < nt) log_gates(p, t0 + base + threadIdx.x, h, sg[threadIdx.x][1], sg[threadIdx.x][0]);
    __syncthreads();
    for (int s = 0; s < nt; ++s) {
      const float gi = sg[s][1], gf = sg[s][0];
      const float top = fmaxf(gf + m, gi), keep = expf(gf + m - top), take = expf(gi - top);
      m = top;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int d = threadIdx.x + 256 * i;
        if (d < p.dim) n[i] = keep * n[i] + take * ldf(p.proj + (long long)(t0 + base + s) * p.ld + p.k_col + h * p.dim + d);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < 2; ++i)
    if (threadIdx.x + 256 * i < p.dim) ng[threadIdx.x + 256 * i] = n[i];
  __syncthreads();
  if (threadIdx.x == 0) p.peak[slot * p.H + h] = m;
}

// y = o / rms(o) * norm * sigmoid(gate): one warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) finish_kernel(const Args<T> p, const float* o, long long rows) {
  const long long r = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (r >= rows) return;
  const int lane = threadIdx.x & 31, h = (int)(r % p.H);
  const long long t = r / p.H;
  const float* x = o + r * p.vdim;
  float ss = 0.f;
  for (int c = lane * 4; c < p.vdim; c += 128) {
    float f[4];
    ldf4(x + c, f);
    ss += f[0] * f[0] + f[1] * f[1] + f[2] * f[2] + f[3] * f[3];
  }
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.rms_dim + p.eps);
  for (int c = lane * 4; c < p.vdim; c += 128) {
    float f[4], g[4], w[4];
    ldf4(x + c, f);
    ldf4(p.proj + t * p.ld + p.g_col + h * p.vdim + c, g);
    ldf4(p.norm + h * p.vdim + c, w);
#pragma unroll
    for (int i = 0; i < 4; ++i) f[i] *= inv * w[i] * out_gate(p, g[i], sigmoid_t<T>(g[i]));
    stf4(p.y + r * p.vdim + c, f);
  }
}

// ---- prompts in chunks (bf16): the pass over the chunks ------------------------------------------------------------
using bf16 = __nv_bfloat16;

__device__ __forceinline__ float4 blend(float x, const float4& a, float y, const float4& b) {
  return make_float4(x * a.x + y * b.x, x * a.y + y * b.y, x * a.z + y * b.z, x * a.w + y * b.w);
}

// grid (state elements / 1024, H, B): four elements per thread, chunk after chunk
__global__ void __launch_bounds__(256) carry_kernel(const Args<bf16> p, const Chunks ch) {
  constexpr int AHEAD = 8;
  const int h = blockIdx.y, b = blockIdx.z;
  const int t0 = p.cu[b], len = p.cu[b + 1] - t0, n = (len + C - 1) / C;
  const long long size = (long long)p.dim * p.vdim, e = ((long long)blockIdx.x * 256 + threadIdx.x) * 4;
  if (len <= 0 || e >= size + (p.decay != nullptr ? 0 : p.dim)) return;
  const long long slot = p.slots[b], id0 = chunk_id(t0, b, 0) * p.H + h;
  const bool old = p.start[b] > 0 && slot >= 0;
  float* mine = e < size ? p.memory + (slot * p.H + h) * size + e : p.nrm + (slot * p.H + h) * p.dim + (e - size);
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  float m = 0.f;
  if (old) {
    s = *reinterpret_cast<const float4*>(mine);
    if (p.decay == nullptr) m = p.peak[slot * p.H + h];
  }
  float* u = ch.state + id0 * (size + p.dim) + e;
  const long long step = p.H * (size + p.dim);
  for (int j0 = 0; j0 < n; j0 += AHEAD) {
    float4 x[AHEAD];
    float tops[AHEAD], sums[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (j0 + i < n) {
        x[i] = *reinterpret_cast<const float4*>(u + (j0 + i) * step);
        tops[i] = ch.top[id0 + (long long)(j0 + i) * p.H];
        sums[i] = ch.sum[id0 + (long long)(j0 + i) * p.H];
      }
    }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (j0 + i < n) {
        const int j = j0 + i;
        *reinterpret_cast<float4*>(u + j * step) = s;
        if (e == 0) ch.before[id0 + (long long)j * p.H] = m;
        const float M = fmaxf(m, tops[i]);
        s = blend(expf(m - M), s, expf(tops[i] - M), x[i]);
        m = sums[i] + M;
      }
    }
  }
  if (slot < 0) return;
  *reinterpret_cast<float4*>(mine) = s;
}

// the new peaks, once every block of `carry` has read the old ones: one thread per (head, sequence)
__global__ void carry_peak_kernel(const Args<bf16> p, const Chunks ch, int batch) {
  const int x = blockIdx.x * blockDim.x + threadIdx.x;
  if (x >= batch * p.H) return;
  const int h = x % p.H, b = x / p.H, t0 = p.cu[b], len = p.cu[b + 1] - t0;
  const long long slot = p.slots[b];
  if (len <= 0 || slot < 0) return;
  const long long id = chunk_id(t0, b, (len - 1) / C) * p.H + h;
  p.peak[slot * p.H + h] = ch.sum[id] + fmaxf(ch.before[id], ch.top[id]);
}

}  // namespace mem
}  // namespace msrl

using namespace msrl;

// ints: H, dim, vdim (multiples of 16), entries of a head that count in its root mean square, columns of q, k, v, gate,
// silu gate; decay: see matrix_memory.cuh;
// floats: scale, cap, floor, eps
MSRL_API int msrl_memory_decode(const void* proj, long long ld, const float* z, long long z_ld, const int* ints,
                                const float* floats, const float* bias, const float* decay, const float* norm,
                                float* memory, float* nrm, float* peak, const int* positions, const long long* slots,
                                void* y, int batch, int is_f32, cudaStream_t st) {
  if (batch == 0) return 0;
  const int H = ints[0], dim = ints[1], vdim = ints[2];
  if (dim % 16 != 0 || vdim % 16 != 0 || batch > 65535 || H > 65535) return (int)cudaErrorInvalidValue;
  // column slices: down to 256 columns where they divide, and while the grid leaves multiprocessors idle down to 32
  int slices = 1;
  while (slices < 8 && vdim % (slices * 2 * 16) == 0 &&
         (vdim / slices > 256 || ((long long)batch * H * slices < 2 * sm_count() && vdim / (slices * 2) >= 32)))
    slices *= 2;
  if (vdim / slices > 256 * mem::DC) return (int)cudaErrorNotSupported;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const auto p = mem::make_args<T>(proj, ld, z, z_ld, ints, floats, bias, decay, norm, memory, nrm, peak, nullptr, positions,
                                     slots, y);
    cudaLaunchConfig_t cfg{};
    cfg.gridDim = dim3((unsigned)slices, (unsigned)H, (unsigned)batch);
    cfg.blockDim = dim3(256);
    cfg.dynamicSmemBytes = 2 * dim * sizeof(float);
    cfg.stream = st;
    cudaLaunchAttribute attr{};
    attr.id = cudaLaunchAttributeClusterDimension;
    attr.val.clusterDim.x = (unsigned)slices;
    attr.val.clusterDim.y = attr.val.clusterDim.z = 1;
    cfg.attrs = &attr;
    cfg.numAttrs = 1;
    return (int)cudaLaunchKernelEx(&cfg, mem::decode_kernel<T>, p);
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

// o: fp32 scratch [tokens, H * vdim]
MSRL_API int msrl_memory_prefill(const void* proj, long long ld, const float* z, long long z_ld, const int* ints,
                                 const float* floats, const float* bias, const float* decay, const float* norm,
                                 float* memory, float* nrm, float* peak, const int* cu, const int* start,
                                 const long long* slots, float* o, void* y, int tokens, int batch, int is_f32, cudaStream_t st) {
  if (batch == 0 || tokens == 0) return 0;
  const int H = ints[0], dim = ints[1], vdim = ints[2];
  if (dim > 512 || dim % 16 != 0 || vdim % 16 != 0 || batch > 65535 || H > 65535) return (int)cudaErrorNotSupported;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const auto p = mem::make_args<T>(proj, ld, z, z_ld, ints, floats, bias, decay, norm, memory, nrm, peak, cu, start, slots, y);
    const dim3 grid((unsigned)((vdim + mem::SC - 1) / mem::SC), (unsigned)H, (unsigned)batch);
    const size_t smem = 2 * mem::ST * (size_t)dim * sizeof(float);
    auto go = [&](auto kernel) {
      const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      if (e != cudaSuccess) return (int)e;
      kernel<<<grid, 256, smem, st>>>(p, o);
      return (int)cudaGetLastError();
    };
    const int rc = dim <= 64 ? go(mem::scan_kernel<T, 8>) : dim <= 128 ? go(mem::scan_kernel<T, 16>)
                   : dim <= 256 ? go(mem::scan_kernel<T, 32>) : go(mem::scan_kernel<T, 64>);
    if (rc != 0) return rc;
    if (decay == nullptr) mem::scan_norm_kernel<T><<<dim3((unsigned)H, (unsigned)batch), 256, 0, st>>>(p);
    const long long rows = (long long)tokens * H;
    mem::finish_kernel<T><<<(unsigned)((rows + 7) / 8), 256, 0, st>>>(p, o, rows);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

MSRL_API int msrl_memory_chunked_serves(const int* ints) { return ints[1] <= 256 && ints[1] % 16 == 0 && ints[2] % 16 == 0; }

// floats
MSRL_API long long msrl_memory_chunk_scratch(const int* ints, int tokens, int batch) {
  const long long H = ints[0], dim = ints[1], vdim = ints[2], chunks = tokens / mem::C + batch;
  return chunks * H * (dim * vdim + dim + 4) + 3 * H * tokens + 16 + (vdim > 128 ? (long long)tokens * H * vdim : 0);
}

// matrix_memory_tcgen05.cu
namespace msrl {
namespace mem {
int launch_chunk_state(const Args<__nv_bfloat16>& p, const Chunks& ch, int most, int batch, int* error, cudaStream_t st);
int launch_chunk_out(const Args<__nv_bfloat16>& p, const Chunks& ch, int most, int batch, int* error, cudaStream_t st);
}  // namespace mem
}  // namespace msrl

// The same for bf16 rows, in chunks; column starts and ld are multiples of 8.  error: device status word (0 = ok)
MSRL_API int msrl_memory_prefill_chunked(const void* proj, long long ld, const float* z, long long z_ld, const int* ints,
                                         const float* floats, const float* bias, const float* decay, const float* norm,
                                         float* memory, float* nrm, float* peak, const int* cu, const int* start,
                                         const long long* slots, float* scratch, void* y, int tokens, int batch, int max_q, int* error,
                                         cudaStream_t st) {
  if (batch == 0 || tokens == 0) return 0;
  const int H = ints[0], dim = ints[1], vdim = ints[2];
  if (!msrl_memory_chunked_serves(ints) || ld % 8 != 0 || batch > 65535 || H > 65535) return (int)cudaErrorNotSupported;
  for (int i = 4; i < 8; ++i)
    if (ints[i] % 8 != 0) return (int)cudaErrorNotSupported;
  const auto p = mem::make_args<__nv_bfloat16>(proj, ld, z, z_ld, ints, floats, bias, decay, norm, memory, nrm, peak, cu, start,
                                               slots, y);
  const long long chunks = tokens / mem::C + batch, size = (long long)dim * vdim + dim;
  mem::Chunks ch{};
  ch.state = scratch;
  ch.top = ch.state + chunks * H * size;
  ch.sum = ch.top + chunks * H;
  ch.before = ch.sum + chunks * H;
  ch.a = ch.before + chunks * H;
  ch.run = ch.a + (long long)H * tokens;
  ch.b = ch.run + (long long)H * tokens;
  ch.o = ch.b + (long long)H * tokens;
  ch.o += (16 - (reinterpret_cast<uintptr_t>(ch.o) & 15)) / 4 % 4;
  ch.tokens = tokens;
  const int most = (max_q + mem::C - 1) / mem::C;
  int rc = mem::launch_chunk_state(p, ch, most, batch, error, st);
  if (rc != 0) return rc;
  mem::carry_kernel<<<dim3((unsigned)((size + 1023) / 1024), (unsigned)H, (unsigned)batch), 256, 0, st>>>(p, ch);
  if (decay == nullptr) mem::carry_peak_kernel<<<(unsigned)(((long long)batch * H + 127) / 128), 128, 0, st>>>(p, ch, batch);
  rc = mem::launch_chunk_out(p, ch, most, batch, error, st);
  if (rc != 0 || vdim <= 128) return rc;
  const long long rows = (long long)tokens * H;
  mem::finish_kernel<__nv_bfloat16><<<(unsigned)((rows + 7) / 8), 256, 0, st>>>(p, ch.o, rows);
  return (int)cudaGetLastError();
}
