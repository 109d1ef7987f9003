// Matrix memory with exponential gates, for prompts (prefill portions) and single-token decode steps.
//
// Per head, state S [dim, vdim], n [dim] and a running maximum m, all fp32 and zero before a sequence's first token:
//
//   i = cap tanh((z_i + b_i) / cap),  f = log sigmoid(cap tanh((z_f + b_f) / cap))
//   m' = max(f + m, i);  S' = e^(f + m - m') S + e^(i - m') k v^T;  n' likewise with k alone
//   o = S'^T q / (max(|n' . q|, e^-m') + floor)            (q carries `scale`)
//   y = o / rms(o) * norm * sigmoid(gate)
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
//             Products run on the tensor cores with 32-bit operands (weights times keys, weighted scores, the state)
//             taken apart into three bf16 terms of 24 bits together; the other operand is exact, sums are fp32.
#include <cooperative_groups.h>

#include "dtype_utils.cuh"
#include "mma_utils.cuh"

namespace msrl {
namespace mem {

namespace cg = cooperative_groups;

template <typename T>
struct Args {
  const T* proj;                         // [tokens, ld]: q | k | v | gate sections at the given columns
  long long ld;
  const float* z;                        // [tokens, z_ld]: input gate logits [H] | forget gate logits [H]
  long long z_ld;
  int H, dim, vdim, rms_dim, q_col, k_col, v_col, g_col;
  float scale, cap, floor, eps;
  const float* bias;                     // [2 H]
  const float* norm;                     // [H * vdim]
  float *memory, *nrm, *peak;
  const int* cu;
  const int* start;                      // position of a portion's first token
  const long long* slots;
  T* y;                                  // [tokens, H * vdim]
};

template <typename T>
__device__ __forceinline__ void log_gates(const Args<T>& p, long long t, int h, float& i, float& f) {
  const float* z = p.z + t * p.z_ld + h;
  i = p.cap * tanhf((z[0] + p.bias[h]) / p.cap);
  const float x = p.cap * tanhf((z[p.H] + p.bias[p.H + h]) / p.cap);
  f = fminf(x, 0.f) - log1pf(expf(-fabsf(x)));
}

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
  float* nr = p.nrm + (slot * p.H + h) * p.dim;
  float gi, gf;
  log_gates(p, b, h, gi, gf);
  const float m0 = fresh ? 0.f : p.peak[slot * p.H + h];
  const float m = fmaxf(gf + m0, gi);
  const float keep = fresh ? 0.f : expf(gf + m0 - m), take = expf(gi - m);
  float nq = 0.f;
  for (int d = threadIdx.x; d < p.dim; d += 256) {
    const float q = ldf(row + p.q_col + h * p.dim + d) * p.scale, k = take * ldf(row + p.k_col + h * p.dim + d);
    sq[d] = q;
    sk[d] = k;
    nq += q * (fresh ? k : keep * nr[d] + k);
  }
  const float den = fmaxf(fabsf(block_sum(nq, red)), expf(-m)) + p.floor;     // (synchronises sq, sk)
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
  if (blockIdx.x == 0) {
    for (int d = threadIdx.x; d < p.dim; d += 256) nr[d] = fresh ? sk[d] : keep * nr[d] + sk[d];
    if (threadIdx.x == 0) p.peak[slot * p.H + h] = m;
  }
  const float inv = 1.f / sqrtf(ss / (float)p.rms_dim + p.eps);
#pragma unroll
  for (int i = 0; i < DC; ++i) {
    const int x = threadIdx.x + i * 256, c = h * p.vdim + c0 + x;
    if (x < width) stf(y + x, val[i] * inv * p.norm[c] * sigmoid_f(ldf(row + p.g_col + c)));
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
  const bool old = p.start[b] > 0 && slot >= 0;
  float S[NR], n[NR], m = old ? p.peak[slot * p.H + h] : 0.f;
  float* Sg = p.memory + (slot * p.H + h) * p.dim * p.vdim;
  float* ng = p.nrm + (slot * p.H + h) * p.dim;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = lane8 + 8 * i;
    const bool in = old && r < p.dim;
    S[i] = in && c < p.vdim ? Sg[(long long)r * p.vdim + c] : 0.f;
    n[i] = in ? ng[r] : 0.f;
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
      const float gi = sg[s][1], gf = sg[s][0];
      const float top = fmaxf(gf + m, gi), keep = expf(gf + m - top), take = expf(gi - top);
      m = top;
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
        o[((long long)(t0 + base + s) * p.H + h) * p.vdim + c] = acc / (fmaxf(fabsf(nq), expf(-m)) + p.floor);
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
    for (int i = 0; i < 4; ++i) f[i] *= inv * w[i] * sigmoid_f(g[i]);
    stf4(p.y + r * p.vdim + c, f);
  }
}

// ---- prompts in chunks (bf16) -------------------------------------------------------------------------------
using bf16 = __nv_bfloat16;
constexpr int C = 128, VW = 128, LDV = VW + 8, SB = 64, DBLK = 32;
constexpr int TERMS = 3;

struct Chunks {
  float* state;                          // [chunks, H, dim * vdim + dim]: U and its n part, then the state before the chunk
  float *top, *sum, *before;             // [chunks, H]: max a, sum of f, m before the chunk
  float *a, *run, *b;                    // [H, tokens]: a, running max of a, sum of f inside the chunk
  float* o;                              // [tokens, H * vdim] when a head does not fit one block's columns
  int tokens;
};

__device__ __forceinline__ long long chunk_id(int t0, int b, int j) { return t0 / C + b + j; }

// x (two values of a fragment register) as TERMS bf16 registers whose sum is x to 24 bits
__device__ __forceinline__ void split(float x0, float x1, uint32_t (&r)[TERMS]) {
#pragma unroll
  for (int i = 0; i < TERMS; ++i) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(x0, x1);
    r[i] = *reinterpret_cast<const uint32_t*>(&v);
    const float2 f = __bfloat1622float2(v);
    x0 -= f.x;
    x1 -= f.y;
  }
}

// rows [row0, row0 + ROWS) of a section (`cols` wide, a multiple of 8) into shared memory; rows past `len` and columns
// [cols, fill) are zero
__device__ __forceinline__ void load_rows(bf16* dst, int ld, const bf16* src, long long src_ld, int rows, int row0, int len,
                                          int cols, int fill) {
  const int vecs = fill / 8;
  for (int i = threadIdx.x; i < rows * vecs; i += 256) {
    const int r = i / vecs, c = (i - r * vecs) * 8;
    const bool ok = row0 + r < len && c < cols;
    cp_async16(dst + r * ld + c, src + (long long)(ok ? row0 + r : 0) * src_ld + (ok ? c : 0), ok);
  }
}

// grid (chunks x column blocks, H, B)
__global__ void __launch_bounds__(256, 2) chunk_state_kernel(const Args<bf16> p, const Chunks ch) {
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float w[C];
  const int ldk = p.dim + 8, vblocks = (p.vdim + VW - 1) / VW;
  bf16* sK = reinterpret_cast<bf16*>(raw);
  bf16* sV = sK + C * ldk;
  const int j = blockIdx.x / vblocks, vb = blockIdx.x % vblocks, h = blockIdx.y, b = blockIdx.z;
  const int t0 = p.cu[b], len = min(p.cu[b + 1] - t0 - j * C, C);
  if (len <= 0) return;
  const long long first = t0 + j * C, id = chunk_id(t0, b, j) * p.H + h;
  const int width = min(VW, p.vdim - vb * VW);
  const bf16* rows = p.proj + first * p.ld;
  load_rows(sK, ldk, rows + p.k_col + h * p.dim, p.ld, C, 0, len, p.dim, p.dim);
  load_rows(sV, LDV, rows + p.v_col + h * p.vdim + vb * VW, p.ld, C, 0, len, width, width);
  cp_async_commit();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (warp == 0) {                       // gates of the chunk, four tokens per lane
    float a[4], run[4], bs[4], sum = 0.f;
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int s = lane * 4 + x;
      float gi = -INFINITY, gf = 0.f;
      if (s < len) log_gates(p, first + s, h, gi, gf);
      a[x] = gi;
      sum += gf;
      bs[x] = sum;
    }
    float before = sum;
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float o = __shfl_up_sync(0xffffffffu, before, d);
      if (lane >= d) before += o;
    }
    const float total = __shfl_sync(0xffffffffu, before, 31);
    before -= sum;
    float top = -INFINITY;
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      bs[x] += before;
      a[x] -= bs[x];
      top = fmaxf(top, a[x]);
      run[x] = top;
    }
    float peak = top;
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const float o = __shfl_up_sync(0xffffffffu, peak, d);
      if (lane >= d) peak = fmaxf(peak, o);
    }
    const float all = __shfl_sync(0xffffffffu, peak, 31);
    float left = __shfl_up_sync(0xffffffffu, peak, 1);
    if (lane == 0) left = -INFINITY;
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int s = lane * 4 + x;
      w[s] = expf(a[x] - all);
      if (vb == 0 && s < len) {
        const long long at = (long long)h * ch.tokens + first + s;
        ch.a[at] = a[x];
        ch.run[at] = fmaxf(run[x], left);
        ch.b[at] = bs[x];
      }
    }
    if (vb == 0 && lane == 0) {
      ch.top[id] = all;
      ch.sum[id] = total;
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  float* U = ch.state + id * ((long long)p.dim * p.vdim + p.dim);
  if (vb == 0) {
    for (int d = threadIdx.x; d < p.dim; d += 256) {
      float s = 0.f;
      for (int x = 0; x < len; ++x) s += w[x] * __bfloat162float(sK[x * ldk + d]);
      U[(long long)p.dim * p.vdim + d] = s;
    }
  }
  const int steps = (len + 15) / 16, ntile = width / 8;
  for (int mt = warp; mt < p.dim / 16; mt += 8) {
    float acc[VW / 8][4];
#pragma unroll
    for (int n = 0; n < VW / 8; ++n)
#pragma unroll
      for (int x = 0; x < 4; ++x) acc[n][x] = 0.f;
    for (int ks = 0; ks < steps; ++ks) {
      // K^T fragment: rows = key entries, columns = tokens
      uint32_t kf[4], at[TERMS][4];
      ldmatrix_x4_trans(kf, smem_u32(sK + (ks * 16 + (lane >> 4) * 8 + (lane & 7)) * ldk + mt * 16 + ((lane >> 3) & 1) * 8));
      const float2 wl = *reinterpret_cast<const float2*>(w + ks * 16 + (lane & 3) * 2);
      const float2 wh = *reinterpret_cast<const float2*>(w + ks * 16 + 8 + (lane & 3) * 2);
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&kf[r]));
        const float2 ww = r < 2 ? wl : wh;
        uint32_t t3[TERMS];
        split(f.x * ww.x, f.y * ww.y, t3);
#pragma unroll
        for (int i = 0; i < TERMS; ++i) at[i][r] = t3[i];
      }
#pragma unroll
      for (int n = 0; n < VW / 16; ++n) {
        if (n * 2 < ntile) {
          uint32_t vf[4];
          ldmatrix_x4_trans(vf, smem_u32(sV + (ks * 16 + (lane & 15)) * LDV + n * 16 + (lane >> 4) * 8));
#pragma unroll
          for (int i = 0; i < TERMS; ++i) {
            mma_16816(acc[2 * n], at[i], vf[0], vf[1]);
            mma_16816(acc[2 * n + 1], at[i], vf[2], vf[3]);
          }
        }
      }
    }
    const int d = mt * 16 + (lane >> 2);
#pragma unroll
    for (int n = 0; n < VW / 8; ++n) {
      if (n < ntile) {
        float* dst = U + (long long)d * p.vdim + vb * VW + n * 8 + (lane & 3) * 2;
        *reinterpret_cast<float2*>(dst) = make_float2(acc[n][0], acc[n][1]);
        *reinterpret_cast<float2*>(dst + 8ll * p.vdim) = make_float2(acc[n][2], acc[n][3]);
      }
    }
  }
}

__device__ __forceinline__ float4 blend(float x, const float4& a, float y, const float4& b) {
  return make_float4(x * a.x + y * b.x, x * a.y + y * b.y, x * a.z + y * b.z, x * a.w + y * b.w);
}

// grid (state elements / 1024, H, B): four elements per thread, chunk after chunk
__global__ void __launch_bounds__(256) carry_kernel(const Args<bf16> p, const Chunks ch) {
  constexpr int AHEAD = 8;
  const int h = blockIdx.y, b = blockIdx.z;
  const int t0 = p.cu[b], len = p.cu[b + 1] - t0, n = (len + C - 1) / C;
  const long long size = (long long)p.dim * p.vdim, e = ((long long)blockIdx.x * 256 + threadIdx.x) * 4;
  if (len <= 0 || e >= size + p.dim) return;
  const long long slot = p.slots[b], id0 = chunk_id(t0, b, 0) * p.H + h;
  const bool old = p.start[b] > 0 && slot >= 0;
  float* mine = e < size ? p.memory + (slot * p.H + h) * size + e : p.nrm + (slot * p.H + h) * p.dim + (e - size);
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  float m = 0.f;
  if (old) {
    s = *reinterpret_cast<const float4*>(mine);
    m = p.peak[slot * p.H + h];
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

// grid (chunks x column blocks, H, B); NT column tiles of 8 per block
template <int NT>
__global__ void __launch_bounds__(256, 2) chunk_out_kernel(const Args<bf16> p, const Chunks ch) {
  extern __shared__ __align__(16) unsigned char raw[];
  __shared__ float sa[C], sM[C], sInter[C], sExp[C], sDen[C];
  const int ld = p.dim + 8, vblocks = (p.vdim + VW - 1) / VW;
  bf16* sQ = reinterpret_cast<bf16*>(raw);
  float* sN = reinterpret_cast<float*>(sQ + C * ld);
  bf16* sK = reinterpret_cast<bf16*>(sN + p.dim);
  bf16* sV = sK + SB * ld;
  bf16* sS = sK;                         // terms of a state block: [TERMS][DBLK][LDV], before the keys and values
  const int j = blockIdx.x / vblocks, vb = blockIdx.x % vblocks, h = blockIdx.y, b = blockIdx.z;
  const int t0 = p.cu[b], len = min(p.cu[b + 1] - t0 - j * C, C);
  if (len <= 0) return;
  const long long first = t0 + j * C, id = chunk_id(t0, b, j) * p.H + h, size = (long long)p.dim * p.vdim;
  const bool inter = j > 0 || p.start[b] > 0;                     // a state before the chunk
  const int width = min(VW, p.vdim - vb * VW), ntile = width / 8;
  const bf16* rows = p.proj + first * p.ld;
  load_rows(sQ, ld, rows + p.q_col + h * p.dim, p.ld, C, 0, len, p.dim, p.dim);
  cp_async_commit();
  const float* S = ch.state + id * (size + p.dim);
  if (threadIdx.x < C) {
    const int s = threadIdx.x;
    const long long at = (long long)h * ch.tokens + first + s;
    const float m = ch.before[id], M = s < len ? fmaxf(m, ch.run[at]) : 0.f;
    sa[s] = s < len ? ch.a[at] : -INFINITY;
    sM[s] = M;
    sInter[s] = s < len ? expf(m - M) * p.scale : 0.f;
    sExp[s] = s < len ? expf(-(ch.b[at] + M)) : 0.f;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r0 = warp * 16;
  float acc[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int x = 0; x < 4; ++x) acc[n][x] = 0.f;
  if (inter) {
    for (int d = threadIdx.x; d < p.dim; d += 256) sN[d] = S[size + d];
    float4 x[DBLK * VW / 4 / 256];
    auto fetch = [&](int d0) {
#pragma unroll
      for (int i = 0; i < DBLK * VW / 4 / 256; ++i) {
        const int idx = i * 256 + threadIdx.x, r = idx / (VW / 4), c = idx % (VW / 4) * 4;
        x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (d0 + r < p.dim && c < width) x[i] = *reinterpret_cast<const float4*>(S + (long long)(d0 + r) * p.vdim + vb * VW + c);
      }
    };
    fetch(0);
    for (int d0 = 0; d0 < p.dim; d0 += DBLK) {
      __syncthreads();
#pragma unroll
      for (int i = 0; i < DBLK * VW / 4 / 256; ++i) {
        const int idx = i * 256 + threadIdx.x, r = idx / (VW / 4), c = idx % (VW / 4) * 4;
        uint32_t lo[TERMS], hi[TERMS];
        split(x[i].x, x[i].y, lo);
        split(x[i].z, x[i].w, hi);
#pragma unroll
        for (int k = 0; k < TERMS; ++k)
          *reinterpret_cast<uint2*>(sS + (k * DBLK + r) * LDV + c) = make_uint2(lo[k], hi[k]);
      }
      if (d0 + DBLK < p.dim) fetch(d0 + DBLK);
      if (d0 == 0) cp_async_wait<0>();
      __syncthreads();
#pragma unroll
      for (int kk = 0; kk < DBLK / 16; ++kk) {
        if (d0 + kk * 16 < p.dim && r0 < len) {
          uint32_t q[4];
          ldmatrix_x4(q, smem_u32(sQ + (r0 + (lane & 15)) * ld + d0 + kk * 16 + (lane >> 4) * 8));
#pragma unroll
          for (int n = 0; n < NT / 2; ++n) {
            if (n * 2 < ntile) {
#pragma unroll
              for (int k = 0; k < TERMS; ++k) {
                uint32_t f[4];
                ldmatrix_x4_trans(f, smem_u32(sS + (k * DBLK + kk * 16 + (lane & 15)) * LDV + n * 16 + (lane >> 4) * 8));
                mma_16816(acc[2 * n], q, f[0], f[1]);
                mma_16816(acc[2 * n + 1], q, f[2], f[3]);
              }
            }
          }
        }
      }
    }
    {
      // q . n of every row, two threads a row
      const int r = threadIdx.x >> 1;
      float s = 0.f;
      for (int d = (threadIdx.x & 1) * 2; d < p.dim; d += 4) {
        const float2 q = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sQ + r * ld + d));
        s += q.x * sN[d] + q.y * sN[d + 1];
      }
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      if ((threadIdx.x & 1) == 0) sDen[r] = s;
    }
    const float i0 = sInter[r0 + (lane >> 2)], i1 = sInter[r0 + (lane >> 2) + 8];
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      acc[n][0] *= i0;
      acc[n][1] *= i0;
      acc[n][2] *= i1;
      acc[n][3] *= i1;
    }
  }
  const int tr = r0 + (lane >> 2);       // this thread's rows: tr, tr + 8
  float rs[2] = {0.f, 0.f};
  for (int s0 = 0; s0 < len; s0 += SB) {
    __syncthreads();
    load_rows(sK, ld, rows + p.k_col + h * p.dim, p.ld, SB, s0, len, p.dim, p.dim);
    load_rows(sV, LDV, rows + p.v_col + h * p.vdim + vb * VW, p.ld, SB, s0, len, width, width);
    cp_async_commit();
    cp_async_wait<0>();
    __syncthreads();
    if (s0 > r0 + 15 || r0 >= len) continue;
    const int tiles = min((r0 + 15 - s0) / 16 + 1, SB / 16);      // 16-token tiles that some row of the warp sees
    float sc[SB / 8][4];
#pragma unroll
    for (int n = 0; n < SB / 8; ++n)
#pragma unroll
      for (int x = 0; x < 4; ++x) sc[n][x] = 0.f;
    for (int kk = 0; kk < p.dim / 16; ++kk) {
      uint32_t q[4];
      ldmatrix_x4(q, smem_u32(sQ + (r0 + (lane & 15)) * ld + kk * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int n = 0; n < SB / 16; ++n) {
        if (n < tiles) {
          uint32_t f[4];
          ldmatrix_x4(f, smem_u32(sK + (n * 16 + (lane & 7) + (lane >> 4) * 8) * ld + kk * 16 + ((lane >> 3) & 1) * 8));
          mma_16816(sc[2 * n], q, f[0], f[1]);
          mma_16816(sc[2 * n + 1], q, f[2], f[3]);
        }
      }
    }
#pragma unroll
    for (int n = 0; n < SB / 16; ++n) {
      if (n < tiles) {
        uint32_t at[TERMS][4];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
#pragma unroll
          for (int x = 0; x < 4; ++x) {
            const int s = s0 + (2 * n + u) * 8 + (lane & 3) * 2 + (x & 1), t = tr + (x >> 1) * 8;
            const float v = s <= t ? sc[2 * n + u][x] * p.scale * expf(sa[s] - sM[t]) : 0.f;
            sc[2 * n + u][x] = v;
            rs[x >> 1] += v;
          }
        }
        // accumulator pairs -> A fragment registers (rows lane / 4 and + 8, columns 2 (lane % 4) and + 8)
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          uint32_t t3[TERMS];
          split(sc[2 * n + (r >> 1)][(r & 1) * 2], sc[2 * n + (r >> 1)][(r & 1) * 2 + 1], t3);
#pragma unroll
          for (int k = 0; k < TERMS; ++k) at[k][r] = t3[k];
        }
#pragma unroll
        for (int c = 0; c < NT / 2; ++c) {
          if (c * 2 < ntile) {
            uint32_t f[4];
            ldmatrix_x4_trans(f, smem_u32(sV + (n * 16 + (lane & 15)) * LDV + c * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int k = 0; k < TERMS; ++k) {
              mma_16816(acc[2 * c], at[k], f[0], f[1]);
              mma_16816(acc[2 * c + 1], at[k], f[2], f[3]);
            }
          }
        }
      }
    }
  }
  if (r0 >= len) return;                 // no barrier follows
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int t = tr + r * 8;
    float den = rs[r] + __shfl_xor_sync(0xffffffffu, rs[r], 1);
    den += __shfl_xor_sync(0xffffffffu, den, 2);
    if (inter) den += sInter[t] * sDen[t];
    const float inv = 1.f / (fmaxf(fabsf(den), sExp[t]) + p.floor);
    float ss = 0.f;
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      acc[n][2 * r] *= inv;
      acc[n][2 * r + 1] *= inv;
      ss += acc[n][2 * r] * acc[n][2 * r] + acc[n][2 * r + 1] * acc[n][2 * r + 1];
    }
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    ss += __shfl_xor_sync(0xffffffffu, ss, 2);
    if (t >= len) continue;
    const int c0 = h * p.vdim + vb * VW + (lane & 3) * 2;
    if (vblocks > 1) {
      float* o = ch.o + (first + t) * p.H * p.vdim + c0;
#pragma unroll
      for (int n = 0; n < NT; ++n)
        if (n < ntile) *reinterpret_cast<float2*>(o + n * 8) = make_float2(acc[n][2 * r], acc[n][2 * r + 1]);
      continue;
    }
    const float nr = 1.f / sqrtf(ss / (float)p.rms_dim + p.eps);
    const bf16* g = p.proj + (first + t) * p.ld + p.g_col + c0;
    bf16* y = p.y + (first + t) * p.H * p.vdim + c0;
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      if (n < ntile) {
        const float2 gg = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(g + n * 8));
        const float2 w = *reinterpret_cast<const float2*>(p.norm + c0 + n * 8);
        *reinterpret_cast<__nv_bfloat162*>(y + n * 8) =
            __floats2bfloat162_rn(acc[n][2 * r] * nr * w.x * sigmoid_f(gg.x), acc[n][2 * r + 1] * nr * w.y * sigmoid_f(gg.y));
      }
    }
  }
}

template <typename T>
Args<T> make_args(const void* proj, long long ld, const float* z, long long z_ld, const int* ints, const float* floats,
                  const float* bias, const float* norm, float* memory, float* nrm, float* peak, const int* cu,
                  const int* start, const long long* slots, void* y) {
  return Args<T>{(const T*)proj, ld, z, z_ld, ints[0], ints[1], ints[2], ints[3], ints[4], ints[5], ints[6], ints[7],
                 floats[0], floats[1], floats[2], floats[3], bias, norm, memory, nrm, peak, cu, start, slots, (T*)y};
}

}  // namespace mem
}  // namespace msrl

using namespace msrl;

// ints: H, dim, vdim (multiples of 16), entries of a head that count in its root mean square, columns of q, k, v, gate;
// floats: scale, cap, floor, eps
MSRL_API int msrl_memory_decode(const void* proj, long long ld, const float* z, long long z_ld, const int* ints,
                                const float* floats, const float* bias, const float* norm, float* memory, float* nrm,
                                float* peak, const int* positions, const long long* slots, void* y, int batch, int is_f32,
                                cudaStream_t st) {
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
    const auto p = mem::make_args<T>(proj, ld, z, z_ld, ints, floats, bias, norm, memory, nrm, peak, nullptr, positions,
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
                                 const float* floats, const float* bias, const float* norm, float* memory, float* nrm,
                                 float* peak, const int* cu, const int* start, const long long* slots, float* o, void* y,
                                 int tokens, int batch, int is_f32, cudaStream_t st) {
  if (batch == 0 || tokens == 0) return 0;
  const int H = ints[0], dim = ints[1], vdim = ints[2];
  if (dim > 512 || dim % 16 != 0 || vdim % 16 != 0 || batch > 65535 || H > 65535) return (int)cudaErrorNotSupported;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const auto p = mem::make_args<T>(proj, ld, z, z_ld, ints, floats, bias, norm, memory, nrm, peak, cu, start, slots, y);
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
    mem::scan_norm_kernel<T><<<dim3((unsigned)H, (unsigned)batch), 256, 0, st>>>(p);
    const long long rows = (long long)tokens * H;
    mem::finish_kernel<T><<<(unsigned)((rows + 7) / 8), 256, 0, st>>>(p, o, rows);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

static size_t memory_out_smem(int dim) {
  const size_t kv = (size_t)mem::SB * (dim + 8) + (size_t)mem::SB * mem::LDV, s = (size_t)mem::TERMS * mem::DBLK * mem::LDV;
  return ((size_t)mem::C * (dim + 8) + (kv > s ? kv : s)) * 2 + dim * 4;
}

MSRL_API int msrl_memory_chunked_serves(const int* ints) { return ints[1] <= 256 && ints[1] % 16 == 0 && ints[2] % 16 == 0; }

// floats
MSRL_API long long msrl_memory_chunk_scratch(const int* ints, int tokens, int batch) {
  const long long H = ints[0], dim = ints[1], vdim = ints[2], chunks = tokens / mem::C + batch;
  return chunks * H * (dim * vdim + dim + 4) + 3 * H * tokens + 16 + (vdim > mem::VW ? (long long)tokens * H * vdim : 0);
}

// The same for bf16 rows, in chunks; column starts and ld are multiples of 8
MSRL_API int msrl_memory_prefill_chunked(const void* proj, long long ld, const float* z, long long z_ld, const int* ints,
                                         const float* floats, const float* bias, const float* norm, float* memory,
                                         float* nrm, float* peak, const int* cu, const int* start, const long long* slots,
                                         float* scratch, void* y, int tokens, int batch, int max_q, cudaStream_t st) {
  if (batch == 0 || tokens == 0) return 0;
  const int H = ints[0], dim = ints[1], vdim = ints[2];
  if (!msrl_memory_chunked_serves(ints) || ld % 8 != 0 || batch > 65535 || H > 65535) return (int)cudaErrorNotSupported;
  for (int i = 4; i < 8; ++i)
    if (ints[i] % 8 != 0) return (int)cudaErrorNotSupported;
  const auto p = mem::make_args<__nv_bfloat16>(proj, ld, z, z_ld, ints, floats, bias, norm, memory, nrm, peak, cu, start,
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
  const int vblocks = (vdim + mem::VW - 1) / mem::VW, most = (max_q + mem::C - 1) / mem::C;
  const dim3 grid((unsigned)(most * vblocks), (unsigned)H, (unsigned)batch);
  const int smem_state = (mem::C * (dim + 8) + mem::C * mem::LDV) * 2, smem_out = (int)memory_out_smem(dim);
  cudaError_t e = cudaFuncSetAttribute(mem::chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_state);
  if (e != cudaSuccess) return (int)e;
  mem::chunk_state_kernel<<<grid, 256, smem_state, st>>>(p, ch);
  mem::carry_kernel<<<dim3((unsigned)((size + 1023) / 1024), (unsigned)H, (unsigned)batch), 256, 0, st>>>(p, ch);
  mem::carry_peak_kernel<<<(unsigned)(((long long)batch * H + 127) / 128), 128, 0, st>>>(p, ch, batch);
  auto go = [&](auto kernel) {
    e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem_out);
    if (e != cudaSuccess) return (int)e;
    kernel<<<grid, 256, smem_out, st>>>(p, ch);
    return (int)cudaGetLastError();
  };
  const int rc = vdim <= 64 ? go(mem::chunk_out_kernel<8>) : go(mem::chunk_out_kernel<16>);
  if (rc != 0 || vblocks == 1) return rc;
  const long long rows = (long long)tokens * H;
  mem::finish_kernel<__nv_bfloat16><<<(unsigned)((rows + 7) / 8), 256, 0, st>>>(p, ch.o, rows);
  return (int)cudaGetLastError();
}
