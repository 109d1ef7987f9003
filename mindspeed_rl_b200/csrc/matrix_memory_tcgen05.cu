// Chunked matrix memory on the 5th-generation tensor cores (tcgen05 + TMEM); see matrix_memory.cu for the equations.
//
// One CTA takes one chunk of 128 tokens, one head and up to 128 value columns:
//
//   chunk_state   U [dim, columns] = (w K)^T V: the gates of the chunk are summed and maximised by one warp, the keys times
//                 their weights go to shared memory as MN-major A operand, 32 tokens at a time, V is the MN-major B
//                 operand
//   chunk_out     S = Q K^T;  O1 = Q S0, the state before the chunk going through shared memory 32 rows at a time;
//                 P = S with the weights, as K-major A operand over the dead Q and K;  O2 = P V into the columns of S;
//                 y = (weight O1 + O2) / denominator, normed and gated
//
// 32-bit operands (weighted keys, P, the state) are taken apart into three bf16 terms of 24 bits together, one product
// each; the other operand is exact and sums are fp32.  Two or three CTAs share an SM (dim <= 128), so that the copies and
// conversions of one run beside the products of the other  All tiles are 128-byte-swizzled.
//
// Every mbarrier wait is bounded; on expiry the kernel records a code in the status word, skips the rest, frees
// TMEM and returns.
#include <cuda.h>

#include "matrix_memory.cuh"
#include "mma_utils.cuh"
#include "tcgen05_utils.cuh"

namespace msrl {
namespace mem {

using namespace t5;
using bf16 = __nv_bfloat16;

constexpr int VW = 128;                  // value columns of a CTA
constexpr int TERMS = 3, TB = 32;        // bf16 terms of a 32-bit operand; tokens or state rows per converted block
constexpr uint32_t HALF = C * 128;       // [128 rows x 64 columns] bf16
constexpr uint32_t BLK = TB * 128;       // [32 rows x 64 columns]
constexpr float LOG2E = 1.4426950408889634f;
constexpr int PITCH = 36;                // floats per row of a warp's [32 x 32] staging patch

enum { ERR_A = 80, ERR_DONE = 81, ERR_S = 82, ERR_Q = 83, ERR_PV = 84 };

constexpr uint32_t idesc_both_mn(int m) { return idesc_bf16(m, 0, true) | (1u << 15); }
__device__ __forceinline__ uint32_t with_n(uint32_t idesc, int n) { return idesc | ((uint32_t)(n >> 3) << 17); }

__device__ __forceinline__ void proxy_fence() { asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory"); }
__device__ __forceinline__ unsigned char* align1k(unsigned char* p) {
  return reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(p) + 1023) & ~static_cast<uintptr_t>(1023));
}
// byte offset of 16-byte piece c (of 8) of row r inside a [rows x 64 columns] swizzled tile
__device__ __forceinline__ uint32_t piece(int r, int c) { return (r >> 3) * 1024 + (r & 7) * 128 + ((c ^ (r & 7)) << 4); }

// 128 rows of a section (`cols` wide) into swizzled halves; rows past `len` are zero
__device__ __forceinline__ void load_tile(unsigned char* dst, const bf16* src, long long ld, int len, int cols) {
  const int vecs = cols / 8;
  if (vecs == 16) {                      // 128 columns: a thread keeps its column piece
    const int c = threadIdx.x & 15, r0 = threadIdx.x >> 4;
    unsigned char* to = dst + (c >> 3) * HALF + piece(r0, c & 7);  // 16 rows on: the same place two row groups later
    const bf16* from = src + (long long)r0 * ld + c * 8;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const bool ok = r0 + i * 16 < len;
      cp_async16(to + i * 2048, ok ? from + (long long)(i * 16) * ld : src, ok);
    }
    return;
  }
  for (int i = threadIdx.x; i < C * vecs; i += 256) {
    const int r = i / vecs, c = i - r * vecs;
    const bool ok = r < len;
    cp_async16(dst + (c >> 3) * HALF + piece(r, c & 7), src + (long long)(ok ? r : 0) * ld + c * 8, ok);
  }
}

// the leading bf16 of eight values as one vector; the values keep what is left
__device__ __forceinline__ bf16x8 take_term(float* v) {
  bf16x8 out;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    out.v[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    const float2 f = __bfloat1622float2(out.v[i]);
    v[2 * i] -= f.x;
    v[2 * i + 1] -= f.y;
  }
  return out;
}

__device__ __forceinline__ void alloc_tmem(uint32_t* slot, uint32_t columns) {
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(smem_u32(slot)), "r"(columns));
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::);
}
__device__ __forceinline__ void free_tmem(uint32_t tmem, uint32_t columns) {
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(columns));
}

__host__ __device__ inline int key_halves(int dim) { return (dim + 63) / 64; }
__host__ __device__ inline uint32_t state_smem(int dim) {
  const uint32_t terms = TERMS * (dim > 128 ? 4u : 2u) * BLK, patches = 8u * 32 * PITCH * 4;
  return 2u * HALF + (terms > patches ? terms : patches);
}
__host__ __device__ inline uint32_t out_keys_bytes(int dim) {      // Q and K, later P
  const uint32_t b = 2u * key_halves(dim) * HALF;
  return b > 4u * HALF ? b : 4u * HALF;
}

// MB 128-row blocks of keys (dim <= 128 MB).  grid (chunks x column blocks, H, B)
template <int MB>
__global__ void __launch_bounds__(256, MB == 1 ? 3 : 2) chunk_state_kernel(const Args<bf16> p, const Chunks ch, int* error) {
  extern __shared__ unsigned char raw[];
  __shared__ float w[C], gate_f[C];
  __shared__ uint64_t used, done;
  __shared__ uint32_t tmem_slot;
  constexpr uint32_t TMEM = 128 * MB, term_bytes = MB * 2 * BLK;
  const int vblocks = (p.vdim + VW - 1) / VW;
  const int j = blockIdx.x / vblocks, vb = blockIdx.x % vblocks, h = blockIdx.y, b = blockIdx.z;
  const int t0 = p.cu[b], len = min(p.cu[b + 1] - t0 - j * C, C);
  if (len <= 0) return;                  // uniform for the CTA, before any allocation
  unsigned char* sV = align1k(raw);
  unsigned char* sA = sV + 2 * HALF;
  const long long first = t0 + j * C, id = chunk_id(t0, b, j) * p.H + h;
  const int width = min(VW, p.vdim - vb * VW);
  const bf16* rows = p.proj + first * p.ld;
  load_tile(sV, rows + p.v_col + h * p.vdim + vb * VW, p.ld, len, width);
  cp_async_commit();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  // keys: a thread keeps its eight entries and takes rows `kr`, `kr` + lanes, ... of a block
  const int vecs = p.dim / 8, lanes = 256 / vecs, kc = threadIdx.x % vecs, kr = threadIdx.x / vecs;
  const bf16* keys = rows + p.k_col + h * p.dim + kc * 8;
  constexpr int ROWS = 2 * MB;           // rows of a thread in a block: 32 / lanes, at most 2 MB
  bf16x8 next[ROWS];
  auto fetch = [&](int blk) {
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int r = kr + i * lanes;
      if (kr < lanes && r < TB && blk * TB + r < len) next[i] = ld8(keys + (long long)(blk * TB + r) * p.ld);
    }
  };
  fetch(0);
  if (threadIdx.x == 32) {
    mbar_init(&used, 1);
    mbar_init(&done, 1);
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  __syncwarp();
  if (warp == 1) alloc_tmem(&tmem_slot, TMEM);
  if (threadIdx.x < C) {                 // log gates, one token per thread
    float gi = -INFINITY, gf = 0.f;
    if (threadIdx.x < len) log_gates(p, first + threadIdx.x, h, gi, gf);
    w[threadIdx.x] = gi;
    gate_f[threadIdx.x] = gf;
    asm volatile("bar.sync 1, 128;\n" ::: "memory");
  }
  if (warp == 0) {                       // sums and maxima over the chunk, four tokens per lane
    float a[4], run[4], bs[4], sum = 0.f;
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      a[x] = w[lane * 4 + x];
      sum += gate_f[lane * 4 + x];
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
  float nsum[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  cp_async_wait<0>();
  fence_before();
  __syncthreads();
  fence_after();
  const uint32_t tmem = tmem_slot;
  const int blocks = (len + TB - 1) / TB;
  bool ok = true;
  for (int blk = 0; blk < blocks; ++blk) {
    if (blk > 0) ok = mbar_wait_warp(&used, (blk - 1) & 1, error, ERR_A);
#pragma unroll
    for (int i = 0; i < ROWS; ++i) {
      const int r = kr + i * lanes, s = blk * TB + r;
      if (ok && kr < lanes && r < TB) {
        float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
        if (s < len) {
          unpack8(next[i], f);
#pragma unroll
          for (int x = 0; x < 8; ++x) {
            f[x] *= w[s];
            nsum[x] += f[x];
          }
        }
        unsigned char* to = sA + (kc >> 3) * BLK + piece(r, kc & 7);
#pragma unroll
        for (int k = 0; k < TERMS; ++k) *reinterpret_cast<bf16x8*>(to + k * term_bytes) = take_term(f);
      }
    }
    if (blk + 1 < blocks) fetch(blk + 1);
    proxy_fence();
    ok = __syncthreads_and(ok);
    if (!ok) break;
    if (warp == 0 && elect_one()) {
      fence_after();
      const uint32_t id_u = with_n(idesc_both_mn(128), width);
      const uint32_t a0 = smem_u32(sA), v0 = smem_u32(sV) + blk * BLK;
#pragma unroll
      for (int mb = 0; mb < MB; ++mb)
#pragma unroll
        for (int k = 0; k < TERMS; ++k)
#pragma unroll
          for (int kk = 0; kk < TB / 16; ++kk)
            umma(tmem + mb * 128, desc_sw128(a0 + k * term_bytes + mb * 2 * BLK + kk * 2048, BLK, 1024),
                 desc_sw128(v0 + kk * 2048, HALF, 1024), id_u, (blk > 0 || k > 0 || kk > 0) ? 1u : 0u);
      commit(&used);
      if (blk + 1 == blocks) commit(&done);
    }
    __syncwarp();
  }
  if (ok) ok = mbar_wait_warp(&done, 0, error, ERR_DONE);
  ok = __syncthreads_and(ok);
  if (ok) {
    fence_after();
    const long long size = (long long)p.dim * p.vdim;
    float* U = ch.state + id * (size + p.dim);
    const int quarter = warp & 3, wg = warp >> 2;
    float* patch = reinterpret_cast<float*>(sA) + warp * 32 * PITCH;
    for (int mb = 0; mb < MB; ++mb) {
      const int d0 = mb * 128 + quarter * 32;
      for (int c0 = wg * 64; c0 < min(wg * 64 + 64, width); c0 += 32) {
        float v[32];
        tmem_ld32(tmem + ((uint32_t)(quarter * 32) << 16) + mb * 128 + c0, v);
#pragma unroll
        for (int i = 0; i < 8; ++i)
          *reinterpret_cast<float4*>(patch + lane * PITCH + i * 4) = make_float4(v[i * 4], v[i * 4 + 1], v[i * 4 + 2], v[i * 4 + 3]);
        __syncwarp();
#pragma unroll
        for (int it = 0; it < 8; ++it) {
          const int r = it * 4 + (lane >> 3), c = c0 + (lane & 7) * 4;
          if (d0 + r < p.dim && c < width)
            *reinterpret_cast<float4*>(U + (long long)(d0 + r) * p.vdim + vb * VW + c) =
                *reinterpret_cast<const float4*>(patch + r * PITCH + (lane & 7) * 4);
        }
        __syncwarp();
      }
    }
    if (vb == 0) {                       // sum of the weighted keys, over the lanes that share entries
      float* red = reinterpret_cast<float*>(sV);
      if (kr < lanes)
#pragma unroll
        for (int x = 0; x < 8; ++x) red[kr * p.dim + kc * 8 + x] = nsum[x];
      __syncthreads();
      for (int d = threadIdx.x; d < p.dim; d += 256) {
        float s = 0.f;
        for (int l = 0; l < lanes; ++l) s += red[l * p.dim + d];
        U[size + d] = s;
      }
    }
  }
  fence_before();
  __syncthreads();
  if (warp == 1) free_tmem(tmem, TMEM);
}

// grid (chunks x column blocks, H, B)
__global__ void __launch_bounds__(256, 2) chunk_out_kernel(const Args<bf16> p, const Chunks ch, int* error) {
  extern __shared__ unsigned char raw[];
  __shared__ float sa[C], sM[C], sInter[C], sExp[C], sDen[C], part[2][C];
  __shared__ uint64_t s_full, q_done, pv_done;
  __shared__ uint32_t tmem_slot;
  constexpr uint32_t TMEM = 256;
  const int vblocks = (p.vdim + VW - 1) / VW;
  const int j = blockIdx.x / vblocks, vb = blockIdx.x % vblocks, h = blockIdx.y, b = blockIdx.z;
  const int t0 = p.cu[b], len = min(p.cu[b + 1] - t0 - j * C, C);
  if (len <= 0) return;                  // uniform for the CTA, before any allocation
  const int nq = key_halves(p.dim);
  unsigned char* sQ = align1k(raw);
  unsigned char* sK = sQ + nq * HALF;
  unsigned char* sY = sQ + out_keys_bytes(p.dim);                 // state terms, then V
  unsigned char* sP = sQ;                                         // [half of the tokens][term], over Q and K
  float* sN = reinterpret_cast<float*>(sY + 2 * HALF);
  const long long first = t0 + j * C, id = chunk_id(t0, b, j) * p.H + h, size = (long long)p.dim * p.vdim;
  const bool inter = j > 0 || p.start[b] > 0;                     // a state before the chunk
  const int width = min(VW, p.vdim - vb * VW);
  const bf16* rows = p.proj + first * p.ld;
  load_tile(sQ, rows + p.q_col + h * p.dim, p.ld, len, p.dim);
  load_tile(sK, rows + p.k_col + h * p.dim, p.ld, len, p.dim);
  cp_async_commit();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(&s_full, 1);
    mbar_init(&q_done, 1);
    mbar_init(&pv_done, 1);
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  if (warp == 1) alloc_tmem(&tmem_slot, TMEM);
  const float* S = ch.state + id * (size + p.dim);
  float4 x[TB * VW / 4 / 256];
  auto fetch = [&](int d0) {
#pragma unroll
    for (int i = 0; i < TB * VW / 4 / 256; ++i) {
      const int idx = i * 256 + threadIdx.x, r = idx / (VW / 4), c = idx % (VW / 4) * 4;
      x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (d0 + r < p.dim && c < width) x[i] = *reinterpret_cast<const float4*>(S + (long long)(d0 + r) * p.vdim + vb * VW + c);
    }
  };
  if (inter) {
    fetch(0);
    if (p.decay == nullptr)
      for (int d = threadIdx.x; d < p.dim; d += 256) sN[d] = S[size + d];
  }
  if (threadIdx.x < C) {
    const int s = threadIdx.x;
    const long long at = (long long)h * ch.tokens + first + s;
    const float m = ch.before[id], M = s < len ? fmaxf(m, ch.run[at]) : 0.f;
    sa[s] = s < len ? ch.a[at] * LOG2E : -INFINITY;
    sM[s] = M * LOG2E;
    sInter[s] = s < len ? expf(m - M) * p.scale : 0.f;
    sExp[s] = s < len ? expf(-(ch.b[at] + M)) : 0.f;
  }
  cp_async_wait<0>();
  proxy_fence();
  fence_before();
  __syncthreads();
  fence_after();
  const uint32_t tmem = tmem_slot, tmem_o1 = tmem + 128;
  const uint32_t q_addr = smem_u32(sQ), k_addr = smem_u32(sK), y_addr = smem_u32(sY), p_addr = smem_u32(sP);
  if (warp == 0 && elect_one()) {
    constexpr uint32_t id_s = idesc_bf16(128, 128, false);
    for (int kk = 0; kk < p.dim / 16; ++kk)
      umma(tmem, desc_sw128(q_addr + (kk >> 2) * HALF + (kk & 3) * 32, 16, 1024),
           desc_sw128(k_addr + (kk >> 2) * HALF + (kk & 3) * 32, 16, 1024), id_s, kk > 0 ? 1u : 0u);
    commit(&s_full);
  }
  __syncwarp();
  bool ok = true;
  if (inter) {
    const uint32_t id_q = with_n(idesc_bf16(128, 0, true), width);
    for (int d0 = 0; d0 < p.dim; d0 += TB) {
      if (d0 > 0) ok = mbar_wait_warp(&q_done, (d0 / TB - 1) & 1, error, ERR_Q);
#pragma unroll
      for (int i = 0; i < TB * VW / 4 / 256; ++i) {
        const int idx = i * 256 + threadIdx.x, r = idx / (VW / 4), c = idx % (VW / 4) * 4;
        unsigned char* dst = sY + (c >> 6) * BLK + piece(r, (c & 63) >> 3) + (c & 7) * 2;
        float v[4] = {x[i].x, x[i].y, x[i].z, x[i].w};
#pragma unroll
        for (int k = 0; k < TERMS; ++k) {
          __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
          const float2 fl = __bfloat1622float2(lo), fh = __bfloat1622float2(hi);
          v[0] -= fl.x;
          v[1] -= fl.y;
          v[2] -= fh.x;
          v[3] -= fh.y;
          *reinterpret_cast<uint2*>(dst + k * 2 * BLK) =
              make_uint2(*reinterpret_cast<uint32_t*>(&lo), *reinterpret_cast<uint32_t*>(&hi));
        }
      }
      if (d0 + TB < p.dim) fetch(d0 + TB);
      proxy_fence();
      ok = __syncthreads_and(ok);
      if (!ok) break;
      if (warp == 0 && elect_one()) {
        fence_after();
        const int steps = min(TB, p.dim - d0) / 16;
        for (int k = 0; k < TERMS; ++k)
          for (int s = 0; s < steps; ++s) {
            const int kk = d0 / 16 + s;
            umma(tmem_o1, desc_sw128(q_addr + (kk >> 2) * HALF + (kk & 3) * 32, 16, 1024),
                 desc_sw128(y_addr + k * 2 * BLK + s * 2048, BLK, 1024), id_q, (d0 > 0 || k > 0 || s > 0) ? 1u : 0u);
          }
        commit(&q_done);
      }
      __syncwarp();
    }
    if (ok && p.decay == nullptr) {
      // q . n of every row, two threads a row
      const int r = threadIdx.x >> 1;
      float s = 0.f;
      for (int c = threadIdx.x & 1; c < p.dim / 8; c += 2) {
        float q[8];
        unpack8(*reinterpret_cast<const bf16x8*>(sQ + (c >> 3) * HALF + piece(r, c & 7)), q);
#pragma unroll
        for (int i = 0; i < 8; ++i) s += q[i] * sN[c * 8 + i];
      }
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      if ((threadIdx.x & 1) == 0) sDen[r] = s;
    }
    if (ok) ok = mbar_wait_warp(&q_done, ((p.dim + TB - 1) / TB - 1) & 1, error, ERR_Q);
  }
  ok = ok && mbar_wait_warp(&s_full, 0, error, ERR_S);
  ok = __syncthreads_and(ok);            // Q, K and the state terms are read, sDen is written
  const int quarter = warp & 3, wg = warp >> 2, row = quarter * 32 + lane;
  const uint32_t lane_base = (uint32_t)(quarter * 32) << 16;
  const bool late = len > C / 2;         // tokens in the second half
  if (ok) {
    load_tile(sY, rows + p.v_col + h * p.vdim + vb * VW, p.ld, len, width);
    cp_async_commit();
    fence_after();
    // P: the thread's row against one half of the tokens
    float v[64];
    float sum = 0.f;
    const bool some = wg == 0 || (late && quarter >= 2);
    if (some) {
      const float M = sM[row];
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        float t[32];
        const int s0 = wg * 64 + c * 32;
        if (s0 > quarter * 32 + 31) {    // past the diagonal for all rows of the warp
#pragma unroll
          for (int i = 0; i < 32; ++i) v[c * 32 + i] = 0.f;
          continue;
        }
        tmem_ld32(tmem + lane_base + s0, t);
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          float e = t[i] * p.scale * exp2f(fminf(sa[s0 + i] - M, 0.f));       // at most 0 up to the diagonal
          e = s0 + i <= row ? e : 0.f;
          v[c * 32 + i] = e;
          sum += e;
        }
      }
    } else {
#pragma unroll
      for (int i = 0; i < 64; ++i) v[i] = 0.f;
    }
    part[wg][row] = sum;
    auto write_term = [&](unsigned char* tile) {
#pragma unroll
      for (int c = 0; c < 8; ++c) *reinterpret_cast<bf16x8*>(tile + piece(row, c)) = take_term(v + c * 8);
    };
    // first half of the tokens: tiles 0 .. 2; second half: its leading term in tile 3, the others later in 0 and 1
    if (wg == 0) {
#pragma unroll 1
      for (int k = 0; k < TERMS; ++k) write_term(sP + k * HALF);
    } else if (late) {
      write_term(sP + TERMS * HALF);
    }
    cp_async_wait<0>();
    proxy_fence();
    fence_before();
    __syncthreads();
    const uint32_t id_p = with_n(idesc_bf16(128, 0, true), width);
    auto product = [&](uint32_t tile, int half, bool start) {
#pragma unroll
      for (int kk = 0; kk < 4; ++kk)
        umma(tmem, desc_sw128(tile + kk * 32, 16, 1024), desc_sw128(y_addr + half * (HALF / 2) + kk * 2048, HALF, 1024), id_p,
             (start && kk == 0) ? 0u : 1u);
    };
    if (warp == 0 && elect_one()) {
      fence_after();
      for (int k = 0; k < TERMS; ++k) product(p_addr + k * HALF, 0, k == 0);
      if (late) product(p_addr + TERMS * HALF, 1, false);
      commit(&pv_done);
    }
    __syncwarp();
    ok = mbar_wait_warp(&pv_done, 0, error, ERR_PV);
    ok = __syncthreads_and(ok);
    if (ok && late) {
      if (wg == 1) {
#pragma unroll 1
        for (int k = 0; k < TERMS - 1; ++k) write_term(sP + k * HALF);
      }
      proxy_fence();
      __syncthreads();
      if (warp == 0 && elect_one()) {
        fence_after();
        for (int k = 0; k < TERMS - 1; ++k) product(p_addr + k * HALF, 1, false);
        commit(&pv_done);
      }
      __syncwarp();
      ok = mbar_wait_warp(&pv_done, 1, error, ERR_PV);
      ok = __syncthreads_and(ok);
    }
  }
  if (ok) {
    fence_after();
    const float weight = sInter[row];
    float inv = 1.f;
    if (p.decay == nullptr) {
      float den = part[0][row] + part[1][row];
      if (inter) den += weight * sDen[row];
      inv = 1.f / (fmaxf(fabsf(den), sExp[row]) + p.floor);
    }
    float o[2][32], ss = 0.f;            // the thread's row, its half of the columns
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      const int c0 = wg * 64 + c * 32;
      if (c0 < width) {
        tmem_ld32(tmem + lane_base + c0, o[c]);
        if (inter) {
          float u[32];
          tmem_ld32(tmem_o1 + lane_base + c0, u);
#pragma unroll
          for (int i = 0; i < 32; ++i) o[c][i] += weight * u[i];
        }
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          o[c][i] *= inv;
          ss += c0 + i < width ? o[c][i] * o[c][i] : 0.f;
        }
      }
    }
    float scale = 1.f;
    if (vblocks == 1) {
      __syncthreads();                   // every thread has read its denominators
      part[wg][row] = ss;
      __syncthreads();
      scale = 1.f / sqrtf((part[0][row] + part[1][row]) / (float)p.rms_dim + p.eps);
    }
    float* patch = reinterpret_cast<float*>(sQ) + warp * 32 * PITCH;
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      const int c0 = wg * 64 + x * 32;
      if (c0 >= width) break;
#pragma unroll
      for (int i = 0; i < 8; ++i)
        *reinterpret_cast<float4*>(patch + lane * PITCH + i * 4) =
            make_float4(o[x][i * 4] * scale, o[x][i * 4 + 1] * scale, o[x][i * 4 + 2] * scale, o[x][i * 4 + 3] * scale);
      __syncwarp();
      const int c = c0 + (lane & 7) * 4, col = h * p.vdim + vb * VW + c;
      float wn[4] = {0.f, 0.f, 0.f, 0.f};
      uint2 gate[8];                     // all loads before the first store
      if (vblocks == 1 && c < width) {
        ldf4(p.norm + col, wn);
#pragma unroll
        for (int it = 0; it < 8; ++it) {
          const int t = min(quarter * 32 + it * 4 + (lane >> 3), len - 1);
          gate[it] = *reinterpret_cast<const uint2*>(p.proj + (first + t) * p.ld + p.g_col + col);
        }
      }
#pragma unroll
      for (int it = 0; it < 8; ++it) {
        const int r = it * 4 + (lane >> 3), t = quarter * 32 + r;
        if (t < len && c < width) {
          const float4 f = *reinterpret_cast<const float4*>(patch + r * PITCH + (lane & 7) * 4);
          const long long at = (first + t) * p.H * p.vdim + col;
          if (vblocks > 1) {
            *reinterpret_cast<float4*>(ch.o + at) = f;
          } else {
            const float2 g0 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gate[it].x));
            const float2 g1 = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&gate[it].y));
            const float y[4] = {f.x * wn[0] * out_gate(p, g0.x, sigmoid_t<bf16>(g0.x)),
                                f.y * wn[1] * out_gate(p, g0.y, sigmoid_t<bf16>(g0.y)),
                                f.z * wn[2] * out_gate(p, g1.x, sigmoid_t<bf16>(g1.x)),
                                f.w * wn[3] * out_gate(p, g1.y, sigmoid_t<bf16>(g1.y))};
            stf4(p.y + at, y);
          }
        }
      }
      __syncwarp();
    }
  }
  fence_before();
  __syncthreads();
  if (warp == 1) free_tmem(tmem, TMEM);
}

static int set_smem(const void* kernel, int bytes) {
  return (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
}

int launch_chunk_state(const Args<bf16>& p, const Chunks& ch, int most, int batch, int* error, cudaStream_t st) {
  auto* kernel = p.dim > 128 ? chunk_state_kernel<2> : chunk_state_kernel<1>;
  const int smem = (int)state_smem(p.dim) + 1024, rc = set_smem((const void*)kernel, smem);
  if (rc != 0) return rc;
  const dim3 grid((unsigned)(most * ((p.vdim + VW - 1) / VW)), (unsigned)p.H, (unsigned)batch);
  kernel<<<grid, 256, smem, st>>>(p, ch, error);
  return (int)cudaGetLastError();
}

int launch_chunk_out(const Args<bf16>& p, const Chunks& ch, int most, int batch, int* error, cudaStream_t st) {
  const int smem = (int)(out_keys_bytes(p.dim) + 2 * HALF) + p.dim * 4 + 1024;
  const int rc = set_smem((const void*)chunk_out_kernel, smem);
  if (rc != 0) return rc;
  const dim3 grid((unsigned)(most * ((p.vdim + VW - 1) / VW)), (unsigned)p.H, (unsigned)batch);
  chunk_out_kernel<<<grid, 256, smem, st>>>(p, ch, error);
  return (int)cudaGetLastError();
}

}  // namespace mem
}  // namespace msrl
