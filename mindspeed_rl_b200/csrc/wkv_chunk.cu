// The wkv recurrence (see wkv.cu) for bf16 prompts, sixteen tokens at a time on the tensor cores.
//
// One block walks a sequence or a segment of one head; the transposed state S^T [value, key] stays in its registers as fp32
// accumulators, sixteen value rows per warp.  Inside sixteen tokens, with the products of decays P_t = w_0 .. w_{t-1},
// Q_s = w_{s+1} .. w_15 and D = w_0 .. w_15 (per key channel; at most one, so nothing is ever divided by a decay):
//
//   R_t = r_t P_t,  K_s = k_s Q_s
//   A_ts = sum_k r_t k_s (w_{s+1} .. w_{t-1}) for s < t,  A_tt = sum_k r_t u k_t      fp32 on the CUDA cores
//   O^T = S^T R^T + V^T A^T,   S^T <- S^T diag(D) + V^T K
//
// Decays differ from channel to channel and may be anything in (0, 1), so scores inside the sixteen tokens cannot be split
// into a factor of t and one of s; this bounds the tile and makes warp-level products the ones that fit.  32-bit operands
// (S, R, K, A) are taken apart into three bf16 terms of 24 bits together: V is exact, so its products take three passes; S and
// R are both 32-bit and take the six products above 2^-24.  Sums are fp32.
#include "mma_utils.cuh"
#include "wkv.cuh"

namespace msrl {
namespace wkv {

using bf16 = __nv_bfloat16;

constexpr int TOK = 16, TERMS = 3, AP = 24;      // tokens of a chunk; bf16 terms of a 32-bit operand; pitch of A's rows

template <int DP>
struct Smem {
  static constexpr int RP = DP + 8, OP = DP + 4;                       // pitches of bf16 rows and of output rows
  static constexpr int RAW = 4 * TOK * RP * 2 + TOK * DP * 4;          // bytes: r | k | v | g | decays
  static constexpr int R_AT = 2 * RAW, K_AT = R_AT + TERMS * TOK * RP * 2, A_AT = K_AT + TERMS * TOK * RP * 2;
  static constexpr int O_AT = A_AT + TERMS * TOK * AP * 2, D_AT = O_AT + TOK * OP * 4, BYTES = D_AT + DP * 4;
};

// the three bf16 terms of a pair
__device__ __forceinline__ void split2(float x, float y, uint32_t (&t)[TERMS]) {
#pragma unroll
  for (int i = 0; i < TERMS; ++i) {
    t[i] = pack_bf16(x, y);
    x -= __uint_as_float(t[i] << 16);
    y -= __uint_as_float(t[i] & 0xffff0000u);
  }
}

// Sums of sixteen values over LANES lanes: N values per lane are halved until a lane keeps one (or two) of them, from `index` on
template <int N, int STEP, int LANES>
__device__ __forceinline__ void sum_lanes(float (&acc)[16], int lane, int& index) {
  if constexpr (STEP < LANES) {
    if constexpr (N > 1) {
      constexpr int H = N / 2;
      const bool up = lane & STEP;
      if (up) index += H;
#pragma unroll
      for (int e = 0; e < H; ++e) {
        const float low = acc[e], high = acc[e + H];
        acc[e] = (up ? high : low) + __shfl_xor_sync(0xffffffffu, up ? low : high, STEP);
      }
      sum_lanes<H, STEP * 2, LANES>(acc, lane, index);
    } else {
      acc[0] += __shfl_xor_sync(0xffffffffu, acc[0], STEP);
      sum_lanes<1, STEP * 2, LANES>(acc, lane, index);
    }
  }
}

// grid (segments, H, B), 2 DP threads
template <int DP, int MODE>
__global__ void __launch_bounds__(2 * DP, DP == 128 ? 2 : DP == 64 ? 4 : 8) chunk_kernel(const Args<bf16> p) {
  using M = Smem<DP>;
  constexpr int THREADS = 2 * DP, NT = DP / 8, RP = M::RP, OP = M::OP;
  extern __shared__ __align__(16) unsigned char raw[];
  bf16 *sR = reinterpret_cast<bf16*>(raw + M::R_AT), *sK = reinterpret_cast<bf16*>(raw + M::K_AT),
       *sA = reinterpret_cast<bf16*>(raw + M::A_AT);
  float *sO = reinterpret_cast<float*>(raw + M::O_AT), *sD = reinterpret_cast<float*>(raw + M::D_AT);
  const int j = blockIdx.x, h = blockIdx.y, b = blockIdx.z, dim = p.dim, hd = p.H * dim;
  const int s0 = p.cu[b], t0 = s0 + j * p.L, len = min(p.cu[b + 1] - t0, MODE == WHOLE ? 0x7fffffff : p.L);
  if (len <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gid = lane >> 2, tig = lane & 3, v0 = warp * 16;
  const int chunks = (len + TOK - 1) / TOK;
  const long long slot = p.slots[b], size = (long long)dim * dim;
  const bool old = p.start[b] > 0 && slot >= 0;
  float* mem = MODE == WHOLE ? p.state + (slot * p.H + h) * size : p.seg + (seg_id(s0, b, j, p.L) * p.H + h) * size;

  auto tile = [&](int stage, int which) { return reinterpret_cast<bf16*>(raw + stage * M::RAW) + which * TOK * RP; };
  auto decays = [&](int stage) { return reinterpret_cast<float*>(raw + stage * M::RAW + 4 * TOK * RP * 2); };
  auto load = [&](int c) {
    const int stage = c & 1, nt = min(TOK, len - c * TOK);
    const long long row0 = (long long)(t0 + c * TOK) * hd + h * dim;
    for (int i = tid; i < TOK * DP / 8; i += THREADS) {
      const int s = i / (DP / 8), d = i % (DP / 8) * 8;
      const bool ok = s < nt && d < dim;
      const long long at = ok ? row0 + (long long)s * hd + d : 0;
      if (MODE != ADDED) {
        cp_async16(tile(stage, 0) + s * RP + d, p.r + at, ok);
        cp_async16(tile(stage, 3) + s * RP + d, p.g + at, ok);
      }
      cp_async16(tile(stage, 1) + s * RP + d, p.k + at, ok);
      cp_async16(tile(stage, 2) + s * RP + d, p.v + at, ok);
    }
    for (int i = tid; i < TOK * DP / 4; i += THREADS) {
      const int s = i / (DP / 4), d = i % (DP / 4) * 4;
      const bool ok = s < nt && d < dim;
      cp_async16(decays(stage) + s * DP + d, p.w + (ok ? row0 + (long long)s * hd + d : 0), ok);
    }
    cp_async_commit();
  };
  load(0);

  float S[NT][4];                        // value rows v0 + gid (+ 8), keys 8 n + 2 tig (+ 1)
  const bool from = MODE == FROM_SEGMENT || (MODE == WHOLE && old);
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int k = n * 8 + 2 * tig + (x & 1), v = v0 + gid + (x >> 1) * 8;
      S[n][x] = from && k < dim && v < dim ? mem[(long long)k * dim + v] : 0.f;
    }
  // scores: a slice of four channels of the token pair (a, 15 - a)
  constexpr int LANES = DP / 4;
  const int slice = tid % LANES, a = tid / LANES;
  float u[4] = {0.f, 0.f, 0.f, 0.f};
  if (MODE != ADDED) {
    for (int i = tid; i < TERMS * TOK * AP / 2; i += THREADS) reinterpret_cast<uint32_t*>(sA)[i] = 0u;
    if (slice * 4 < dim) ldf4(p.u + h * dim + slice * 4, u);
  }
  float product = 1.f;

  // R, K and D of a chunk
  auto prep = [&](int c) {
    const int stage = c & 1, nt = min(TOK, len - c * TOK);
    const float* w = decays(stage);
    const int d = tid % (DP / 2) * 2, q = tid / (DP / 2);
    auto w_of = [&](int s) { return s < nt ? *reinterpret_cast<const float2*>(w + s * DP + d) : make_float2(1.f, 1.f); };
    auto put = [&](bf16* terms, int s, const bf16* x, const float2& m) {
      const float2 f = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(x + s * RP + d));
      uint32_t t[TERMS];
      split2(f.x * m.x, f.y * m.y, t);
#pragma unroll
      for (int i = 0; i < TERMS; ++i) *reinterpret_cast<uint32_t*>(terms + (i * TOK + s) * RP + d) = t[i];
    };
    float2 m = make_float2(1.f, 1.f);
    auto times = [&](int s) {
      const float2 x = w_of(s);
      m.x *= x.x;
      m.y *= x.y;
    };
    if (MODE != ADDED && q < 2) {        // R: tokens 0 .. 7 and 8 .. 15
      if (q == 1)
#pragma unroll
        for (int s = 0; s < TOK / 2; ++s) times(s);
#pragma unroll
      for (int s = 0; s < TOK / 2; ++s) {
        put(sR, q * (TOK / 2) + s, tile(stage, 0), m);
        times(q * (TOK / 2) + s);
      }
      if (q == 1) *reinterpret_cast<float2*>(sD + d) = m;
    } else {                             // K, from the last token of a part to its first
      constexpr int PART = MODE == ADDED ? TOK / 4 : TOK / 2;
      const int first = (MODE == ADDED ? q : q - 2) * PART;
      for (int s = TOK - 1; s >= first + PART; --s) times(s);
#pragma unroll
      for (int s = PART - 1; s >= 0; --s) {
        put(sK, first + s, tile(stage, 1), m);
        times(first + s);
      }
      if (MODE == ADDED && q == 0) *reinterpret_cast<float2*>(sD + d) = m;
    }
  };

  auto scores = [&](int c) {
    const int stage = c & 1;
    const bf16 *r = tile(stage, 0) + slice * 4, *k = tile(stage, 1) + slice * 4;
    const float* w = decays(stage) + slice * 4;
    float x[4], last[4], acc[16];
    ldf4(k + a * RP, x);
    ldf4(k + (15 - a) * RP, last);
    auto dot = [](const float (&y)[4], const float (&z)[4]) { return y[0] * z[0] + y[1] * z[1] + y[2] * z[2] + y[3] * z[3]; };
    float f[4], own;
    ldf4(r + a * RP, f);
    acc[15] = (f[0] * u[0] * x[0] + f[1] * u[1] * x[1]) + (f[2] * u[2] * x[2] + f[3] * u[3] * x[3]);
    ldf4(r + (15 - a) * RP, f);
    own = (f[0] * u[0] * last[0] + f[1] * u[1] * last[1]) + (f[2] * u[2] * last[2] + f[3] * u[3] * last[3]);
#pragma unroll
    for (int i = 0; i < 15; ++i) {       // the chain of a, then the one of 15 - a: fifteen steps together
      const bool second = i >= 15 - a;
      if (i == 15 - a) {
#pragma unroll
        for (int e = 0; e < 4; ++e) x[e] = last[e];
      }
      const int t = second ? i + 1 : a + 1 + i;
      ldf4(r + t * RP, f);
      const float4 wt = *reinterpret_cast<const float4*>(w + t * DP);
      acc[i] = dot(f, x);
      x[0] *= wt.x;
      x[1] *= wt.y;
      x[2] *= wt.z;
      x[3] *= wt.w;
    }
    int index = 0;
    sum_lanes<16, 1, LANES>(acc, slice, index);
#pragma unroll
    for (int m = 1; m < LANES; m <<= 1) own += __shfl_xor_sync(0xffffffffu, own, m);
    auto put = [&](int t, int s, float y) {
#pragma unroll
      for (int i = 0; i < TERMS; ++i) {
        const bf16 z = __float2bfloat16_rn(y);
        sA[(i * TOK + t) * AP + s] = z;
        y -= __bfloat162float(z);
      }
    };
    if (slice < 16) {
#pragma unroll
      for (int e = 0; e < (LANES < 16 ? 16 / LANES : 1); ++e) {
        const int i = index + e;
        if (i == 15) put(a, a, acc[e]);
        else if (i < 15 - a) put(a + 1 + i, a, acc[e]);
        else put(i + 1, 15 - a, acc[e]);
      }
    }
    if (slice == 0) put(15 - a, 15 - a, own);
  };

  // norm, gate and store of a chunk's outputs
  auto finish = [&](int c) {
    constexpr int G = THREADS / TOK;
    const int s = tid / G, gl = tid % G, nt = min(TOK, len - c * TOK);
    const float* o = sO + s * OP;
    float ss = 0.f;
#pragma unroll
    for (int d = gl * 4; d < DP; d += G * 4) {         // padding is zero
      const float4 x = *reinterpret_cast<const float4*>(o + d);
      ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
    }
#pragma unroll
    for (int m = G / 2; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
    if (s >= nt) return;
    const float inv = 1.f / sqrtf(ss / (float)dim + p.eps);
    bf16* y = p.y + (long long)(t0 + c * TOK + s) * hd + h * dim;
#pragma unroll
    for (int d = gl * 4; d < DP; d += G * 4) {
      if (d >= dim) break;
      float x[4], n[4], z[4];
      ldf4(o + d, x);
      ldf4(p.norm + h * dim + d, n);
      ldf4(tile(c & 1, 3) + s * RP + d, z);
#pragma unroll
      for (int e = 0; e < 4; ++e) x[e] *= inv * n[e] * z[e] * sigmoid_t<bf16>(z[e]);
      stf4(y + d, x);
    }
  };

  const uint32_t r_at = smem_u32(sR), k_at = smem_u32(sK), a_at = smem_u32(sA);
  const int quad = lane >> 3, in8 = lane & 7;
  for (int c = 0; c < chunks; ++c) {
    cp_async_wait<0>();
    __syncthreads();                     // rows of c are there; the products of c - 1 are done, its outputs complete
    prep(c);
    if (MODE != ADDED) {
      scores(c);
      if (c > 0) finish(c - 1);
    }
    __syncthreads();
    if (c + 1 < chunks) load(c + 1);
    uint32_t vt[4];                      // V^T: value rows v0 .. v0 + 15, tokens
    ldmatrix_x4_trans(vt, smem_u32(tile(c & 1, 2) + ((quad >> 1) * 8 + in8) * RP + v0 + (quad & 1) * 8));
    if (MODE != ADDED) {
      float o[2][2][4] = {};             // [chain][eight tokens]
      const int row = (quad >> 1) * 8 + in8, col = (quad & 1) * 8;
#pragma unroll
      for (int n = 0; n < NT; n += 2) {
        uint32_t st[TERMS][4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          uint32_t t[TERMS];
          split2(S[n + (e >> 1)][(e & 1) * 2], S[n + (e >> 1)][(e & 1) * 2 + 1], t);
#pragma unroll
          for (int i = 0; i < TERMS; ++i) st[i][e] = t[i];
        }
#pragma unroll
        for (int i = 0; i < TERMS; ++i) {
          uint32_t rt[4];
          ldmatrix_x4(rt, r_at + ((i * TOK + row) * RP + n * 8 + col) * 2);
#pragma unroll
          for (int e = 0; e + i < TERMS; ++e) {
            mma_16816(o[(i + e) & 1][0], st[e], rt[0], rt[1]);
            mma_16816(o[(i + e) & 1][1], st[e], rt[2], rt[3]);
          }
        }
      }
#pragma unroll
      for (int i = 0; i < TERMS; ++i) {
        uint32_t at[4];
        ldmatrix_x4(at, a_at + ((i * TOK + row) * AP + col) * 2);
        mma_16816(o[i & 1][0], vt, at[0], at[1]);
        mma_16816(o[i & 1][1], vt, at[2], at[3]);
      }
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int x = 0; x < 4; ++x)
          sO[(e * 8 + 2 * tig + (x & 1)) * OP + v0 + gid + (x >> 1) * 8] = o[0][e][x] + o[1][e][x];
    }
#pragma unroll
    for (int n = 0; n < NT; n += 2) {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float2 d = *reinterpret_cast<const float2*>(sD + (n + e) * 8 + 2 * tig);
        S[n + e][0] *= d.x;
        S[n + e][1] *= d.y;
        S[n + e][2] *= d.x;
        S[n + e][3] *= d.y;
      }
#pragma unroll
      for (int i = 0; i < TERMS; ++i) {
        uint32_t kt[4];
        ldmatrix_x4_trans(kt, k_at + ((i * TOK + (quad & 1) * 8 + in8) * RP + n * 8 + (quad >> 1) * 8) * 2);
        mma_16816(S[n], vt, kt[0], kt[1]);
        mma_16816(S[n + 1], vt, kt[2], kt[3]);
      }
    }
    if (MODE == ADDED && tid < dim) product *= sD[tid];
  }
  if (MODE != ADDED) {
    __syncthreads();
    finish(chunks - 1);
  }
  if (MODE == FROM_SEGMENT || (MODE == WHOLE && slot < 0)) return;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int x = 0; x < 4; ++x) {
      const int k = n * 8 + 2 * tig + (x & 1), v = v0 + gid + (x >> 1) * 8;
      if (k < dim && v < dim) mem[(long long)k * dim + v] = S[n][x];
    }
  if (MODE == ADDED && tid < dim) p.seg_w[(seg_id(s0, b, j, p.L) * p.H + h) * dim + tid] = product;
}

// ---- decays: w = exp(-exp(tanh(a) w2^T + w0)), tanh(a) as three bf16 terms ------------------------------------------
constexpr int DM = 64, DN = 256;         // tokens of a tile, channels of a block

__host__ __device__ inline int rank_pitch(int rank) { return (rank + 15) / 16 * 16 + 8; }
__host__ __device__ inline int decay_smem(int rank) { return (TERMS * DM + DN) * rank_pitch(rank) * 2; }

// grid (channels / DN, tokens / (DM tiles)); eight warps of 32 channels
__global__ void __launch_bounds__(256, 2)
decay_mma_kernel(const float* a, const bf16* w2, const float* w0, float* w, int tokens, int rank, int channels, int tiles) {
  extern __shared__ __align__(16) unsigned char raw[];
  const int rp = rank_pitch(rank), k16 = rp - 8;
  bf16 *sA = reinterpret_cast<bf16*>(raw), *sB = sA + TERMS * DM * rp;
  const int c0 = blockIdx.x * DN, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (rank % 16 == 0) {
    for (int i = threadIdx.x; i < DN * rank / 8; i += 256) {
      const int c = i / (rank / 8), k = i % (rank / 8) * 8;
      const bool ok = c0 + c < channels;
      cp_async16(sB + c * rp + k, w2 + (ok ? (long long)(c0 + c) * rank + k : 0), ok);
    }
    cp_async_commit();
  } else {
    for (int i = threadIdx.x; i < DN * k16; i += 256) {
      const int c = i / k16, k = i % k16;
      sB[c * rp + k] = c0 + c < channels && k < rank ? w2[(long long)(c0 + c) * rank + k] : __float2bfloat16_rn(0.f);
    }
  }
  const uint32_t a_at = smem_u32(sA), b_at = smem_u32(sB);
  const int quad = lane >> 3, in8 = lane & 7, n0 = warp * 32, gid = lane >> 2, tig = lane & 3;
  float2 bias[4];
#pragma unroll
  for (int n = 0; n < 4; ++n) {
    const int c = c0 + n0 + n * 8 + 2 * tig;                       // channels are even
    bias[n] = c < channels ? *reinterpret_cast<const float2*>(w0 + c) : make_float2(0.f, 0.f);
  }
  for (int tile = 0; tile < tiles; ++tile) {
    const int t0 = (blockIdx.y * tiles + tile) * DM;
    if (t0 >= tokens) break;
    if (tile > 0) __syncthreads();       // the products of the tile before are done
    for (int i = threadIdx.x; i < DM * k16 / 2; i += 256) {
      const int s = i / (k16 / 2), k = i % (k16 / 2) * 2;
      float x[2] = {0.f, 0.f};
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (t0 + s < tokens && k + e < rank) x[e] = tanhf(a[(long long)(t0 + s) * rank + k + e]);
      uint32_t t[TERMS];
      split2(x[0], x[1], t);
#pragma unroll
      for (int e = 0; e < TERMS; ++e) *reinterpret_cast<uint32_t*>(sA + (e * DM + s) * rp + k) = t[e];
    }
    cp_async_wait<0>();
    __syncthreads();
    float acc[4][4][4] = {};             // [sixteen tokens][eight channels]
    for (int k = 0; k < k16; k += 16) {
      uint32_t bt[2][4];
#pragma unroll
      for (int n = 0; n < 2; ++n)
        ldmatrix_x4(bt[n], b_at + ((n0 + n * 16 + (quad >> 1) * 8 + in8) * rp + k + (quad & 1) * 8) * 2);
#pragma unroll
      for (int e = 0; e < TERMS; ++e)
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          uint32_t at[4];
          ldmatrix_x4(at, a_at + ((e * DM + m * 16 + (quad & 1) * 8 + in8) * rp + k + (quad >> 1) * 8) * 2);
#pragma unroll
          for (int n = 0; n < 4; ++n) mma_16816(acc[m][n], at, bt[n >> 1][(n & 1) * 2], bt[n >> 1][(n & 1) * 2 + 1]);
        }
    }
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const int c = c0 + n0 + n * 8 + 2 * tig;
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = t0 + m * 16 + gid + e * 8;
          if (t < tokens && c < channels)
            *reinterpret_cast<float2*>(w + (long long)t * channels + c) =
                make_float2(expf(-__expf(acc[m][n][2 * e] + bias[n].x)), expf(-__expf(acc[m][n][2 * e + 1] + bias[n].y)));
        }
    }
  }
}

int launch_decay(const float* a, const bf16* w2, const float* w0, float* w, int tokens, int rank, int channels, cudaStream_t st) {
  const int smem = decay_smem(rank);
  const cudaError_t rc = cudaFuncSetAttribute(decay_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (rc != cudaSuccess) return (int)rc;
  const int columns = (channels + DN - 1) / DN, rows = (tokens + DM - 1) / DM;
  const int tiles = columns * rows >= 8 * sm_count() ? 4 : 1;      // of a block: they share the weights
  decay_mma_kernel<<<dim3((unsigned)columns, (unsigned)((rows + tiles - 1) / tiles)), 256, smem, st>>>(a, w2, w0, w, tokens, rank,
                                                                                                       channels, tiles);
  return (int)cudaGetLastError();
}

template <int DP>
static int launch_dim(const Args<bf16>& p, int mode, int segments, int batch, cudaStream_t st) {
  auto go = [&](auto* kernel) {
    const cudaError_t rc = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, Smem<DP>::BYTES);
    if (rc != cudaSuccess) return (int)rc;
    kernel<<<dim3((unsigned)segments, (unsigned)p.H, (unsigned)batch), 2 * DP, Smem<DP>::BYTES, st>>>(p);
    return (int)cudaGetLastError();
  };
  if (mode == WHOLE) return go(chunk_kernel<DP, WHOLE>);
  return mode == ADDED ? go(chunk_kernel<DP, ADDED>) : go(chunk_kernel<DP, FROM_SEGMENT>);
}

int launch_chunked(const Args<bf16>& p, int mode, int segments, int batch, cudaStream_t st) {
  return p.dim <= 32 ? launch_dim<32>(p, mode, segments, batch, st) : p.dim <= 64 ? launch_dim<64>(p, mode, segments, batch, st)
                                                                                  : launch_dim<128>(p, mode, segments, batch, st);
}

}  // namespace wkv
}  // namespace msrl
