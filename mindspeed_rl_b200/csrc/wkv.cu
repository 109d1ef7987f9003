// Linear attention whose state decays per head and key channel by what the token says (wkv), for prompts (prefill portions)
// and single-token decode steps.  Everything is fp32 apart from rows in the activation type.
//
//   mix     five rows per token, h + (h' - h) mu_m with h' the previous token's h (zero before a sequence's first token); the
//           last token's h is carried in a state slot
//   decay   w = exp(-exp(tanh(a) w2^T + w0)) of the bottleneck's rows a [tokens, rank]
//   scan    per head, state S [dim, dim], zero before a sequence's first token:
//               o = S^T r + (sum_k r u k) v;   S <- diag(w) S + k v^T
//           and  y = o / rms(o) * norm * silu(gate)
//
// The scan keeps S in registers: KL lanes share two value columns, state entries of neighbouring keys go through packed
// fp32 instructions.  A batch that fills the machine runs each sequence from end to end.  Otherwise sequences are cut into
// segments: what every segment adds to the state and the product of its decays (all segments in parallel), a pass over the
// segments that leaves the state before each one, and the scan of every segment from there.  Decays are only ever
// multiplied.  bf16 rows of the usual sizes take sixteen tokens at a time on the tensor cores (wkv_chunk.cu), others one
// after the other.  Decode is one kernel: S read and written once, coalesced.
#include "packed_f32.cuh"
#include "wkv.cuh"

namespace msrl {
namespace wkv {

// ---- mixes of neighbouring tokens -----------------------------------------------------------------------------
constexpr int MIXES = 5;

// One block per token.  cu == nullptr: every token is a sequence's next one and `start` its position.
template <typename T, int V>
__global__ void __launch_bounds__(256)
mix_kernel(const T* h, const float* mu, float* last, const int* tok_seq, const int* cu, const int* start,
           const long long* slots, T* out, long long tokens, int W) {
  const long long t = blockIdx.x;
  const int b = cu != nullptr ? tok_seq[t] : (int)t;
  const long long first = cu != nullptr ? cu[b] : t, end = cu != nullptr ? cu[b + 1] : t + 1;
  const long long slot = slots[b];
  const bool lead = t == first, carried = lead && start[b] > 0 && slot >= 0;
  float* mem = last + slot * W;
  for (int c = threadIdx.x * V; c < W; c += 256 * V) {
    float x[4], y[4] = {0.f, 0.f, 0.f, 0.f};
    ldv<V>(h + t * W + c, x);
    if (!lead) ldv<V>(h + (t - 1) * W + c, y);
    else if (carried) ldv<V>(mem + c, y);
    if (lead && slot >= 0) {             // the same thread has read what was there
      float z[4];
      ldv<V>(h + (end - 1) * W + c, z);
      stv<V>(mem + c, z);
    }
#pragma unroll
    for (int i = 0; i < V; ++i) y[i] -= x[i];
#pragma unroll
    for (int m = 0; m < MIXES; ++m) {
      float f[4];
      ldv<V>(mu + m * W + c, f);
#pragma unroll
      for (int i = 0; i < V; ++i) f[i] = x[i] + y[i] * f[i];
      stv<V>(out + (m * tokens + t) * W + c, f);
    }
  }
}

// ---- decays --------------------------------------------------------------------------------------------------
__device__ __forceinline__ float decay_of(float x) { return expf(-expf(x)); }

constexpr int DT = 16;                   // tokens of a block

// grid (channels / 256, tokens / DT); dynamic shared memory: tanh(a) of the tokens
template <typename T>
__global__ void __launch_bounds__(256)
decay_kernel(const float* a, const T* w2, const float* w0, float* w, int tokens, int rank, int channels) {
  extern __shared__ float sm[];          // [rank][DT]
  const int t0 = blockIdx.y * DT, nt = min(DT, tokens - t0);
  for (int i = threadIdx.x; i < DT * rank; i += 256) {
    const int s = i / rank, j = i - s * rank;
    sm[j * DT + s] = s < nt ? tanhf(a[(long long)(t0 + s) * rank + j]) : 0.f;
  }
  __syncthreads();
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c >= channels) return;
  float acc[DT];
  const float bias = w0[c];
#pragma unroll
  for (int s = 0; s < DT; ++s) acc[s] = bias;
  const T* row = w2 + (long long)c * rank;
  for (int j = 0; j < rank; ++j) {
    const float f = ldf(row + j);
#pragma unroll
    for (int s = 0; s < DT; s += 4) {
      const float4 x = *reinterpret_cast<const float4*>(sm + j * DT + s);
      acc[s] += f * x.x;
      acc[s + 1] += f * x.y;
      acc[s + 2] += f * x.z;
      acc[s + 3] += f * x.w;
    }
  }
#pragma unroll
  for (int s = 0; s < DT; ++s)
    if (s < nt) w[(long long)(t0 + s) * channels + c] = decay_of(acc[s]);
}

// ---- recurrence, token by token ----------------------------------------------------------------------------------
constexpr int scan_floats(int DP, int CS) { return TT * (3 * DP + 3 * CS + 1); }

// DP: padded dim; CS value columns of a block; KL lanes share a pair of columns.  grid (segments x column slices, H, B)
template <typename T, int DP, int CS, int KL, int MODE, int V>
__global__ void __launch_bounds__(CS / 2 * KL) scan_kernel(const Args<T> p) {
  constexpr int THREADS = CS / 2 * KL, PIECES = DP / KL / 4, WARPS = THREADS / 32;
  extern __shared__ __align__(16) float sm[];
  float *sk = sm, *sw = sk + TT * DP, *sr = sw + TT * DP, *sv = sr + TT * DP, *sg = sv + TT * CS, *so = sg + TT * CS,
        *sb = so + TT * CS;
  const int slices = (p.dim + CS - 1) / CS, j = blockIdx.x / slices, slice = blockIdx.x % slices;
  const int h = blockIdx.y, b = blockIdx.z, dim = p.dim, hd = p.H * dim;
  const int s0 = p.cu[b], t0 = s0 + j * p.L, len = min(p.cu[b + 1] - t0, MODE == WHOLE ? 0x7fffffff : p.L);
  if (len <= 0) return;
  const int kl = threadIdx.x % KL, c = threadIdx.x / KL * 2, c0 = slice * CS, width = min(CS, dim - c0);
  const long long slot = p.slots[b];
  const bool old = p.start[b] > 0 && slot >= 0;
  const long long size = (long long)dim * dim;
  float* seg = MODE == WHOLE ? nullptr : p.seg + (seg_id(s0, b, j, p.L) * p.H + h) * size;
  float* mem = MODE == WHOLE ? p.state + (slot * p.H + h) * size : seg;
  const bool load = MODE == FROM_SEGMENT || (MODE == WHOLE && old);
  f2 S[2][PIECES * 2];
#pragma unroll
  for (int i = 0; i < PIECES * 2; ++i) {
    const int k = (i >> 1) * KL * 4 + kl * 4 + (i & 1) * 2;
    float x[2][2] = {{0.f, 0.f}, {0.f, 0.f}};
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int q = 0; q < 2; ++q)
        if (load && k + e < dim && c + q < width) x[q][e] = mem[(long long)(k + e) * dim + c0 + c + q];
    S[0][i] = pack2(x[0][0], x[0][1]);
    S[1][i] = pack2(x[1][0], x[1][1]);
  }
  float product = 1.f;
  for (int base = 0; base < len; base += TT) {
    const int nt = min(TT, len - base);
    const long long row0 = (long long)(t0 + base) * hd + h * dim;
    __syncthreads();
    for (int i = threadIdx.x * V; i < TT * DP; i += THREADS * V) {
      const int s = i / DP, d = i % DP;
      float fk[4] = {0.f, 0.f, 0.f, 0.f}, fw[4] = {1.f, 1.f, 1.f, 1.f}, fr[4] = {0.f, 0.f, 0.f, 0.f};
      if (s < nt && d < dim) {
        const long long at = row0 + (long long)s * hd + d;
        ldv<V>(p.k + at, fk);
        ldv<V>(p.w + at, fw);
        if (MODE != ADDED) ldv<V>(p.r + at, fr);
      }
      stv<V>(sk + i, fk);
      stv<V>(sw + i, fw);
      if (MODE != ADDED) stv<V>(sr + i, fr);
    }
    for (int i = threadIdx.x * V; i < TT * CS; i += THREADS * V) {
      const int s = i / CS, d = i % CS;
      float fv[4] = {0.f, 0.f, 0.f, 0.f}, fg[4] = {0.f, 0.f, 0.f, 0.f};
      if (s < nt && d < width) {
        const long long at = row0 + (long long)s * hd + c0 + d;
        ldv<V>(p.v + at, fv);
        if (MODE != ADDED) ldv<V>(p.g + at, fg);
      }
      stv<V>(sv + i, fv);
      if (MODE != ADDED) stv<V>(sg + i, fg);
    }
    __syncthreads();
    if constexpr (MODE == ADDED) {
      if (slice == 0 && threadIdx.x < dim)
        for (int s = 0; s < nt; ++s) product *= sw[s * DP + threadIdx.x];
    } else {
      const int lane = threadIdx.x & 31;
      for (int s = threadIdx.x >> 5; s < nt; s += WARPS) {
        float x = 0.f;
        for (int d = lane; d < dim; d += 32) x += sr[s * DP + d] * p.u[h * dim + d] * sk[s * DP + d];
        x = warp_sum(x);
        if (lane == 0) sb[s] = x;
      }
      __syncthreads();
    }
#pragma unroll 2
    for (int s = 0; s < nt; ++s) {
      const float2 v = *reinterpret_cast<const float2*>(sv + s * CS + c);
      const f2 v0 = pack2(v.x, v.x), v1 = pack2(v.y, v.y);
      f2 a0 = pack2(0.f, 0.f), a1 = a0;
#pragma unroll
      for (int q = 0; q < PIECES; ++q) {
        const int at = s * DP + q * KL * 4 + kl * 4;
        const ulonglong2 k2 = *reinterpret_cast<const ulonglong2*>(sk + at), w2 = *reinterpret_cast<const ulonglong2*>(sw + at);
        if constexpr (MODE != ADDED) {
          const ulonglong2 r2 = *reinterpret_cast<const ulonglong2*>(sr + at);
          a0 = fma2(r2.x, S[0][2 * q], a0);
          a1 = fma2(r2.x, S[1][2 * q], a1);
          a0 = fma2(r2.y, S[0][2 * q + 1], a0);
          a1 = fma2(r2.y, S[1][2 * q + 1], a1);
        }
        S[0][2 * q] = fma2(S[0][2 * q], w2.x, mul2(k2.x, v0));
        S[1][2 * q] = fma2(S[1][2 * q], w2.x, mul2(k2.x, v1));
        S[0][2 * q + 1] = fma2(S[0][2 * q + 1], w2.y, mul2(k2.y, v0));
        S[1][2 * q + 1] = fma2(S[1][2 * q + 1], w2.y, mul2(k2.y, v1));
      }
      if constexpr (MODE != ADDED) {     // lanes 0 and 1 of the KL end up with one column each
        const float2 x0 = unpack2(a0), x1 = unpack2(a1);
        const float mine0 = x0.x + x0.y, mine1 = x1.x + x1.y;
        float x = kl & 1 ? mine1 : mine0;
        x += __shfl_xor_sync(0xffffffffu, kl & 1 ? mine0 : mine1, 1);
#pragma unroll
        for (int d = 2; d < KL; d <<= 1) x += __shfl_xor_sync(0xffffffffu, x, d);
        if (kl < 2) so[s * CS + c + kl] = x + sb[s] * (kl ? v.y : v.x);
      }
    }
    if constexpr (MODE != ADDED) {
      __syncthreads();
      constexpr int G = THREADS / TT < 32 ? THREADS / TT : 32;     // threads of a token
      const int gl = threadIdx.x % G;
      for (int s = threadIdx.x / G; s < TT; s += THREADS / G) {
        if (p.o != nullptr) {
          if (s < nt)
            for (int d = gl; d < width; d += G) p.o[row0 + (long long)s * hd + c0 + d] = so[s * CS + d];
          continue;
        }
        float ss = 0.f;
        if (s < nt)
          for (int d = gl; d < width; d += G) ss += so[s * CS + d] * so[s * CS + d];
#pragma unroll
        for (int x = G / 2; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
        if (s >= nt) continue;
        const float inv = 1.f / sqrtf(ss / (float)dim + p.eps);
        for (int d = gl * V; d < width; d += G * V) {
          float f[4], n[4];
          ldv<V>(p.norm + h * dim + d, n);
#pragma unroll
          for (int i = 0; i < V; ++i) {
            const float z = sg[s * CS + d + i];
            f[i] = so[s * CS + d + i] * inv * n[i] * z * sigmoid_t<T>(z);
          }
          stv<V>(p.y + row0 + (long long)s * hd + d, f);
        }
      }
    }
  }
  if (MODE == FROM_SEGMENT || (MODE == WHOLE && slot < 0)) return;
#pragma unroll
  for (int i = 0; i < PIECES * 2; ++i) {
    const int k = (i >> 1) * KL * 4 + kl * 4 + (i & 1) * 2;
    const float2 x0 = unpack2(S[0][i]), x1 = unpack2(S[1][i]);
    const float x[2][2] = {{x0.x, x0.y}, {x1.x, x1.y}};
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int q = 0; q < 2; ++q)
        if (k + e < dim && c + q < width) mem[(long long)(k + e) * dim + c0 + c + q] = x[q][e];
  }
  if (MODE == ADDED && slice == 0 && threadIdx.x < dim)
    p.seg_w[(seg_id(s0, b, j, p.L) * p.H + h) * dim + threadIdx.x] = product;
}

// grid (state elements / 256, H, B): one element per thread, segment after segment
template <typename T>
__global__ void __launch_bounds__(256) carry_kernel(const Args<T> p) {
  constexpr int AHEAD = 8;
  const int h = blockIdx.y, b = blockIdx.z, dim = p.dim;
  const int t0 = p.cu[b], len = p.cu[b + 1] - t0, n = (len + p.L - 1) / p.L, e = blockIdx.x * 256 + threadIdx.x;
  const int size = dim * dim;
  if (len <= 0 || e >= size) return;
  const long long slot = p.slots[b], id = seg_id(t0, b, 0, p.L) * p.H + h;
  float* mine = p.state + (slot * p.H + h) * size + e;
  float s = p.start[b] > 0 && slot >= 0 ? *mine : 0.f;
  float* x = p.seg + id * size + e;
  const float* w = p.seg_w + id * dim + e / dim;
  for (int j0 = 0; j0 < n; j0 += AHEAD) {
    float added[AHEAD], keep[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (j0 + i < n) {
        added[i] = x[(long long)(j0 + i) * p.H * size];
        keep[i] = w[(long long)(j0 + i) * p.H * dim];
      }
    }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (j0 + i < n) {
        x[(long long)(j0 + i) * p.H * size] = s;
        s = keep[i] * s + added[i];
      }
    }
  }
  if (slot >= 0) *mine = s;
}

// y = o / rms(o) * norm * silu(gate): one warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) finish_kernel(const Args<T> p, long long rows) {
  const long long r = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (r >= rows) return;
  const int lane = threadIdx.x & 31, h = (int)(r % p.H);
  const float* x = p.o + r * p.dim;
  float ss = 0.f;
  for (int c = lane; c < p.dim; c += 32) ss += x[c] * x[c];
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
  for (int c = lane; c < p.dim; c += 32) {
    const float z = ldf(p.g + r * p.dim + c);
    stf(p.y + r * p.dim + c, x[c] * inv * p.norm[h * p.dim + c] * z * sigmoid_t<T>(z));
  }
}

// ---- decode ----------------------------------------------------------------------------------------------------
constexpr int DB = 4;                    // state rows of a thread in flight

// One block per (head, sequence); `start` holds positions.  V columns of a row per thread.  Decays are read, or come from the
// bottleneck's row a, `per` lanes a channel.  dynamic shared memory: r, k, w [dim], tanh(a) [rank], partial outputs [lanes][dim]
template <typename T, int V>
__global__ void __launch_bounds__(256)
decode_kernel(const Args<T> p, const float* a, const T* w2, const float* w0, int rank, int lanes, int per) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  const int h = blockIdx.x, b = blockIdx.y, dim = p.dim;
  float *part = sm, *sr = part + lanes * dim, *sk = sr + dim, *sw = sk + dim, *sa = sw + dim;
  const long long slot = p.slots[b], at = ((long long)b * p.H + h) * dim;
  if (slot < 0) {
    for (int c = threadIdx.x; c < dim; c += 256) stf(p.y + at + c, 0.f);
    return;
  }
  const bool fresh = p.start[b] == 0;
  const int units = dim / V, cu = threadIdx.x % units, rl = threadIdx.x / units;
  float* S = p.state + (slot * p.H + h) * dim * dim + cu * V;
  float s[DB][4];
  auto fetch = [&](int r0) {
#pragma unroll
    for (int i = 0; i < DB; ++i) {
      const int r = r0 + i * lanes;
#pragma unroll
      for (int x = 0; x < V; ++x) s[i][x] = 0.f;
      if (rl < lanes && !fresh && r < dim) ldv<V>(S + (long long)r * dim, s[i]);
    }
  };
  fetch(rl);                             // everything that comes from memory is on its way before the first wait
  const int own = threadIdx.x;           // the thread's column of the output and key channel (dim <= 256)
  const bool mine = own < dim;
  float v[4], bonus = 0.f, value = 0.f, z = 0.f, weight = 0.f;
  if (rl < lanes) ldv<V>(p.v + at + cu * V, v);
  if (mine) {
    const float r = ldf(p.r + at + own), k = ldf(p.k + at + own), u = p.u[h * dim + own];
    if (p.w != nullptr) sw[own] = p.w[at + own];
    value = ldf(p.v + at + own);
    z = ldf(p.g + at + own);
    weight = p.norm[h * dim + own];
    sr[own] = r;
    sk[own] = k;
    bonus = r * u * k;
  }
  if (p.w == nullptr) {
    for (int j = threadIdx.x; j < rank; j += 256) sa[j] = tanhf(a[(long long)b * rank + j]);
    __syncthreads();
    const int part_of = threadIdx.x % per;
    for (int d0 = 0; d0 < dim; d0 += 256 / per) {
      const int d = d0 + threadIdx.x / per;
      float x = 0.f;
      if (d < dim) {
        const T* row = w2 + (long long)(h * dim + d) * rank;
        if (rank % 4 == 0) {
#pragma unroll 4
          for (int j = part_of * 4; j < rank; j += per * 4) {
            float f[4];
            ldf4(row + j, f);
            x += f[0] * sa[j] + f[1] * sa[j + 1] + f[2] * sa[j + 2] + f[3] * sa[j + 3];
          }
        } else {
          for (int j = part_of; j < rank; j += per) x += ldf(row + j) * sa[j];
        }
      }
      for (int m = per / 2; m > 0; m >>= 1) x += __shfl_xor_sync(0xffffffffu, x, m);
      if (d < dim && part_of == 0) sw[d] = decay_of(x + w0[h * dim + d]);
    }
  }
  bonus = block_sum(bonus, red);         // (synchronises sr, sk, sw)
  float o[4] = {0.f, 0.f, 0.f, 0.f};
  if (rl < lanes) {
    for (int r0 = rl; r0 < dim; r0 += lanes * DB) {
      if (r0 != rl) fetch(r0);
#pragma unroll
      for (int i = 0; i < DB; ++i) {
        const int r = r0 + i * lanes;
        if (r < dim) {
          const float k = sk[r], q = sr[r], w = sw[r];
#pragma unroll
          for (int x = 0; x < V; ++x) {
            o[x] += q * s[i][x];
            s[i][x] = w * s[i][x] + k * v[x];
          }
          stv<V>(S + (long long)r * dim, s[i]);
        }
      }
    }
    stv<V>(part + rl * dim + cu * V, o);
  }
  __syncthreads();
  float x = 0.f;
  if (mine) {
    x = bonus * value;
    for (int l = 0; l < lanes; ++l) x += part[l * dim + own];
  }
  const float inv = 1.f / sqrtf(block_sum(x * x, red) / (float)dim + p.eps);
  if (mine) stf(p.y + at + own, x * inv * weight * z * sigmoid_t<T>(z));
}

template <typename T>
int launch_carry(const Args<T>& p, int batch, cudaStream_t st) {
  carry_kernel<T><<<dim3((unsigned)((p.dim * p.dim + 255) / 256), (unsigned)p.H, (unsigned)batch), 256, 0, st>>>(p);
  return (int)cudaGetLastError();
}

template <typename T, int DP, int CS, int KL, int V>
int launch_scan(const Args<T>& p, int most, int batch, cudaStream_t st) {
  const int slices = (p.dim + CS - 1) / CS, smem = scan_floats(DP, CS) * (int)sizeof(float);
  auto go = [&](auto* kernel, int segments) {
    const cudaError_t rc = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (rc != cudaSuccess) return (int)rc;
    kernel<<<dim3((unsigned)(segments * slices), (unsigned)p.H, (unsigned)batch), CS / 2 * KL, smem, st>>>(p);
    return (int)cudaGetLastError();
  };
  if (most == 1) return go(scan_kernel<T, DP, CS, KL, WHOLE, V>, 1);
  int rc = go(scan_kernel<T, DP, CS, KL, ADDED, V>, most);
  if (rc == 0) rc = launch_carry(p, batch, st);
  return rc != 0 ? rc : go(scan_kernel<T, DP, CS, KL, FROM_SEGMENT, V>, most);
}

template <typename T, int V>
int launch_by_dim(const Args<T>& p, int most, int batch, cudaStream_t st) {
  if (p.dim <= 32) return launch_scan<T, 32, 32, 4, V>(p, most, batch, st);
  if (p.dim <= 64) return launch_scan<T, 64, 64, 4, V>(p, most, batch, st);
  if (p.dim <= 128) return launch_scan<T, 128, 128, 8, V>(p, most, batch, st);
  return launch_scan<T, 256, 64, 16, V>(p, most, batch, st);
}

static int launch_chunks(const Args<__nv_bfloat16>& p, int most, int batch, cudaStream_t st) {
  if (most == 1) return launch_chunked(p, WHOLE, 1, batch, st);
  int rc = launch_chunked(p, ADDED, most, batch, st);
  if (rc == 0) rc = launch_carry(p, batch, st);
  return rc != 0 ? rc : launch_chunked(p, FROM_SEGMENT, most, batch, st);
}

// Tokens per segment: a few blocks for every multiprocessor, no segment shorter than 64 tokens
static int segment_length(int H, int tokens, int max_q) {
  const long long want = (long long)tokens * H / (8LL * sm_count());
  const long long L = (want < 64 ? 64 : want + TT - 1) / TT * TT;
  return 2 * L > max_q ? (max_q > 0 ? max_q : 1) : (int)L;
}

}  // namespace wkv
}  // namespace msrl

using namespace msrl;

// h [tokens, W] -> out [5, tokens, W]; cu == null: one token per sequence, `start` holds positions
MSRL_API int msrl_wkv_mix(const void* h, const float* mu, float* last, const int* tok_seq, const int* cu, const int* start,
                          const long long* slots, void* out, long long tokens, int W, int is_f32, cudaStream_t st) {
  if (tokens == 0) return 0;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    if (W % 4 == 0) wkv::mix_kernel<T, 4><<<(unsigned)tokens, 256, 0, st>>>((const T*)h, mu, last, tok_seq, cu, start, slots,
                                                                            (T*)out, tokens, W);
    else wkv::mix_kernel<T, 1><<<(unsigned)tokens, 256, 0, st>>>((const T*)h, mu, last, tok_seq, cu, start, slots, (T*)out,
                                                                 tokens, W);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

MSRL_API int msrl_wkv_decay(const float* a, const void* w2, const float* w0, float* w, int tokens, int rank, int channels,
                            int is_f32, cudaStream_t st) {
  if (tokens == 0) return 0;
  if (rank > 512) return (int)cudaErrorNotSupported;
  if (!is_f32 && channels % 2 == 0 && rank <= 128)
    return wkv::launch_decay(a, (const __nv_bfloat16*)w2, w0, w, tokens, rank, channels, st);
  const dim3 grid((unsigned)((channels + 255) / 256), (unsigned)((tokens + wkv::DT - 1) / wkv::DT));
  const size_t smem = (size_t)rank * wkv::DT * sizeof(float);
  auto run = [&](auto tag) {
    using T = decltype(tag);
    wkv::decay_kernel<T><<<grid, 256, smem, st>>>(a, (const T*)w2, w0, w, tokens, rank, channels);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

// floats of scratch for `segment` tokens per segment (0: chosen here)
MSRL_API long long msrl_wkv_scratch(int H, int dim, int tokens, int batch, int max_q, int segment) {
  const int L = segment > 0 ? segment : wkv::segment_length(H, tokens, max_q);
  const long long segments = max_q > L ? (long long)tokens / L + batch : 0;
  return segments * H * ((long long)dim * dim + dim) + (dim > 128 ? (long long)tokens * H * dim : 0) + 4;
}

MSRL_API int msrl_wkv_prefill(const void* r, const void* k, const void* v, const void* g, const float* w, const float* u,
                              const float* norm, float* state, const int* cu, const int* start, const long long* slots, int H,
                              int dim, float eps, int tokens, int batch, int max_q, int segment, int chunked, float* scratch,
                              void* y, int is_f32, cudaStream_t st) {
  if (batch == 0 || tokens == 0) return 0;
  if (dim > 256 || batch > 65535 || H > 65535) return (int)cudaErrorNotSupported;
  const int L = segment > 0 ? segment : wkv::segment_length(H, tokens, max_q);
  const long long segments = max_q > L ? (long long)tokens / L + batch : 0;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    wkv::Args<T> p{(const T*)r, (const T*)k, (const T*)v, (const T*)g, w, u, norm, state, cu, start, slots, (T*)y, H, dim, eps,
                   L, scratch, scratch + segments * H * dim * dim, nullptr};
    if (dim > 128) p.o = p.seg_w + segments * H * dim;
    const int most = (max_q + L - 1) / L;
    if constexpr (sizeof(T) == 2)
      if (chunked && dim % 8 == 0 && dim <= 128) return wkv::launch_chunks(p, most, batch, st);
    const int rc = dim % 4 == 0 ? wkv::launch_by_dim<T, 4>(p, most, batch, st) : wkv::launch_by_dim<T, 1>(p, most, batch, st);
    if (rc != 0 || dim <= 128) return rc;
    const long long rows = (long long)tokens * H;
    wkv::finish_kernel<T><<<(unsigned)((rows + 7) / 8), 256, 0, st>>>(p, rows);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

// One token per sequence; w: decays [batch, H * dim], or null: from the bottleneck's rows a [batch, rank]
MSRL_API int msrl_wkv_decode(const void* r, const void* k, const void* v, const void* g, const float* w, const float* a,
                             const void* w2, const float* w0, const float* u, const float* norm, float* state, const int* positions,
                             const long long* slots, int H, int dim, int rank, float eps, int batch, void* y, int is_f32,
                             cudaStream_t st) {
  if (batch == 0) return 0;
  if (dim > 256 || rank > 512 || batch > 65535) return (int)cudaErrorNotSupported;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const wkv::Args<T> p{(const T*)r, (const T*)k, (const T*)v, (const T*)g, w, u, norm, state, nullptr, positions, slots,
                         (T*)y, H, dim, eps, 1, nullptr, nullptr, nullptr};
    const int units = dim % 4 == 0 ? dim / 4 : dim, lanes = 256 / units;
    int per = 1;                         // lanes of a channel's decay
    while (per < 16 && per * 2 * dim <= 256) per *= 2;
    const size_t smem = ((size_t)(lanes + 3) * dim + rank) * sizeof(float);
    const dim3 grid((unsigned)H, (unsigned)batch);
    if (dim % 4 == 0) wkv::decode_kernel<T, 4><<<grid, 256, smem, st>>>(p, a, (const T*)w2, w0, rank, lanes, per);
    else wkv::decode_kernel<T, 1><<<grid, 256, smem, st>>>(p, a, (const T*)w2, w0, rank, lanes, per);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}
