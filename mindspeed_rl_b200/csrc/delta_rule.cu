// Gated delta rule with a decay per key channel or per head, for prompts (prefill portions) and single-token decode steps.
//
// Per value head h, with key head hk = h / (H / KVH), state S [dim, vdim] in fp32:
//
//   q, k, v = silu(causal conv over time of the projections)          (last tap = current token)
//   q = q / |q| * dim^-1/2,  k = k / |k|                              (|x| = sqrt(sum x^2 + unit_eps))
//   g = exp(-exp(A_log[h]) * softplus(a + dt_bias))   [dim] or one per head,   beta = sigmoid(b)
//   S <- g * S;  u = beta * (v - S^T k);  S <- S + k u^T;  o = S^T q
//   y = o / rms(o) * norm * (sigmoid or silu)(gate)
//
// What a sequence carries from step to step lives in a state slot: S, and the ring of the short convolutions
// (short_conv.cuh).
//
//   prefill: `prep` (conv, silu, unit norms, decays, step sizes of every token), `scan` (the recurrence: one
//            block per sequence, head and column group; S in registers, LPC lanes share a column) and
//            `out` (norm and gate).  The usual shapes run the recurrence four tokens at a time
//            (`delta_group_kernel`, `delta_group_scan_kernel`), the others token by token;
//   decode:  one fused kernel per (sequence, head): all of the above with S read and written once, coalesced.
//
// Both sum (S^T k, S^T q) over the decayed state in one pass: o = (gS)^T q + (k.q) u.
#include "packed_f32.cuh"
#include "short_conv.cuh"

namespace msrl {

template <typename T>
struct DeltaIn : ConvIn<T> { // proj: q | k | v | b ... sections at the given columns
  int q_col, k_col, v_col, b_col;
  const T* a;                // decay projection, [tokens, H * dim] (a_h = dim, a_d = 1) or [tokens, H] (a_h = 1, a_d = 0)
  long long a_ld;
  int a_h, a_d;
  int silu_gate;
  const float* a_log;        // [H]
  const float* dt_bias;      // like a row of a
  float* state;              // [slots, H, dim, vdim]
  int H, KVH, dim, vdim;
  float unit_eps;
  __device__ __forceinline__ float decay(long long t, int h, int d) const {
    const int c = h * a_h + d * a_d;
    return expf(-expf(a_log[h]) * softplus_f(ldf(a + t * a_ld + c) + dt_bias[c]));
  }
  __device__ __forceinline__ float gate_of(float z) const { return silu_gate ? z * sigmoid_f(z) : sigmoid_f(z); }
};

template <int TAPS, typename T>
__device__ __forceinline__ float conv_silu(const DeltaIn<T>& p, long long t, int i, int pos, long long slot, int col, int ch) {
  const float s = conv_one<TAPS>(static_cast<const ConvIn<T>&>(p), t, i, pos, slot, col, ch);
  return s * sigmoid_t<T>(s);
}

constexpr int DELTA_MAX_DIM = 256;

// ---- prefill: everything that does not depend on the state -------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
delta_prep_kernel(const DeltaIn<T> p, const int* tok_seq, const int* cu, const int* start_pos, const long long* slots,
                  float* qn, float* kn, float* kq, float* vv, float* g, float* beta) {
  const long long t = blockIdx.x;
  const int b = tok_seq[t];
  const int i = (int)(t - cu[b]);
  const int pos = start_pos[b] + i;
  const long long slot = slots[b];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kd = p.KVH * p.dim;
  const float qscale = 1.f / sqrtf((float)p.dim);
  for (int hk = warp; hk < p.KVH; hk += 8) {
    float q[DELTA_MAX_DIM / 32], k[DELTA_MAX_DIM / 32];
    float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
    for (int n = 0; n < DELTA_MAX_DIM / 32; ++n) {
      const int d = n * 32 + lane;
      if (d < p.dim) {
        const int ch = hk * p.dim + d;
        q[n] = conv_silu<0>(p, t, i, pos, slot, p.q_col + ch, ch);
        k[n] = conv_silu<0>(p, t, i, pos, slot, p.k_col + ch, kd + ch);
        qq += q[n] * q[n];
        kk += k[n] * k[n];
        qk += q[n] * k[n];
      }
    }
    const float qs = qscale / sqrtf(warp_sum(qq) + p.unit_eps), ks = 1.f / sqrtf(warp_sum(kk) + p.unit_eps);
    qk = warp_sum(qk) * qs * ks;
#pragma unroll
    for (int n = 0; n < DELTA_MAX_DIM / 32; ++n) {
      const int d = n * 32 + lane;
      if (d < p.dim) {
        qn[t * kd + hk * p.dim + d] = q[n] * qs;
        kn[t * kd + hk * p.dim + d] = k[n] * ks;
      }
    }
    if (lane == 0) kq[t * p.KVH + hk] = qk;
  }
  const int nv = p.H * p.vdim;
  for (int c = threadIdx.x; c < nv; c += 256) vv[t * nv + c] = conv_silu<0>(p, t, i, pos, slot, p.v_col + c, 2 * kd + c);
  const int ng = p.H * p.dim;
  for (int c = threadIdx.x; c < ng; c += 256)
    g[t * ng + c] = p.decay(t, c / p.dim, c % p.dim);
  for (int h = threadIdx.x; h < p.H; h += 256) beta[t * p.H + h] = sigmoid_f(ldf(p.proj + t * p.ld + p.b_col + h));
}

// ---- prefill, usual shapes (dim a multiple of 4 up to 128, vdim a multiple of 4, 2 to 4 taps): a warp walks
// consecutive tokens with the convolution window of its channels in registers, four channels per lane.
constexpr int PREP_TT = 16;

template <typename T>
__device__ __forceinline__ void silu4(float (&y)[4]) {
#pragma unroll
  for (int c = 0; c < 4; ++c) y[c] *= sigmoid_t<T>(y[c]);
}

constexpr int PREP_U = 4;       // tokens whose projections are loaded together

// v of every token: warps of 128 channels, PREP_TT tokens each
template <typename T, int TAPS>
__global__ void __launch_bounds__(256)
delta_value_kernel(const DeltaIn<T> p, const int* tok_seq, const int* cu, const int* start_pos, const long long* slots,
                   int tokens, float* vv) {
  const int kd = p.KVH * p.dim, nv = p.H * p.vdim;
  const int c = (blockIdx.x * 8 + (threadIdx.x >> 5)) * 128 + (threadIdx.x & 31) * 4;
  const int t0 = blockIdx.y * PREP_TT, t1 = min(tokens, t0 + PREP_TT);
  if (c >= nv) return;
  ConvWindow<TAPS, T> cv;
  cv.weights(p.conv, 2 * kd + c);
  int seq = -1;
  float rv[PREP_U][4];
  int sq[PREP_U];
  for (int tb = t0; tb < t1; tb += PREP_U) {
#pragma unroll
    for (int x = 0; x < PREP_U; ++x) {
      const int t = min(tb + x, t1 - 1);
      sq[x] = tok_seq[t];
      ldf4(p.proj + t * p.ld + p.v_col + c, rv[x]);
    }
#pragma unroll
    for (int x = 0; x < PREP_U; ++x) {
      const int t = tb + x;
      if (t >= t1) break;
      if (sq[x] != seq) {
        seq = sq[x];
        const int i = t - cu[seq];
        cv.fill(p, t, i, start_pos[seq] + i, slots[seq], p.v_col + c, 2 * kd + c);
      }
      float y[4];
      cv.step(rv[x], y);
      silu4<T>(y);
      stf4(vv + (long long)t * nv + c, y);
    }
  }
}

// Groups of four tokens.  With G_j = g_0 ... g_j inside a group and S the state before it,
//
//   r_j = S^T (G_j k_j)                    u_j = beta_j (v_j - r_j - sum_{i<j} a_ji u_i)
//   p_j = S^T (G_j q_j)                    o_j = p_j + sum_{i<=j} b_ji u_i
//   S  <- G_3 S + sum_j (k_j g_{j+1} ... g_3) u_j^T
//   a_ji = k_j . (g_{i+1} ... g_j k_i)     b_ji = q_j . (g_{i+1} ... g_j k_i)
//
// which is the recurrence with the tokens' mutual terms taken out of the state: only products of decays (never a
// quotient) appear.  A group and head is one record: G k (4 x DP), G q (4 x DP), the write vectors (4 x DP), G_3 (DP),
// a (6), b (10), beta (4), padding (4).  A sequence's groups start at its first token; record slot of its group n:
// cu[b] / 4 + b + n.  Missing tokens of a last group have k = q = 0, g = 1, beta = 0.
constexpr int GRP = 4, COEF = 24;

__host__ __device__ constexpr int group_floats(int dp) { return 13 * dp + COEF; }

template <typename T, int TAPS, bool HEAD>        // HEAD: one decay per head
__global__ void __launch_bounds__(256, 2)
delta_group_kernel(const DeltaIn<T> p, const int* cu, const int* start_pos, const long long* slots, int batch,
                   int total_slots, int DP, float* rec) {
  const int lane = threadIdx.x & 31, h = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (h >= p.H) return;
  const int hk = h / (p.H / p.KVH), kd = p.KVH * p.dim;
  const int d = lane * 4, ch = hk * p.dim + d;
  const bool on = d < p.dim, pad = !on && d < DP;
  const int CH = group_floats(DP);
  const float rate = -expf(p.a_log[h]);
  const float qscale = 1.f / sqrtf((float)p.dim);
  ConvWindow<TAPS, T> cq, ck;
  float bias[4] = {0.f, 0.f, 0.f, 0.f};
  if (on) {
    cq.weights(p.conv, ch);
    ck.weights(p.conv, kd + ch);
#pragma unroll
    for (int c = 0; c < 4; ++c) bias[c] = p.dt_bias[HEAD ? h : h * p.dim + d + c];
  }
  const int s0 = blockIdx.y * 4, s1 = min(total_slots, s0 + 4);
  int last_b = -1;
  for (int s = s0; s < s1; ++s) {
    int lo = 0, hi = batch - 1;                          // the last sequence whose first slot is at most s
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (cu[mid] / GRP + mid <= s) lo = mid;
      else hi = mid - 1;
    }
    const int b = lo, len = cu[b + 1] - cu[b], i0 = (s - (cu[b] / GRP + b)) * GRP;
    if (i0 >= len) {                                     // a slot between two sequences
      last_b = -1;
      continue;
    }
    const int t0 = cu[b] + i0, cnt = min(GRP, len - i0);
    float q[GRP][4], k[GRP][4], g[GRP][4];
#pragma unroll
    for (int j = 0; j < GRP; ++j) {
      const long long t = t0 + min(j, cnt - 1);
#pragma unroll
      for (int c = 0; c < 4; ++c) q[j][c] = k[j][c] = g[j][c] = 0.f;
      if (on) {
        ldf4(p.proj + t * p.ld + p.q_col + ch, q[j]);
        ldf4(p.proj + t * p.ld + p.k_col + ch, k[j]);
        if constexpr (HEAD) g[j][0] = ldf(p.a + t * p.a_ld + h);
        else ldf4(p.a + t * p.a_ld + h * p.dim + d, g[j]);
      }
    }
    if (on && b != last_b) {
      const int pos = start_pos[b] + i0;
      cq.fill(p, t0, i0, pos, slots[b], p.q_col + ch, ch);
      ck.fill(p, t0, i0, pos, slots[b], p.k_col + ch, kd + ch);
    }
    last_b = b;
    float beta = 0.f;
    if (lane < cnt) beta = sigmoid_f(ldf(p.proj + (long long)(t0 + lane) * p.ld + p.b_col + h));
    float v[8];
#pragma unroll
    for (int j = 0; j < GRP; ++j) {
      v[2 * j] = v[2 * j + 1] = 0.f;
      if (on && j < cnt) {
        cq.step(q[j], q[j]);
        ck.step(k[j], k[j]);
        silu4<T>(q[j]);
        silu4<T>(k[j]);
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          g[j][c] = HEAD && c > 0 ? g[j][0] : expf(rate * softplus_f(g[j][c] + bias[c]));
          v[2 * j] += q[j][c] * q[j][c];
          v[2 * j + 1] += k[j][c] * k[j][c];
        }
      } else {
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          q[j][c] = k[j][c] = 0.f;
          g[j][c] = 1.f;
        }
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
      for (int x = 0; x < 8; ++x) v[x] += __shfl_xor_sync(0xffffffffu, v[x], o);
#pragma unroll
    for (int j = 0; j < GRP; ++j) {
      const float qs = qscale / sqrtf(v[2 * j] + p.unit_eps), ks = 1.f / sqrtf(v[2 * j + 1] + p.unit_eps);
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        q[j][c] *= qs;
        k[j][c] *= ks;
      }
    }
    // mutual terms: w = g_{i+1} ... g_j k_i, extended token by token
    float co[16];
#pragma unroll
    for (int x = 0; x < 16; ++x) co[x] = 0.f;
#pragma unroll
    for (int i = 0; i < GRP; ++i) {
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        float w = k[i][c];
#pragma unroll
        for (int j = i; j < GRP; ++j) {
          if (j > i) {
            w *= g[j][c];
            co[j * (j - 1) / 2 + i] += k[j][c] * w;
          }
          co[6 + j * (j + 1) / 2 + i] += q[j][c] * w;
        }
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
      for (int x = 0; x < 16; ++x) co[x] += __shfl_xor_sync(0xffffffffu, co[x], o);
    float* r = rec + ((long long)s * p.H + h) * CH;
    if (on || pad) {
      float cum[4] = {1.f, 1.f, 1.f, 1.f}, tail[4] = {1.f, 1.f, 1.f, 1.f}, y[4];
#pragma unroll
      for (int j = 0; j < GRP; ++j) {
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          cum[c] *= g[j][c];
          y[c] = k[j][c] * cum[c];
        }
        stf4(r + j * DP + d, y);
#pragma unroll
        for (int c = 0; c < 4; ++c) y[c] = q[j][c] * cum[c];
        stf4(r + (GRP + j) * DP + d, y);
      }
      stf4(r + 12 * DP + d, cum);
#pragma unroll
      for (int j = GRP - 1; j >= 0; --j) {
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          y[c] = k[j][c] * tail[c];
          tail[c] *= g[j][c];
        }
        stf4(r + (8 + j) * DP + d, y);
      }
    }
    if (lane < COEF) {
      float mine = 0.f;
#pragma unroll
      for (int x = 0; x < 16; ++x) mine = lane == x ? co[x] : mine;
      const float bt = __shfl_sync(0x00ffffffu, beta, lane >= 16 && lane < 20 ? lane - 16 : 0);
      r[13 * DP + lane] = lane < 16 ? mine : lane < 20 ? bt : 0.f;
    }
  }
}

// ---- prefill: the recurrence --------------------------------------------------------------------------
__device__ __forceinline__ void cp_async4(void* smem, const void* gmem) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;\n" ::"r"(smem_u32(smem)), "l"(gmem));
}
__device__ __forceinline__ void cp_async16b(void* smem, const void* gmem) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(smem_u32(smem)), "l"(gmem));
}

constexpr int SCAN_TB = 16;      // tokens staged at a time

// LPC lanes share CPT neighbouring columns, each lane with DPL rows of them (row = 4 * (LPC * n + lane) + j);
// COLS columns per block.  Every value of q, k and g that a thread loads serves its CPT columns.
template <int DPL, int LPC, int CPT, int COLS, bool VEC>
__global__ void __launch_bounds__(COLS / CPT * LPC)
delta_scan_kernel(const float* qn, const float* kn, const float* kq, const float* vv, const float* g,
                  const float* beta, float* state, const int* cu, const int* start_pos, const long long* slots, int H,
                  int KVH, int dim, int vdim, float* o) {
  constexpr int DP = DPL * LPC, THREADS = COLS / CPT * LPC;
  extern __shared__ __align__(16) float sm[];
  // two buffers of [q TB*DP | k TB*DP | g TB*DP | v TB*COLS | beta TB | kq TB]
  constexpr int BUF = SCAN_TB * (3 * DP + COLS + 2);
  const int h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * COLS;
  const int hk = h / (H / KVH);
  const long long t0 = cu[b];
  const int len = cu[b + 1] - cu[b];
  if (len <= 0) return;
  const int col_l = threadIdx.x / LPC * CPT, lr = threadIdx.x % LPC;
  const int col = c0 + col_l;
  const long long slot = slots[b];
  float* Sg = state + ((slot * H + h) * dim) * (long long)vdim + col;

  for (int i = threadIdx.x; i < 2 * BUF; i += THREADS) sm[i] = 0.f;      // pad rows stay zero
  f2 s[CPT][DPL / 2];
  const bool fresh = start_pos[b] == 0;
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int n = 0; n < DPL; n += 2) {
      const int r = 4 * (LPC * (n / 4) + lr) + (n & 3);
      const bool have = !fresh && col + c < vdim;
      s[c][n / 2] = pack2(have && r < dim ? Sg[(long long)r * vdim + c] : 0.f,
                          have && r + 1 < dim ? Sg[(long long)(r + 1) * vdim + c] : 0.f);
    }
  __syncthreads();

  auto stage = [&](int blk) {
    float* buf = sm + (blk & 1) * BUF;
    const int first = blk * SCAN_TB, n = min(SCAN_TB, len - first);
    if constexpr (VEC) {
      const int per = dim / 4;
      for (int i = threadIdx.x; i < n * per; i += THREADS) {
        const int tt = i / per, d = (i % per) * 4;
        const long long t = t0 + first + tt;
        cp_async16b(buf + tt * DP + d, qn + (t * KVH + hk) * dim + d);
        cp_async16b(buf + SCAN_TB * DP + tt * DP + d, kn + (t * KVH + hk) * dim + d);
        cp_async16b(buf + 2 * SCAN_TB * DP + tt * DP + d, g + (t * H + h) * dim + d);
      }
    } else {
      for (int i = threadIdx.x; i < n * dim; i += THREADS) {
        const int tt = i / dim, d = i % dim;
        const long long t = t0 + first + tt;
        cp_async4(buf + tt * DP + d, qn + (t * KVH + hk) * dim + d);
        cp_async4(buf + SCAN_TB * DP + tt * DP + d, kn + (t * KVH + hk) * dim + d);
        cp_async4(buf + 2 * SCAN_TB * DP + tt * DP + d, g + (t * H + h) * dim + d);
      }
    }
    float* bv = buf + 3 * SCAN_TB * DP;
    for (int i = threadIdx.x; i < n * COLS; i += THREADS) {
      const int tt = i / COLS, c = i % COLS;
      if (c0 + c < vdim) cp_async4(bv + i, vv + ((t0 + first + tt) * H + h) * vdim + c0 + c);
    }
    float* bb = bv + SCAN_TB * COLS;
    for (int i = threadIdx.x; i < 2 * n; i += THREADS) {
      const int tt = i % n;
      if (i < n) cp_async4(bb + tt, beta + (t0 + first + tt) * H + h);
      else cp_async4(bb + SCAN_TB + tt, kq + (t0 + first + tt) * KVH + hk);
    }
    asm volatile("cp.async.commit_group;\n" ::);
  };

  const int blocks = (len + SCAN_TB - 1) / SCAN_TB;
  stage(0);
  for (int blk = 0; blk < blocks; ++blk) {
    if (blk + 1 < blocks) {
      stage(blk + 1);
      asm volatile("cp.async.wait_group 1;\n" ::);
    } else {
      asm volatile("cp.async.wait_group 0;\n" ::);
    }
    __syncthreads();
    const float* buf = sm + (blk & 1) * BUF;
    const int first = blk * SCAN_TB, n = min(SCAN_TB, len - first);
    const float* bv = buf + 3 * SCAN_TB * DP;
    const float* bb = bv + SCAN_TB * COLS;
    auto rows = [&](int which, int tt) {
      return reinterpret_cast<const ulonglong2*>(buf + (which * SCAN_TB + tt) * DP) + lr;
    };
#pragma unroll 2
    for (int tt = 0; tt < n; ++tt) {
      const ulonglong2 *q4 = rows(0, tt), *k4 = rows(1, tt), *g4 = rows(2, tt);
      const float bt = bb[tt], kqt = bb[SCAN_TB + tt];
      f2 kk[DPL / 2];
      f2 pk[CPT][2], pq[CPT][2];
#pragma unroll
      for (int c = 0; c < CPT; ++c) pk[c][0] = pk[c][1] = pq[c][0] = pq[c][1] = 0ull;
#pragma unroll
      for (int m = 0; m < DPL / 4; ++m) {
        const ulonglong2 gg = g4[m * LPC], kv = k4[m * LPC], qq = q4[m * LPC];
        kk[2 * m] = kv.x;
        kk[2 * m + 1] = kv.y;
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          s[c][2 * m] = mul2(s[c][2 * m], gg.x);
          s[c][2 * m + 1] = mul2(s[c][2 * m + 1], gg.y);
          pk[c][0] = fma2(s[c][2 * m], kv.x, pk[c][0]);
          pk[c][1] = fma2(s[c][2 * m + 1], kv.y, pk[c][1]);
          pq[c][0] = fma2(s[c][2 * m], qq.x, pq[c][0]);
          pq[c][1] = fma2(s[c][2 * m + 1], qq.y, pq[c][1]);
        }
      }
      float dk[CPT], dq[CPT];
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        const float2 k0 = unpack2(pk[c][0]), k1 = unpack2(pk[c][1]), q0 = unpack2(pq[c][0]), q1 = unpack2(pq[c][1]);
        dk[c] = (k0.x + k0.y) + (k1.x + k1.y);
        dq[c] = (q0.x + q0.y) + (q1.x + q1.y);
      }
#pragma unroll
      for (int x = LPC / 2; x > 0; x >>= 1) {
#pragma unroll
        for (int c = 0; c < CPT; ++c) dk[c] += __shfl_xor_sync(0xffffffffu, dk[c], x);
#pragma unroll
        for (int c = 0; c < CPT; ++c) dq[c] += __shfl_xor_sync(0xffffffffu, dq[c], x);
      }
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        const float u = bt * (bv[tt * COLS + col_l + c] - dk[c]);
        const f2 uu = pack2(u, u);
#pragma unroll
        for (int m = 0; m < DPL / 2; ++m) s[c][m] = fma2(kk[m], uu, s[c][m]);
        dq[c] += kqt * u;
      }
      // one lane per column writes it
      if (lr < CPT) {
        float mine = dq[0];
#pragma unroll
        for (int c = 1; c < CPT; ++c) mine = lr == c ? dq[c] : mine;
        if (col + lr < vdim) o[((t0 + first + tt) * H + h) * vdim + col + lr] = mine;
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int n = 0; n < DPL; n += 2) {
      const int r = 4 * (LPC * (n / 4) + lr) + (n & 3);
      const float2 v = unpack2(s[c][n / 2]);
      if (col + c < vdim && r < dim) Sg[(long long)r * vdim + c] = v.x;
      if (col + c < vdim && r + 1 < dim) Sg[(long long)(r + 1) * vdim + c] = v.y;
    }
}

// ---- prefill: the recurrence over groups of four tokens ------------------------------------------------
// Lane layout of delta_scan_kernel with sixteen lanes on four neighbouring columns: what a thread reads of a record
// serves four columns.  A group costs one pass over the state for its eight dot products and one for its four
// writes, and one exchange between lanes.
constexpr int SG = 2;            // groups staged at a time

template <int DPL, int COLS>
__global__ void __launch_bounds__(COLS * 4)
delta_group_scan_kernel(const float* rec, const float* vv, float* state, const int* cu, const int* start_pos,
                        const long long* slots, int H, int dim, int vdim, float* o) {
  constexpr int LPC = 16, CPT = 4, DP = DPL * LPC, THREADS = COLS / CPT * LPC, CH = group_floats(DP);
  constexpr int BUF = SG * (CH + GRP * COLS);
  extern __shared__ __align__(16) float sm[];            // two buffers of SG x [record | v of four tokens]
  const int h = blockIdx.y, b = blockIdx.z, c0 = blockIdx.x * COLS;
  const long long t0 = cu[b];
  const int len = cu[b + 1] - cu[b];
  if (len <= 0) return;
  const int col_l = threadIdx.x / LPC * CPT, lr = threadIdx.x % LPC, col = c0 + col_l;
  const float* rb = rec + ((long long)(cu[b] / GRP + b) * H + h) * CH;
  float* Sg = state + ((slots[b] * H + h) * dim) * (long long)vdim + col;
  const bool fresh = start_pos[b] == 0;
  f2 s[CPT][DPL / 2];
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int n = 0; n < DPL; n += 2) {
      const int r = 4 * (LPC * (n / 4) + lr) + (n & 3);
      const bool have = !fresh && col + c < vdim;
      s[c][n / 2] = pack2(have && r < dim ? Sg[(long long)r * vdim + c] : 0.f,
                          have && r + 1 < dim ? Sg[(long long)(r + 1) * vdim + c] : 0.f);
    }
  for (int i = threadIdx.x; i < 2 * BUF; i += THREADS) sm[i] = 0.f;      // columns past vdim, missing tokens: finite
  __syncthreads();

  const int groups = (len + GRP - 1) / GRP, rounds = (groups + SG - 1) / SG;
  auto stage = [&](int rd) {
    float* buf = sm + (rd & 1) * BUF;
#pragma unroll
    for (int x = 0; x < SG; ++x) {
      const int gi = rd * SG + x;
      if (gi < groups) {
        const float* src = rb + (long long)gi * H * CH;
        float* dst = buf + x * (CH + GRP * COLS);
        for (int i = threadIdx.x; i < CH / 4; i += THREADS) cp_async16b(dst + i * 4, src + i * 4);
        for (int i = threadIdx.x; i < GRP * COLS / 4; i += THREADS) {
          const int tt = i / (COLS / 4), c = (i % (COLS / 4)) * 4;
          if (gi * GRP + tt < len && c0 + c < vdim)
            cp_async16b(dst + CH + tt * COLS + c, vv + ((t0 + gi * GRP + tt) * H + h) * vdim + c0 + c);
        }
      }
    }
    asm volatile("cp.async.commit_group;\n" ::);
  };

  stage(0);
  for (int rd = 0; rd < rounds; ++rd) {
    if (rd + 1 < rounds) {
      stage(rd + 1);
      asm volatile("cp.async.wait_group 1;\n" ::);
    } else {
      asm volatile("cp.async.wait_group 0;\n" ::);
    }
    __syncthreads();
#pragma unroll
    for (int x = 0; x < SG; ++x) {
      const int gi = rd * SG + x;
      if (gi >= groups) break;
      const float* r = sm + (rd & 1) * BUF + x * (CH + GRP * COLS);
      const float* co = r + 13 * DP;
      auto rows = [&](int which) { return reinterpret_cast<const ulonglong2*>(r + which * DP) + lr; };
      f2 acc[2 * GRP][CPT];                              // r_0 .. r_3, p_0 .. p_3
#pragma unroll
      for (int v = 0; v < 2 * GRP; ++v)
#pragma unroll
        for (int c = 0; c < CPT; ++c) acc[v][c] = 0ull;
#pragma unroll
      for (int m = 0; m < DPL / 4; ++m)
#pragma unroll
        for (int v = 0; v < 2 * GRP; ++v) {
          const ulonglong2 w = rows(v)[m * LPC];
#pragma unroll
          for (int c = 0; c < CPT; ++c) {
            acc[v][c] = fma2(s[c][2 * m], w.x, acc[v][c]);
            acc[v][c] = fma2(s[c][2 * m + 1], w.y, acc[v][c]);
          }
        }
      // sums over the sixteen lanes: lane l ends with value l / 2 of columns 2 (l % 2) and 2 (l % 2) + 1
      float val[2 * GRP][CPT];
#pragma unroll
      for (int v = 0; v < 2 * GRP; ++v)
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          const float2 t = unpack2(acc[v][c]);
          val[v][c] = t.x + t.y;
        }
#pragma unroll
      for (int half = 4; half > 0; half >>= 1) {
        const bool up = lr & (2 * half);
#pragma unroll
        for (int v = 0; v < half; ++v)
#pragma unroll
          for (int c = 0; c < CPT; ++c) {
            const float mine = up ? val[v + half][c] : val[v][c], theirs = up ? val[v][c] : val[v + half][c];
            val[v][c] = mine + __shfl_xor_sync(0xffffffffu, theirs, 2 * half);
          }
      }
      float two[2];
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const float mine = lr & 1 ? val[0][c + 2] : val[0][c], theirs = lr & 1 ? val[0][c] : val[0][c + 2];
        two[c] = mine + __shfl_xor_sync(0xffffffffu, theirs, 1);
      }
      // every lane solves for the four writes
      float u[GRP][CPT];
#pragma unroll
      for (int j = 0; j < GRP; ++j) {
        const float bt = co[16 + j];
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          float t = r[CH + j * COLS + col_l + c] - __shfl_sync(0xffffffffu, two[c & 1], 2 * j + (c >> 1), LPC);
#pragma unroll
          for (int i = 0; i < j; ++i) t -= co[j * (j - 1) / 2 + i] * u[i][c];
          u[j][c] = bt * t;
        }
      }
#pragma unroll
      for (int m = 0; m < DPL / 4; ++m) {
        const ulonglong2 ga = rows(12)[m * LPC];
#pragma unroll
        for (int c = 0; c < CPT; ++c) {
          s[c][2 * m] = mul2(s[c][2 * m], ga.x);
          s[c][2 * m + 1] = mul2(s[c][2 * m + 1], ga.y);
        }
#pragma unroll
        for (int j = 0; j < GRP; ++j) {
          const ulonglong2 w = rows(8 + j)[m * LPC];
#pragma unroll
          for (int c = 0; c < CPT; ++c) {
            const f2 uu = pack2(u[j][c], u[j][c]);
            s[c][2 * m] = fma2(w.x, uu, s[c][2 * m]);
            s[c][2 * m + 1] = fma2(w.y, uu, s[c][2 * m + 1]);
          }
        }
      }
      // lanes 8 + 2 j and 9 + 2 j hold p_j and write token j
      const int j = lr / 2 - GRP, cp = 2 * (lr & 1);
      if (j >= 0 && gi * GRP + j < len) {
        const float* bj = co + 6 + j * (j + 1) / 2;
#pragma unroll
        for (int i = 0; i < GRP; ++i)
          if (i <= j) {
            const float w = bj[i];
            two[0] += w * (cp ? u[i][2] : u[i][0]);
            two[1] += w * (cp ? u[i][3] : u[i][1]);
          }
        float* dst = o + ((t0 + gi * GRP + j) * H + h) * vdim + col + cp;
        if (col + cp + 1 < vdim) *reinterpret_cast<float2*>(dst) = make_float2(two[0], two[1]);   // vdim % 4 == 0
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int c = 0; c < CPT; ++c)
#pragma unroll
    for (int n = 0; n < DPL; n += 2) {
      const int r = 4 * (LPC * (n / 4) + lr) + (n & 3);
      const float2 v = unpack2(s[c][n / 2]);
      if (col + c < vdim && r < dim) Sg[(long long)r * vdim + c] = v.x;
      if (col + c < vdim && r + 1 < dim) Sg[(long long)(r + 1) * vdim + c] = v.y;
    }
}

// ---- prefill: norm and gate ------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
delta_out_kernel(const DeltaIn<T> p, const float* o, const T* gate, long long gate_ld, const float* norm, float eps, T* y, long long rows,
                 int H, int vdim) {
  const long long r = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);     // (token, head)
  const int lane = threadIdx.x & 31;
  if (r >= rows) return;
  const long long t = r / H;
  const int h = (int)(r % H);
  const float* x = o + r * vdim;
  float ss = 0.f;
  for (int c = lane; c < vdim; c += 32) ss += x[c] * x[c];
  const float inv = 1.f / sqrtf(warp_sum(ss) / (float)vdim + eps);
  for (int c = lane; c < vdim; c += 32)
    stf(y + r * vdim + c, x[c] * inv * norm[c] * p.gate_of(ldf(gate + t * gate_ld + h * vdim + c)));
}

// ---- decode: one token per sequence, everything in one kernel -----------------------------------------------
// block = (head, sequence).  Threads tile the state as [row groups RG][column groups of V]; a thread keeps its
// NI row slices in registers between the decayed dot products and the rank-one update.
template <typename T, int V, int NI, int THREADS, int TAPS>
__global__ void __launch_bounds__(THREADS, NI * V <= 32 && THREADS == 512 ? 2 : 1)
delta_decode_kernel(const DeltaIn<T> p, const T* gate, long long gate_ld, const float* norm, float eps,
                    const int* positions, const long long* slots, T* y) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  __shared__ float scal[3];
  const int h = blockIdx.x, b = blockIdx.y;
  const long long slot = slots[b];
  if (slot < 0) return;
  const int dim = p.dim, vdim = p.vdim, kd = p.KVH * dim, channels = 2 * kd + p.H * vdim;
  const int rep = p.H / p.KVH, hk = h / rep;
  const int pos = positions[b];
  const int CW = vdim / V, RG = THREADS / CW;
  float* sq = sm;
  float* sk = sq + dim;
  float* sg = sk + dim;
  float* sv = sg + dim;
  float* su = sv + vdim;
  float* so = su + vdim;
  float* part = so + vdim;                       // [RG][2][vdim]
  const int rg = threadIdx.x / CW, cg = threadIdx.x % CW;
  const bool on = rg < RG;
  float* S = p.state + ((slot * p.H + h) * dim) * (long long)vdim + cg * V;
  float s[NI][4];
#pragma unroll
  for (int n = 0; n < NI; ++n) {
    const int r = rg + n * RG;
#pragma unroll
    for (int j = 0; j < 4; ++j) s[n][j] = 0.f;
    if (on && r < dim && pos > 0) ldv<V>(S + (long long)r * vdim, s[n]);
  }
  const bool lead = h % rep == 0;                // writes the key head's ring entries
  T* ring = p.ring + (slot * p.taps + pos % p.taps) * channels;
  const T* row = p.proj + (long long)b * p.ld;
  // q | k | v channels of this head side by side, one per thread
  for (int x = threadIdx.x; x < 2 * dim + vdim; x += THREADS) {
    const int d = x < dim ? x : x < 2 * dim ? x - dim : x - 2 * dim;
    const int ch = x < 2 * dim ? hk * dim + d : h * vdim + d;
    const int base = x < dim ? 0 : x < 2 * dim ? kd : 2 * kd;
    const int col = (x < dim ? p.q_col : x < 2 * dim ? p.k_col : p.v_col) + ch;
    (x < dim ? sq : x < 2 * dim ? sk : sv)[d] = conv_silu<TAPS>(p, b, 0, pos, slot, col, base + ch);
    if (lead || x >= 2 * dim) ring[base + ch] = row[col];
  }
  for (int d = threadIdx.x; d < dim; d += THREADS)
    sg[d] = p.decay(b, h, d);
  __syncthreads();
  {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (warp < 3) {
      const float* x = warp == 1 ? sk : sq;
      const float* z = warp == 0 ? sq : sk;
      float a = 0.f;
      for (int d = lane; d < dim; d += 32) a += x[d] * z[d];
      a = warp_sum(a);
      if (lane == 0) scal[warp] = a;
    }
  }
  float pk[4] = {0.f, 0.f, 0.f, 0.f}, pq[4] = {0.f, 0.f, 0.f, 0.f};
  if (on) {
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const int r = rg + n * RG;
      if (r < dim) {
        const float gr = sg[r], kr = sk[r], qr = sq[r];
#pragma unroll
        for (int j = 0; j < V; ++j) {
          s[n][j] *= gr;
          pk[j] += s[n][j] * kr;
          pq[j] += s[n][j] * qr;
        }
      }
    }
    stv<V>(part + (rg * 2 + 0) * vdim + cg * V, pk);
    stv<V>(part + (rg * 2 + 1) * vdim + cg * V, pq);
  }
  __syncthreads();
  const float qs = 1.f / (sqrtf(scal[0] + p.unit_eps) * sqrtf((float)dim)), ks = 1.f / sqrtf(scal[1] + p.unit_eps);
  const float kq = scal[2] * qs * ks;
  const float beta = sigmoid_f(ldf(row + p.b_col + h));
  float ss = 0.f;
  for (int c = threadIdx.x; c < vdim; c += THREADS) {
    float dk = 0.f, dq = 0.f;
    for (int r = 0; r < RG; ++r) {
      dk += part[(r * 2 + 0) * vdim + c];
      dq += part[(r * 2 + 1) * vdim + c];
    }
    const float u = beta * (sv[c] - dk * ks);
    const float oc = dq * qs + kq * u;
    su[c] = u * ks;
    so[c] = oc;
    ss += oc * oc;
  }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)vdim + eps);     // also orders su before the reads below
  if (on) {
    float u[4];
    ldv<V>(su + cg * V, u);
#pragma unroll
    for (int n = 0; n < NI; ++n) {
      const int r = rg + n * RG;
      if (r < dim) {
        const float kr = sk[r];
#pragma unroll
        for (int j = 0; j < V; ++j) s[n][j] += kr * u[j];
        stv<V>(S + (long long)r * vdim, s[n]);
      }
    }
  }
  for (int c = threadIdx.x; c < vdim; c += THREADS)
    stf(y + ((long long)b * p.H + h) * vdim + c,
        so[c] * inv * norm[c] * p.gate_of(ldf(gate + b * gate_ld + h * vdim + c)));
}

}  // namespace msrl

using namespace msrl;

// ints: taps, H, KVH, dim, vdim, q_col, k_col, v_col, b_col, one decay per head, silu gate
template <typename T>
static DeltaIn<T> delta_in(const void* proj, long long ld, const void* a, long long a_ld, const float* conv,
                           const float* a_log, const float* dt_bias, void* ring, float* state, const int* ints,
                           float unit_eps) {
  DeltaIn<T> p{};
  p.proj = (const T*)proj;
  p.ld = ld;
  p.a = (const T*)a;
  p.a_ld = a_ld;
  p.conv = conv;
  p.a_log = a_log;
  p.dt_bias = dt_bias;
  p.ring = (T*)ring;
  p.state = state;
  p.taps = ints[0];
  p.H = ints[1];
  p.KVH = ints[2];
  p.dim = ints[3];
  p.vdim = ints[4];
  p.q_col = ints[5];
  p.k_col = ints[6];
  p.v_col = ints[7];
  p.b_col = ints[8];
  p.a_h = ints[9] ? 1 : p.dim;
  p.a_d = ints[9] ? 0 : 1;
  p.silu_gate = ints[10];
  p.channels = 2 * p.KVH * p.dim + p.H * p.vdim;
  p.unit_eps = unit_eps;
  return p;
}

template <typename F>
static int allow_smem(F* kernel, size_t bytes) {
  if (bytes <= 48 * 1024) return 0;
  return (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}

template <int DPL, int LPC, int CPT, int COLS>
static int launch_scan(const float* qn, const float* kn, const float* kq, const float* vv, const float* g,
                       const float* beta, float* state, const int* cu, const int* start_pos, const long long* slots,
                       int batch, int H, int KVH, int dim, int vdim, float* o, cudaStream_t st) {
  const size_t smem = 2 * sizeof(float) * SCAN_TB * (3 * DPL * LPC + COLS + 2);
  const dim3 grid((unsigned)((vdim + COLS - 1) / COLS), (unsigned)H, (unsigned)batch);
  if (dim % 4 == 0) {
    const int e = allow_smem(delta_scan_kernel<DPL, LPC, CPT, COLS, true>, smem);
    if (e) return e;
    delta_scan_kernel<DPL, LPC, CPT, COLS, true><<<grid, COLS / CPT * LPC, smem, st>>>(qn, kn, kq, vv, g, beta, state, cu,
                                                                            start_pos, slots, H, KVH, dim, vdim, o);
  } else {
    const int e = allow_smem(delta_scan_kernel<DPL, LPC, CPT, COLS, false>, smem);
    if (e) return e;
    delta_scan_kernel<DPL, LPC, CPT, COLS, false><<<grid, COLS / CPT * LPC, smem, st>>>(qn, kn, kq, vv, g, beta, state, cu,
                                                                             start_pos, slots, H, KVH, dim, vdim, o);
  }
  return (int)cudaGetLastError();
}

template <int DPL>
static int launch_group_scan(const float* rec, const float* vv, float* state, const int* cu, const int* start_pos,
                             const long long* slots, int batch, int H, int dim, int vdim, float* o, cudaStream_t st) {
  constexpr int COLS = 32;
  const size_t smem = 2 * sizeof(float) * SG * (group_floats(DPL * 16) + GRP * COLS);
  const int e = allow_smem(delta_group_scan_kernel<DPL, COLS>, smem);
  if (e) return e;
  const dim3 grid((unsigned)((vdim + COLS - 1) / COLS), (unsigned)H, (unsigned)batch);
  delta_group_scan_kernel<DPL, COLS><<<grid, COLS * 4, smem, st>>>(rec, vv, state, cu, start_pos, slots, H, dim, vdim, o);
  return (int)cudaGetLastError();
}

// the shapes of the grouped path (four channels per lane, at most four taps)
static bool grouped_shape(const int* ints, long long ld, long long a_ld) {
  const int taps = ints[0], dim = ints[3], vdim = ints[4];
  return dim % 4 == 0 && dim <= 128 && vdim % 4 == 0 && taps >= 2 && taps <= 4 && ints[5] % 4 == 0 && ints[6] % 4 == 0 &&
         ints[7] % 4 == 0 && ld % 4 == 0 && (ints[9] || a_ld % 4 == 0);
}
static int padded_dim(int dim) { return dim <= 64 ? 64 : 128; }

// fp32 scratch of msrl_delta_prefill
MSRL_API long long msrl_delta_prefill_scratch(const int* ints, long long ld, long long a_ld, int tokens, int batch) {
  const long long H = ints[1], KVH = ints[2], dim = ints[3], vdim = ints[4], t = tokens;
  if (grouped_shape(ints, ld, a_ld))
    return 8 + 2 * t * H * vdim + (t / GRP + batch) * H * group_floats(padded_dim((int)dim));
  return 2 * t * H * vdim + 2 * t * KVH * dim + t * H * dim + t * (KVH + H) + 64;
}

MSRL_API int msrl_delta_prefill(const void* proj, long long ld, const void* a, long long a_ld, const float* conv,
                                const float* a_log, const float* dt_bias, void* ring, float* state, const int* ints,
                                float unit_eps, const void* gate, long long gate_ld, const float* norm, float eps,
                                const int* tok_seq, const int* cu, const int* start_pos, const long long* slots,
                                int tokens, int batch, float* scratch, void* y, int is_f32, cudaStream_t st) {
  if (tokens == 0 || batch == 0) return 0;
  const int H = ints[1], KVH = ints[2], dim = ints[3], vdim = ints[4];
  if (dim > DELTA_MAX_DIM || H % KVH != 0 || batch > 65535 || H > 65535) return (int)cudaErrorInvalidValue;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const DeltaIn<T> p = delta_in<T>(proj, ld, a, a_ld, conv, a_log, dt_bias, ring, state, ints, unit_eps);
    auto up4 = [](long long n) { return (n + 3) / 4 * 4; };       // every array starts on 16 bytes
    const long long nv = up4((long long)tokens * H * vdim);
    float *vv = scratch, *o = vv + nv;
    int e;
    const int gslots = tokens / GRP + batch;
    const dim3 vgrid((unsigned)((H * vdim + 1023) / 1024), (unsigned)((tokens + PREP_TT - 1) / PREP_TT));
    const dim3 ggrid((unsigned)((H + 7) / 8), (unsigned)((gslots + 3) / 4));
    if (grouped_shape(ints, ld, a_ld) && vgrid.y <= 65535 && ggrid.y <= 65535) {
      float* rec = o + nv;
      const int DP = padded_dim(dim);
#define MSRL_PREP(N)                                                                                       \
  do {                                                                                                     \
    delta_value_kernel<T, N><<<vgrid, 256, 0, st>>>(p, tok_seq, cu, start_pos, slots, tokens, vv);           \
    if (ints[9]) delta_group_kernel<T, N, true><<<ggrid, 256, 0, st>>>(p, cu, start_pos, slots, batch, gslots, DP, rec); \
    else delta_group_kernel<T, N, false><<<ggrid, 256, 0, st>>>(p, cu, start_pos, slots, batch, gslots, DP, rec);        \
  } while (0)
      if (p.taps == 4) MSRL_PREP(4);
      else if (p.taps == 3) MSRL_PREP(3);
      else MSRL_PREP(2);
#undef MSRL_PREP
      if (DP == 64) e = launch_group_scan<4>(rec, vv, state, cu, start_pos, slots, batch, H, dim, vdim, o, st);
      else e = launch_group_scan<8>(rec, vv, state, cu, start_pos, slots, batch, H, dim, vdim, o, st);
    } else {
      const long long nk = up4((long long)tokens * KVH * dim);
      float *qn = o + nv, *kn = qn + nk, *g = kn + nk, *beta = g + up4((long long)tokens * H * dim), *kq = beta + up4((long long)tokens * H);
      delta_prep_kernel<T><<<tokens, 256, 0, st>>>(p, tok_seq, cu, start_pos, slots, qn, kn, kq, vv, g, beta);
#define MSRL_SCAN(D, L, C, N) launch_scan<D, L, C, N>(qn, kn, kq, vv, g, beta, state, cu, start_pos, slots, batch, H, KVH, dim, vdim, o, st)
      if (dim <= 32) e = MSRL_SCAN(8, 4, 1, 32);
      else if (dim <= 64) e = MSRL_SCAN(8, 8, 2, 32);
      else if (dim <= 128) e = MSRL_SCAN(16, 8, 2, 32);
      else e = MSRL_SCAN(32, 8, 1, 32);
#undef MSRL_SCAN
    }
    if (e) return e;
    conv_ring_kernel<T><<<dim3((unsigned)((p.channels + 255) / 256), (unsigned)batch), 256, 0, st>>>(
        p, KVH * dim, KVH * dim, p.q_col, p.k_col, p.v_col, cu, start_pos, slots);
    const long long rows = (long long)tokens * H;
    delta_out_kernel<T><<<(unsigned)((rows + 7) / 8), 256, 0, st>>>(p, o, (const T*)gate, gate_ld, norm, eps, (T*)y, rows, H, vdim);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

template <typename T, int V, int NI, int THREADS, int TAPS>
static int launch_delta_decode_taps(const DeltaIn<T>& p, const T* gate, long long gate_ld, const float* norm, float eps,
                               const int* positions, const long long* slots, T* y, int batch, cudaStream_t st) {
  const int rg = THREADS / (p.vdim / V);
  const size_t smem = sizeof(float) * (3 * (size_t)p.dim + 3 * (size_t)p.vdim + 2 * (size_t)rg * p.vdim);
  const int e = allow_smem(delta_decode_kernel<T, V, NI, THREADS, TAPS>, smem);
  if (e) return e;
  delta_decode_kernel<T, V, NI, THREADS, TAPS><<<dim3((unsigned)p.H, (unsigned)batch), THREADS, smem, st>>>(
      p, gate, gate_ld, norm, eps, positions, slots, y);
  return (int)cudaGetLastError();
}

template <typename T, int V, int NI, int THREADS>
static int launch_delta_decode(const DeltaIn<T>& p, const T* gate, long long gate_ld, const float* norm, float eps,
                               const int* positions, const long long* slots, T* y, int batch, cudaStream_t st) {
  if constexpr (V == 4 && NI <= 8) {
    if (p.taps == 4)
      return launch_delta_decode_taps<T, V, NI, THREADS, 4>(p, gate, gate_ld, norm, eps, positions, slots, y, batch, st);
    if (p.taps == 3)
      return launch_delta_decode_taps<T, V, NI, THREADS, 3>(p, gate, gate_ld, norm, eps, positions, slots, y, batch, st);
    if (p.taps == 2)
      return launch_delta_decode_taps<T, V, NI, THREADS, 2>(p, gate, gate_ld, norm, eps, positions, slots, y, batch, st);
  }
  return launch_delta_decode_taps<T, V, NI, THREADS, 0>(p, gate, gate_ld, norm, eps, positions, slots, y, batch, st);
}

template <typename T, int V>
static int pick_delta_decode(const DeltaIn<T>& p, const T* gate, long long gate_ld, const float* norm, float eps,
                             const int* positions, const long long* slots, T* y, int batch, cudaStream_t st) {
  // the smallest block that keeps few row slices per thread: registers for two blocks of 512 threads on an SM
  auto slices = [&](int threads) {
    const int rg = threads / (p.vdim / V);
    return rg == 0 ? 1 << 20 : (p.dim + rg - 1) / rg;
  };
#define MSRL_TRY(NI, THREADS) \
  if (slices(THREADS) <= NI)  \
    return launch_delta_decode<T, V, NI, THREADS>(p, gate, gate_ld, norm, eps, positions, slots, y, batch, st);
  MSRL_TRY(4, 128)
  MSRL_TRY(4, 256)
  MSRL_TRY(8, 128)
  MSRL_TRY(8, 256)
  MSRL_TRY(8, 512)
  MSRL_TRY(16, 512)
  MSRL_TRY(16, 1024)
  MSRL_TRY(64, 512)
#undef MSRL_TRY
  return (int)cudaErrorInvalidValue;
}

MSRL_API int msrl_delta_decode(const void* proj, long long ld, const void* a, long long a_ld, const float* conv,
                               const float* a_log, const float* dt_bias, void* ring, float* state, const int* ints,
                               float unit_eps, const void* gate, long long gate_ld, const float* norm, float eps,
                               const int* positions, const long long* slots, int batch, void* y, int is_f32,
                               cudaStream_t st) {
  if (batch == 0) return 0;
  if (ints[3] > DELTA_MAX_DIM || ints[1] % ints[2] != 0 || batch > 65535) return (int)cudaErrorInvalidValue;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    const DeltaIn<T> p = delta_in<T>(proj, ld, a, a_ld, conv, a_log, dt_bias, ring, state, ints, unit_eps);
    return p.vdim % 4 == 0
               ? pick_delta_decode<T, 4>(p, (const T*)gate, gate_ld, norm, eps, positions, slots, (T*)y, batch, st)
               : pick_delta_decode<T, 1>(p, (const T*)gate, gate_ld, norm, eps, positions, slots, (T*)y, batch, st);
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}
