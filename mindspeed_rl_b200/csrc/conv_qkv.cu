// Between the q | k | v projection and grouped-head attention, everything in fp32:
//
//   x  <- causal convolution over time, one filter per channel (short_conv.cuh)
//   q, k <- x / sqrt(mean over the head of x^2 + eps) * weight, then rotation of the first `rot` entries of the head,
//           entry 2i with entry 2i + 1;   v <- x
//
// Prepared rows hold the heads padded (qp, vp; pad entries are written as zeros), and so do the cache rows of k and v.
// Prompt portions are followed by conv_ring_kernel; a decode step (one token per sequence) writes its ring entry itself.
//
//   conv_qkv4_kernel, conv_qkv4_step_kernel   heads of up to 128 entries, sizes and columns multiples of 4, 2 to 4 taps: a
//                      warp walks consecutive tokens of one head with the convolution windows in registers, four
//                      channels per lane; in decode steps it takes one token
//   conv_qkv_kernel    any sizes: a warp per token and head, every entry convolved where it is needed
#include "short_conv.cuh"

namespace msrl {

template <typename T>
struct ConvQkvArgs : ConvIn<T> {
  int H, G, dim, vdim, qp, vp;
  int q_col, k_col, v_col;               // in proj
  int oq, ok, ov;                        // in out
  T* out;                                // prepared rows; decode steps: query heads only
  long long out_ld;
  const float *q_norm, *k_norm;
  float eps;
  const float* table;                    // [table_rows, rot]: cos | sin
  int rot, table_rows;
  const int* positions;
  const long long* slots;                // cache row per token, < 0: not cached
  T *k_cache, *v_cache;                  // [rows, G, qp], [rows, G, vp]
  const long long* state_slots;          // per sequence, < 0: none
  const int *tok_seq, *cu, *start_pos;   // null in decode steps
  int tokens;
};

// one head of q, k or v: where it is read, where it goes
template <typename T>
struct HeadOf {
  int size, pad, col, ch, h;
  bool is_q, is_v;
  __device__ __forceinline__ HeadOf(const ConvQkvArgs<T>& p, int u) {
    is_q = u < p.H;
    is_v = u >= p.H + p.G;
    h = is_q ? u : is_v ? u - p.H - p.G : u - p.H;
    size = is_v ? p.vdim : p.dim;
    pad = is_v ? p.vp : p.qp;
    col = (is_q ? p.q_col : is_v ? p.v_col : p.k_col) + h * size;
    ch = (is_q ? 0 : is_v ? (p.H + p.G) * p.dim : p.H * p.dim) + h * size;
  }
  __device__ __forceinline__ T* row(const ConvQkvArgs<T>& p, long long t) const {
    if (p.cu == nullptr && !is_q) return nullptr;
    return p.out + t * p.out_ld + (is_q ? p.oq : is_v ? p.ov : p.ok) + h * pad;
  }
  __device__ __forceinline__ T* cached(const ConvQkvArgs<T>& p, long long slot) const {
    return is_q || slot < 0 ? nullptr : (is_v ? p.v_cache : p.k_cache) + (slot * p.G + h) * pad;
  }
};

constexpr int CQ_TT = 32, CQ_U = 4;      // tokens per warp (one a lane looks up), tokens in flight together

template <typename T>
__device__ __forceinline__ float inv_rms(float ss, float inv_n, float eps) {
  if constexpr (sizeof(T) == 2) return rsqrtf(fmaf(ss, inv_n, eps));     // within 2^-22, far below the rounding of the result
  else return 1.f / sqrtf(ss * inv_n + eps);
}

// cosines and sines of the two pairs from entry d on (a multiple of 4, below rot)
__device__ __forceinline__ void pair_angles(const float* row, int d, int rot, float (&cs)[4]) {
  const float* tab = row + (d >> 1);
  if (rot % 4 == 0) {
    const float2 a = *reinterpret_cast<const float2*>(tab), b = *reinterpret_cast<const float2*>(tab + (rot >> 1));
    cs[0] = a.x; cs[1] = a.y; cs[2] = b.x; cs[3] = b.y;
  } else {
    const bool two = d + 2 < rot;
    cs[0] = tab[0];
    cs[1] = two ? tab[1] : 1.f;
    cs[2] = tab[rot >> 1];
    cs[3] = two ? tab[(rot >> 1) + 1] : 0.f;
  }
}
__device__ __forceinline__ void turn_pairs(float (&y)[4], const float (&cs)[4]) {
#pragma unroll
  for (int c = 0; c < 2; ++c) {
    const float a = y[2 * c], b = y[2 * c + 1];
    y[2 * c] = a * cs[c] - b * cs[2 + c];
    y[2 * c + 1] = b * cs[c] + a * cs[2 + c];
  }
}

// Sums over the warp of four values per lane: lanes 8 n to 8 n + 7 end with the sum of value n.
__device__ __forceinline__ float sum_of_four(const float (&v)[4], int lane) {
  float two[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const float keep = lane & 16 ? v[2 + i] : v[i], give = lane & 16 ? v[i] : v[2 + i];
    two[i] = keep + __shfl_xor_sync(0xffffffffu, give, 16);
  }
  const float keep = lane & 8 ? two[1] : two[0], give = lane & 8 ? two[0] : two[1];
  float s = keep + __shfl_xor_sync(0xffffffffu, give, 8);
#pragma unroll
  for (int o = 4; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
  return s;
}

// prompt portions: the tokens of a sequence follow one another from start_pos on
template <typename T, int TAPS>
__global__ void __launch_bounds__(256, 3) conv_qkv4_kernel(const ConvQkvArgs<T> p) {
  const int u = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, d = lane * 4;
  if (u >= p.H + 2 * p.G) return;
  const HeadOf<T> hd(p, u);
  const int t0 = blockIdx.y * CQ_TT, t1 = min(p.tokens, t0 + CQ_TT);
  const bool on = d < hd.size, wr = d < hd.pad, turned = on && !hd.is_v && d < p.rot;
  ConvWindow<TAPS, T> cv;
  float w[4] = {0.f, 0.f, 0.f, 0.f};
  if (on) {
    cv.weights(p.conv, hd.ch + d);
    if (!hd.is_v) ldf4((hd.is_q ? p.q_norm : p.k_norm) + d, w);
  }
  const float inv_n = 1.f / (float)p.dim;
  T* cache = hd.is_q ? nullptr : (hd.is_v ? p.v_cache : p.k_cache) + hd.h * hd.pad + d;
  const int cache_row = p.G * hd.pad;
  const int mine = min(t0 + lane, t1 - 1), my_slot = hd.is_q ? -1 : (int)p.slots[mine];
  for (int ts = t0; ts < t1;) {                          // the sequences of this run, one after the other
    const int b = p.tok_seq[ts], first = p.cu[b], te = min(t1, p.cu[b + 1]);
    int pos = p.start_pos[b] + ts - first;
    if (on) cv.fill(p, ts, ts - first, pos, p.state_slots[b], hd.col + d, hd.ch + d);
    const T* src = p.proj + ts * p.ld + hd.col + d;
    T* out = hd.row(p, ts) + d;
    for (int tb = ts; tb < te; tb += CQ_U) {
      const int last = te - 1 - tb;                      // what is computed past it is not written
      float y[CQ_U][4];
#pragma unroll
      for (int n = 0; n < CQ_U; ++n) {
#pragma unroll
        for (int c = 0; c < 4; ++c) y[n][c] = 0.f;
        if (on && n <= last) ldf4(src + n * p.ld, y[n]);
      }
      if (on) cv.template steps<CQ_U>(y);
      if (!hd.is_v) {
        float ss[CQ_U];
#pragma unroll
        for (int n = 0; n < CQ_U; ++n) ss[n] = y[n][0] * y[n][0] + y[n][1] * y[n][1] + y[n][2] * y[n][2] + y[n][3] * y[n][3];
        const float inv = inv_rms<T>(sum_of_four(ss, lane), inv_n, p.eps);      // of token lane / 8
#pragma unroll
        for (int n = 0; n < CQ_U; ++n) {
          const float r = __shfl_sync(0xffffffffu, inv, n * 8);
#pragma unroll
          for (int c = 0; c < 4; ++c) y[n][c] *= r * w[c];
          if (turned) {
            float cs[4];
            pair_angles(p.table + min(pos + n, p.table_rows - 1) * p.rot, d, p.rot, cs);
            turn_pairs(y[n], cs);
          }
        }
        pos += CQ_U;
      }
#pragma unroll
      for (int n = 0; n < CQ_U; ++n) {
        const int slot = hd.is_q ? -1 : __shfl_sync(0xffffffffu, my_slot, tb - t0 + min(n, last));
        if (n <= last && wr) {
          stf4(out + n * p.out_ld, y[n]);
          if (slot >= 0) stf4(cache + (long long)slot * cache_row, y[n]);
        }
      }
      src += CQ_U * p.ld;
      out += CQ_U * p.out_ld;
    }
    ts = te;
  }
}

// decode: one token per sequence, a warp per head
template <typename T, int TAPS>
__global__ void __launch_bounds__(256) conv_qkv4_step_kernel(const ConvQkvArgs<T> p) {
  const int u = blockIdx.x * 8 + (threadIdx.x >> 5), d = (threadIdx.x & 31) * 4;
  if (u >= p.H + 2 * p.G) return;
  const HeadOf<T> hd(p, u);
  const long long t = blockIdx.y, state = p.state_slots[t], slot = p.slots[t];
  const int pos = p.positions[t];
  const bool on = d < hd.size;
  float y[4] = {0.f, 0.f, 0.f, 0.f}, x[4], cs[4];
  if (on) {
    ConvWindow<TAPS, T> cv;
    ldf4(p.proj + t * p.ld + hd.col + d, x);
    cv.weights(p.conv, hd.ch + d);
    cv.fill(p, t, 0, state < 0 ? 0 : pos, state, hd.col + d, hd.ch + d);      // without a state: no history
    if (state >= 0) stf4(p.ring + (state * TAPS + pos % TAPS) * p.channels + hd.ch + d, x);
    cv.step(x, y);
  }
  if (!hd.is_v) {
    if (on && d < p.rot) pair_angles(p.table + min(max(pos, 0), p.table_rows - 1) * p.rot, d, p.rot, cs);
    const float ss = warp_sum(y[0] * y[0] + y[1] * y[1] + y[2] * y[2] + y[3] * y[3]);
    if (on) {
      float w[4];
      ldf4((hd.is_q ? p.q_norm : p.k_norm) + d, w);
      const float inv = inv_rms<T>(ss, 1.f / (float)p.dim, p.eps);
#pragma unroll
      for (int c = 0; c < 4; ++c) y[c] *= inv * w[c];
      if (d < p.rot) turn_pairs(y, cs);
    }
  }
  if (d < hd.pad) {
    T* o = hd.is_q ? hd.row(p, t) : hd.cached(p, slot);
    if (o != nullptr) stf4(o + d, y);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) conv_qkv_kernel(const ConvQkvArgs<T> p) {
  const long long t = blockIdx.x;
  const bool decode = p.cu == nullptr;
  const int b = decode ? (int)t : p.tok_seq[t], lane = threadIdx.x & 31;
  const int pos = p.positions[t];
  const long long slot = p.state_slots[b];
  const int i = decode ? 0 : (int)(t - p.cu[b]);
  const int seen = slot < 0 ? 0 : pos;                   // a row that is not in use has no history
  const float* cs = p.table + (long long)min(max(pos, 0), p.table_rows - 1) * p.rot;
  for (int u = threadIdx.x >> 5; u < p.H + 2 * p.G; u += 8) {
    const HeadOf<T> hd(p, u);
    auto conv = [&](int d) {
      return d < hd.size ? conv_one<0>(static_cast<const ConvIn<T>&>(p), t, i, seen, max(slot, 0ll), hd.col + d, hd.ch + d) : 0.f;
    };
    float inv = 1.f;
    if (!hd.is_v) {
      float ss = 0.f;
      for (int d = lane; d < hd.size; d += 32) {
        const float y = conv(d);
        ss += y * y;
      }
      inv = 1.f / sqrtf(warp_sum(ss) / (float)p.dim + p.eps);
    }
    const float* w = hd.is_q ? p.q_norm : p.k_norm;
    T *o = hd.row(p, t), *k = hd.cached(p, p.slots[t]);
    for (int d = 2 * lane; d < hd.pad; d += 64) {
      float y[2] = {conv(d), conv(d + 1)};
      if (!hd.is_v) {
#pragma unroll
        for (int c = 0; c < 2; ++c)
          if (d + c < hd.size) y[c] *= inv * w[d + c];
        if (d < p.rot) {
          const float co = cs[d >> 1], si = cs[(p.rot + d) >> 1], a = y[0];
          y[0] = a * co - y[1] * si;
          y[1] = y[1] * co + a * si;
        }
      }
#pragma unroll
      for (int c = 0; c < 2; ++c)
        if (d + c < hd.pad) {
          if (o != nullptr) stf(o + d + c, y[c]);
          if (k != nullptr) stf(k + d + c, y[c]);
        }
    }
    if (decode && slot >= 0)
      for (int d = lane; d < hd.size; d += 32)
        p.ring[(slot * p.taps + pos % p.taps) * p.channels + hd.ch + d] = p.proj[t * p.ld + hd.col + d];
  }
}

}  // namespace msrl

using namespace msrl;

// ints: H, G, dim, vdim, qp, vp, taps, columns of q, k, v in proj and in out, rot, table rows, sequences.  Prompt portions
// give tok_seq, cu and start_pos; without cu every token is a sequence's next one.
MSRL_API int msrl_conv_qkv(const void* proj, long long ld, const int* ints, const float* conv, const float* q_norm,
                           const float* k_norm, float eps, const float* table, const int* positions, const long long* slots,
                           void* k_cache, void* v_cache, void* ring, const long long* state_slots, const int* tok_seq,
                           const int* cu, const int* start_pos, void* out, long long out_ld, int tokens, int is_f32,
                           cudaStream_t st) {
  if (tokens == 0) return 0;
  const int batch = ints[15];
  if (ints[13] % 2 != 0 || ints[13] > ints[2] || ints[6] < 1 || batch > 65535) return (int)cudaErrorInvalidValue;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    ConvQkvArgs<T> p{};
    p.proj = (const T*)proj;
    p.ld = ld;
    p.conv = conv;
    p.taps = ints[6];
    p.ring = (T*)ring;
    p.H = ints[0];
    p.G = ints[1];
    p.dim = ints[2];
    p.vdim = ints[3];
    p.qp = ints[4];
    p.vp = ints[5];
    p.channels = (p.H + p.G) * p.dim + p.G * p.vdim;
    p.q_col = ints[7];
    p.k_col = ints[8];
    p.v_col = ints[9];
    p.oq = ints[10];
    p.ok = ints[11];
    p.ov = ints[12];
    p.out = (T*)out;
    p.out_ld = out_ld;
    p.q_norm = q_norm;
    p.k_norm = k_norm;
    p.eps = eps;
    p.table = table;
    p.rot = ints[13];
    p.table_rows = ints[14];
    p.positions = positions;
    p.slots = slots;
    p.k_cache = (T*)k_cache;
    p.v_cache = (T*)v_cache;
    p.state_slots = state_slots;
    p.tok_seq = tok_seq;
    p.cu = cu;
    p.start_pos = start_pos;
    p.tokens = tokens;
    const bool decode = cu == nullptr;
    const dim3 grid((unsigned)((p.H + 2 * p.G + 7) / 8), (unsigned)(decode ? tokens : (tokens + CQ_TT - 1) / CQ_TT));
    const int odd = p.dim | p.vdim | p.qp | p.vp | p.q_col | p.k_col | p.v_col | p.oq | p.ok | p.ov | (int)(ld & 3) | (int)(out_ld & 3);
    if ((odd & 3) == 0 && (long long)p.table_rows * p.rot < (1ll << 31) && p.qp <= 128 && p.vp <= 128 && p.taps >= 2 && p.taps <= 4 &&
        grid.y <= 65535) {
      auto go = [&](auto prompt, auto step) {
        if (decode) step<<<grid, 256, 0, st>>>(p);
        else prompt<<<grid, 256, 0, st>>>(p);
      };
      if (p.taps == 4) go(conv_qkv4_kernel<T, 4>, conv_qkv4_step_kernel<T, 4>);
      else if (p.taps == 3) go(conv_qkv4_kernel<T, 3>, conv_qkv4_step_kernel<T, 3>);
      else go(conv_qkv4_kernel<T, 2>, conv_qkv4_step_kernel<T, 2>);
    } else {
      conv_qkv_kernel<T><<<(unsigned)tokens, 256, 0, st>>>(p);
    }
    if (cu != nullptr)
      conv_ring_kernel<T><<<dim3((unsigned)((p.channels + 255) / 256), (unsigned)batch), 256, 0, st>>>(
          p, p.H * p.dim, p.G * p.dim, p.q_col, p.k_col, p.v_col, cu, start_pos, state_slots);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}
