// Between the q | k | v projection and grouped-head attention, everything in fp32:
//
//   x  <- causal convolution over time, one filter per channel (short_conv.cuh)
//   q, k <- x / sqrt(mean over the head of x^2 + eps) * weight, then rotation of the first `rot` entries of the head,
//           entry 2i with entry 2i + 1;   v <- x
//
// Prepared rows hold the heads padded (qp, vp; pad entries are written as zeros), and so do the cache rows of k and v.
// Prompt portions are followed by conv_ring_kernel; a decode step (one token per sequence) writes its ring entry itself.
//
//   conv_qkv4_kernel   heads of up to 128 entries, sizes and columns multiples of 4, 2 to 4 taps: a warp walks consecutive
//                      tokens of one head with the convolution windows in registers, four channels per lane
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

constexpr int CQ_TT = 32, CQ_U = 4;      // tokens per warp, tokens in flight together

template <typename T, int TAPS>
__global__ void __launch_bounds__(256, 2) conv_qkv4_kernel(const ConvQkvArgs<T> p, int per_warp) {
  const int u = blockIdx.x * 8 + (threadIdx.x >> 5), d = (threadIdx.x & 31) * 4;
  if (u >= p.H + 2 * p.G) return;
  const HeadOf<T> hd(p, u);
  const int t0 = blockIdx.y * per_warp, t1 = min(p.tokens, t0 + per_warp);
  const bool on = d < hd.size, wr = d < hd.pad, decode = p.cu == nullptr;
  const bool turned = on && !hd.is_v && d < p.rot, whole = p.rot % 4 == 0;
  ConvWindow<TAPS, T> cv;
  float w[4] = {0.f, 0.f, 0.f, 0.f};
  if (on) {
    cv.weights(p.conv, hd.ch + d);
    if (!hd.is_v) ldf4((hd.is_q ? p.q_norm : p.k_norm) + d, w);
  }
  int seq = -1;
  for (int tb = t0; tb < t1; tb += CQ_U) {
    float y[CQ_U][4], cs[CQ_U][4];                       // cs: two cosines, two sines
    int sq[CQ_U], pos[CQ_U];
    long long slot[CQ_U];
#pragma unroll
    for (int n = 0; n < CQ_U; ++n) {
      const int t = min(tb + n, t1 - 1);
      sq[n] = decode ? t : p.tok_seq[t];
      pos[n] = p.positions[t];
      slot[n] = hd.is_q ? -1 : p.slots[t];
#pragma unroll
      for (int c = 0; c < 4; ++c) y[n][c] = 0.f;
      if (on) ldf4(p.proj + t * p.ld + hd.col + d, y[n]);
    }
    if (turned) {
#pragma unroll
      for (int n = 0; n < CQ_U; ++n) {
        const float* tab = p.table + (long long)min(max(pos[n], 0), p.table_rows - 1) * p.rot + (d >> 1);
        if (whole) {
          const float2 a = *reinterpret_cast<const float2*>(tab), b = *reinterpret_cast<const float2*>(tab + (p.rot >> 1));
          cs[n][0] = a.x; cs[n][1] = a.y; cs[n][2] = b.x; cs[n][3] = b.y;
        } else {
          const bool two = d + 2 < p.rot;
          cs[n][0] = tab[0];
          cs[n][1] = two ? tab[1] : 1.f;
          cs[n][2] = tab[p.rot >> 1];
          cs[n][3] = two ? tab[(p.rot >> 1) + 1] : 0.f;
        }
      }
    }
#pragma unroll
    for (int n = 0; n < CQ_U; ++n) {
      const int t = tb + n;
      if (t >= t1 || !on) continue;                      // what is past the end is not written
      if (sq[n] != seq) {
        seq = sq[n];
        const long long state = p.state_slots[seq];
        if (state < 0) cv.fill(p, t, 0, 0, 0, hd.col + d, hd.ch + d);         // a row that is not in use
        else cv.fill(p, t, decode ? 0 : t - p.cu[seq], pos[n], state, hd.col + d, hd.ch + d);
        if (decode && state >= 0) stf4(p.ring + (state * TAPS + pos[n] % TAPS) * p.channels + hd.ch + d, y[n]);
      }
      cv.step(y[n], y[n]);
    }
    if (!hd.is_v) {
      float ss[CQ_U];
#pragma unroll
      for (int n = 0; n < CQ_U; ++n) ss[n] = y[n][0] * y[n][0] + y[n][1] * y[n][1] + y[n][2] * y[n][2] + y[n][3] * y[n][3];
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int n = 0; n < CQ_U; ++n) ss[n] += __shfl_xor_sync(0xffffffffu, ss[n], o);
#pragma unroll
      for (int n = 0; n < CQ_U; ++n) {
        const float inv = 1.f / sqrtf(ss[n] / (float)p.dim + p.eps);
#pragma unroll
        for (int c = 0; c < 4; ++c) y[n][c] *= inv * w[c];
        if (turned) {
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            const float a = y[n][2 * c], b = y[n][2 * c + 1];
            y[n][2 * c] = a * cs[n][c] - b * cs[n][2 + c];
            y[n][2 * c + 1] = b * cs[n][c] + a * cs[n][2 + c];
          }
        }
      }
    }
#pragma unroll
    for (int n = 0; n < CQ_U; ++n) {
      const int t = tb + n;
      if (t < t1 && wr) {
        T *o = hd.row(p, t), *k = hd.cached(p, slot[n]);
        if (o != nullptr) stf4(o + d, y[n]);
        if (k != nullptr) stf4(k + d, y[n]);
      }
    }
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
    const int units = p.H + 2 * p.G, per_warp = cu == nullptr ? 1 : CQ_TT;
    const dim3 grid((unsigned)((units + 7) / 8), (unsigned)((tokens + per_warp - 1) / per_warp));
    const int odd = p.dim | p.vdim | p.qp | p.vp | p.q_col | p.k_col | p.v_col | p.oq | p.ok | p.ov | (int)(ld & 3) | (int)(out_ld & 3);
    if ((odd & 3) == 0 && p.qp <= 128 && p.vp <= 128 && p.taps >= 2 && p.taps <= 4 && grid.y <= 65535) {
      if (p.taps == 4) conv_qkv4_kernel<T, 4><<<grid, 256, 0, st>>>(p, per_warp);
      else if (p.taps == 3) conv_qkv4_kernel<T, 3><<<grid, 256, 0, st>>>(p, per_warp);
      else conv_qkv4_kernel<T, 2><<<grid, 256, 0, st>>>(p, per_warp);
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
