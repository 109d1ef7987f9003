// Latent attention over a paged cache of one latent row per token.
//
// A cache row is [latent (RP, zero padded) | rotated key part (CP - RP, zero padded)]: all heads share it.
// Scores are (q_unrotated . W_uk c + q_rotated . k_rotated) * scale and values W_uv c; the up-projections are
// linear, so prompts expand them per head and decode steps fold them into the query (q W_uk) and the output
// (W_uv sum p c) and attend to the rows themselves.
//
//   prep        RMS norm of the latent (and of the queries' own latent, where there is one), rotation of the shared
//               key part and of every head's query part (fp32; neighbours, or entries half a part away), cache write;
//               the row also goes to `lat` (prompts), the rotated query part to the decode query
//   spread      the rotated key part into every head's expanded key
//   decode_simt one query per sequence over the paged rows, any sizes, fp32 arithmetic
//   decode_mma  the same on the legacy tensor path for bf16 (block sizes that latent_decode_tcgen05.cu does not
//               take): a block takes 16 / 32 / 64 heads of one sequence and a range of its keys, so that a row is
//               read once for all of them; `combine` merges the ranges
//
// Decode kernels see the last `window` rows (0: all), may add exp(sink[h]) to a head's soft-max sum and may scale a head
// by sigmoid(gate).
#include "dtype_utils.cuh"
#include "head_tail.cuh"
#include "mma_utils.cuh"

namespace msrl {
namespace mla {

template <typename T>
struct PrepArgs {
  T* qkv;                      // [tokens, ld] rows with the query heads (H of them; 0: they are not there)
  long long ld;
  int H, q_stride, dn, dr;     // head h's query: columns h * q_stride + [0, dn) unrotated, then dr rotated
  const T* latent;             // [tokens, ld] latent and shared key part, or null: queries only
  int rank;
  const float* norm_w;
  float eps;
  const float* table;          // [positions, rot_dims]: cos | sin
  int rot_dims, table_rows, halves;
  const int* positions;
  const long long* slots;      // cache row per token, < 0: not cached
  T* cache;
  int RP, CP;
  T* lat;                      // [tokens, CP] or null
  T* qdec;                     // [tokens, H, CP] or null: receives the rotated query part at column RP
  int q_rank, QP, dq;          // the queries' latent lies dq columns behind `latent`
  const float* q_norm;
  T* cq;                       // [tokens, QP] or null: it normed, zero padded
};

// entry d of a rotated part
template <typename T>
__device__ __forceinline__ float rotated(const T* x, int d, const float* cs, int rot_dims, int halves) {
  if (d >= rot_dims) return ldf(x + d);
  const int half = rot_dims / 2, i = halves ? d % half : d >> 1;
  const bool second = halves ? d >= half : d & 1;
  const float c = cs[i], s = cs[half + i];
  const float u = ldf(x + (halves ? i : d & ~1)), v = ldf(x + (halves ? i + half : d | 1));
  return second ? v * c + u * s : u * c - v * s;
}

// entries d .. d + 3 (d a multiple of 4) of a rotated part whose rot_dims is a multiple of 4 (of 8 with halves)
template <typename T>
__device__ __forceinline__ void rotated4(const T* x, int d, const float* cs, int rot_dims, int halves, float (&y)[4]) {
  ldf4(x + d, y);
  if (d >= rot_dims) return;
  const int half = rot_dims / 2;
  if (halves) {
    const bool second = d >= half;
    const int i = second ? d - half : d;
    float o[4], c[4], s[4];
    ldf4(x + (second ? i : d + half), o);
    ldf4(cs + i, c);
    ldf4(cs + half + i, s);
#pragma unroll
    for (int k = 0; k < 4; ++k) y[k] = second ? y[k] * c[k] + o[k] * s[k] : y[k] * c[k] - o[k] * s[k];
    return;
  }
  const int i = d >> 1;
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const float c = cs[i + k], s = cs[half + i + k], u = y[2 * k], v = y[2 * k + 1];
    y[2 * k] = u * c - v * s;
    y[2 * k + 1] = v * c + u * s;
  }
}

// prep for sizes and columns that are multiples of 4: four entries per load and store
template <typename T>
__global__ void __launch_bounds__(256) prep4_kernel(const PrepArgs<T> p) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  T* row = p.qkv + t * p.ld;
  const T* lat_in = p.latent + t * p.ld;
  float ss = 0.f, sq = 0.f;
  if (p.latent != nullptr) {
    for (int c = threadIdx.x * 4; c < p.rank; c += 1024) {
      float x[4];
      ldf4(lat_in + c, x);
#pragma unroll
      for (int j = 0; j < 4; ++j) ss += x[j] * x[j];
    }
    if (p.cq != nullptr)
      for (int c = threadIdx.x * 4; c < p.q_rank; c += 1024) {
        float x[4];
        ldf4(lat_in + p.dq + c, x);
#pragma unroll
        for (int j = 0; j < 4; ++j) sq += x[j] * x[j];
      }
  }
  const int pos = min(max(p.positions[t], 0), p.table_rows - 1);
  const float* cs = p.table + (long long)pos * p.rot_dims;
  // queries first: they do not wait for the norm
  if (p.H > 0 && p.qdec != nullptr) {
    const int w = (p.CP - p.RP) / 4;
    for (int i = threadIdx.x; i < p.H * w; i += 256) {
      const int h = i / w, d = (i - h * w) * 4;
      float y[4] = {0.f, 0.f, 0.f, 0.f};
      if (d < p.dr) rotated4(row + h * p.q_stride + p.dn, d, cs, p.rot_dims, p.halves, y);
      stf4(p.qdec + (t * p.H + h) * p.CP + p.RP + d, y);
    }
  } else if (p.H > 0 && p.halves) {
    // in place: one thread owns both entries of a pair
    const int half = p.rot_dims / 2, quads = half / 4;
    for (int i = threadIdx.x; i < p.H * quads; i += 256) {
      const int h = i / quads, d = (i - h * quads) * 4;
      T* x = row + h * p.q_stride + p.dn;
      float a[4], b[4];
      rotated4(x, d, cs, p.rot_dims, 1, a);
      rotated4(x, d + half, cs, p.rot_dims, 1, b);
      stf4(x + d, a);
      stf4(x + d + half, b);
    }
  } else if (p.H > 0) {
    const int quads = p.rot_dims / 4;
    for (int i = threadIdx.x; i < p.H * quads; i += 256) {
      const int h = i / quads, d = (i - h * quads) * 4;
      T* x = row + h * p.q_stride + p.dn;
      float y[4];
      rotated4(x, d, cs, p.rot_dims, 0, y);
      stf4(x + d, y);
    }
  }
  if (p.latent == nullptr) return;
  if (p.cq != nullptr) {
    const float inv = 1.f / sqrtf(block_sum(sq, red) / (float)p.q_rank + p.eps);
    for (int c = threadIdx.x * 4; c < p.QP; c += 1024) {
      float y[4] = {0.f, 0.f, 0.f, 0.f};
      if (c < p.q_rank) {
        float w[4];
        ldf4(lat_in + p.dq + c, y);
        ldf4(p.q_norm + c, w);
#pragma unroll
        for (int j = 0; j < 4; ++j) y[j] *= inv * w[j];
      }
      stf4(p.cq + t * p.QP + c, y);
    }
  }
  const long long slot = p.slots[t];
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)p.rank + p.eps);
  T* crow = slot >= 0 ? p.cache + slot * p.CP : nullptr;
  T* lrow = p.lat != nullptr ? p.lat + t * p.CP : nullptr;
  for (int c = threadIdx.x * 4; c < p.CP; c += 1024) {
    float y[4] = {0.f, 0.f, 0.f, 0.f};
    if (c < p.rank) {
      float w[4];
      ldf4(lat_in + c, y);
      ldf4(p.norm_w + c, w);
#pragma unroll
      for (int j = 0; j < 4; ++j) y[j] *= inv * w[j];
    } else if (c >= p.RP && c < p.RP + p.dr) {
      rotated4(lat_in + p.rank, c - p.RP, cs, p.rot_dims, p.halves, y);
    }
    if (crow != nullptr) stf4(crow + c, y);
    if (lrow != nullptr) stf4(lrow + c, y);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) prep_kernel(const PrepArgs<T> p) {
  __shared__ float red[32];
  const long long t = blockIdx.x;
  T* row = p.qkv + t * p.ld;
  const int pos = min(max(p.positions[t], 0), p.table_rows - 1);
  const float* cs = p.table + (long long)pos * p.rot_dims;
  if (p.latent != nullptr) {
    const T* lat_in = p.latent + t * p.ld;
    float ss = 0.f, sq = 0.f;
    for (int c = threadIdx.x; c < p.rank; c += 256) {
      const float x = ldf(lat_in + c);
      ss += x * x;
    }
    const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)p.rank + p.eps);
    const long long slot = p.slots[t];
    T* crow = slot >= 0 ? p.cache + slot * p.CP : nullptr;
    T* lrow = p.lat != nullptr ? p.lat + t * p.CP : nullptr;
    for (int c = threadIdx.x; c < p.CP; c += 256) {
      float v = 0.f;
      if (c < p.rank) v = ldf(lat_in + c) * inv * p.norm_w[c];
      else if (c >= p.RP && c < p.RP + p.dr) v = rotated(lat_in + p.rank, c - p.RP, cs, p.rot_dims, p.halves);
      if (crow != nullptr) stf(crow + c, v);
      if (lrow != nullptr) stf(lrow + c, v);
    }
    if (p.cq != nullptr) {
      for (int c = threadIdx.x; c < p.q_rank; c += 256) {
        const float x = ldf(lat_in + p.dq + c);
        sq += x * x;
      }
      const float iq = 1.f / sqrtf(block_sum(sq, red) / (float)p.q_rank + p.eps);
      for (int c = threadIdx.x; c < p.QP; c += 256)
        stf(p.cq + t * p.QP + c, c < p.q_rank ? ldf(lat_in + p.dq + c) * iq * p.q_norm[c] : 0.f);
    }
  }
  if (p.H == 0) return;
  if (p.qdec != nullptr) {
    const int w = p.CP - p.RP;
    for (int i = threadIdx.x; i < p.H * w; i += 256) {
      const int h = i / w, d = i % w;
      stf(p.qdec + (t * p.H + h) * p.CP + p.RP + d,
          d < p.dr ? rotated(row + h * p.q_stride + p.dn, d, cs, p.rot_dims, p.halves) : 0.f);
    }
  } else {
    // in place: one thread owns both entries of a pair
    const int half = p.rot_dims / 2;
    for (int i = threadIdx.x; i < p.H * half; i += 256) {
      const int h = i / half, j = i % half, d0 = p.halves ? j : 2 * j, d1 = p.halves ? j + half : 2 * j + 1;
      T* x = row + h * p.q_stride + p.dn;
      const float a = rotated(x, d0, cs, p.rot_dims, p.halves), b = rotated(x, d1, cs, p.rot_dims, p.halves);
      stf(x + d0, a);
      stf(x + d1, b);
    }
  }
}

// kv[t, h * stride + dn + d] = lat[t, RP + d]
template <typename T>
__global__ void spread_kernel(const T* lat, int CP, int RP, T* kv, long long ld, int H, int stride, int dn, int dr,
                              long long tokens) {
  const long long t = blockIdx.x;
  if (dr % 4 == 0 && dn % 4 == 0 && stride % 4 == 0 && ld % 4 == 0) {
    const int quads = dr / 4;
    for (int i = threadIdx.x; i < H * quads; i += blockDim.x) {
      const int h = i / quads, d = (i - h * quads) * 4;
      float x[4];
      ldf4(lat + t * CP + RP + d, x);
      stf4(kv + t * ld + h * stride + dn + d, x);
    }
    return;
  }
  for (int i = threadIdx.x; i < H * dr; i += blockDim.x)
    kv[t * ld + (i / dr) * stride + dn + i % dr] = lat[t * CP + RP + i % dr];
}

// ---- decode on the CUDA cores -----------------------------------------------------------------------------
constexpr int DS_ACC = 8;                // latent columns per thread: RP <= 2048

template <typename T>
__global__ void __launch_bounds__(256)
decode_simt_kernel(const T* q, const T* cache, const int* block_tables, int max_blocks, int block_size,
                   const int* context_lens, float scale, int CP, int RP, int window, const HeadTail<T> tail, T* out) {
  extern __shared__ float smf[];
  __shared__ float sS[32];
  float* sQ = smf;
  const int h = blockIdx.x, b = blockIdx.y, H = gridDim.x;
  const int n = context_lens[b];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const T* qr = q + ((long long)b * H + h) * CP;
  for (int c = threadIdx.x; c < CP; c += 256) sQ[c] = ldf(qr + c);
  const int* bt = block_tables + (long long)b * max_blocks;
  float acc[DS_ACC];
#pragma unroll
  for (int i = 0; i < DS_ACC; ++i) acc[i] = 0.f;
  float m_run = -INFINITY, l_run = 0.f;
  for (int kb = window > 0 ? max(n - window, 0) : 0; kb < n; kb += 32) {
    __syncthreads();
    for (int j = warp; j < 32; j += 8) {
      const int key = kb + j;
      float s = -INFINITY;
      if (key < n) {
        const T* r = cache + ((long long)bt[key / block_size] * block_size + key % block_size) * CP;
        s = 0.f;
        for (int c = lane; c < CP; c += 32) s += sQ[c] * ldf(r + c);
        s = warp_sum(s) * scale;
      }
      if (lane == 0) sS[j] = s;
    }
    __syncthreads();
    float m_new = m_run;
    for (int j = 0; j < 32; ++j) m_new = fmaxf(m_new, sS[j]);
    const float corr = expf(m_run - m_new);
    l_run *= corr;
    m_run = m_new;
#pragma unroll
    for (int i = 0; i < DS_ACC; ++i) acc[i] *= corr;
    const int keys = min(32, n - kb);
    for (int j = 0; j < keys; ++j) {
      const int key = kb + j;
      const float pj = expf(sS[j] - m_new);
      l_run += pj;
      const T* r = cache + ((long long)bt[key / block_size] * block_size + key % block_size) * CP;
#pragma unroll
      for (int i = 0; i < DS_ACC; ++i) {
        const int c = threadIdx.x + 256 * i;
        if (c < RP) acc[i] += pj * ldf(r + c);
      }
    }
  }
  const float inv = tail.scale(b, h, m_run, l_run);
#pragma unroll
  for (int i = 0; i < DS_ACC; ++i) {
    const int c = threadIdx.x + 256 * i;
    if (c < RP) stf(out + ((long long)b * H + h) * RP + c, acc[i] * inv);
  }
}

// ---- decode on the tensor cores (bf16) -------------------------------------------------------------------
struct MmaArgs {
  const __nv_bfloat16* q;      // [B, H, CP]
  const __nv_bfloat16* cache;  // [rows, CP]
  const int* block_tables;
  int max_blocks, block_size;
  const int* context_lens;
  float scale_log2;
  int H, CP, RP, nsplit;
  int window;                  // keys a query sees, itself included (0: all)
  HeadTail<__nv_bfloat16> tail;
  float* part_o;               // [B, H, nsplit, RP]
  float* part_ml;              // [B, H, nsplit, 2]
  __nv_bfloat16* out;          // [B, H, RP], written directly when nsplit == 1
};

// MT 16-head tiles per block, NT 8-column output tiles per warp (RP <= 64 * NT), KT keys per tile
template <int MT, int NT, int KT>
__global__ void __launch_bounds__(256, 1) decode_mma_kernel(const MmaArgs p) {
  constexpr int HM = 16 * MT, WK = 8 / MT, NK8 = KT / 8 / WK;      // warps: WK key groups x MT head tiles
  constexpr int TPR = 256 / HM, KPT = KT / TPR;                    // soft-max: threads per head row, keys per thread
  constexpr int LDS_S = KT + 4, LDS_P = KT + 8;
  static_assert(NK8 >= 1 && KPT >= 1, "tile sizes");
  extern __shared__ __align__(16) unsigned char raw[];
  const int ld = p.CP + 8;
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(raw);
  __nv_bfloat16* sKV = sQ + HM * ld;                               // two buffers
  float* sS = reinterpret_cast<float*>(sKV + 2 * KT * ld);
  __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(sS + HM * LDS_S);
  float* sCorr = reinterpret_cast<float*>(sP + HM * LDS_P);        // [HM]
  float* sL = sCorr + HM;                                          // [HM]
  const int split = blockIdx.x, h0 = blockIdx.y * HM, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = p.context_lens[b];
  const int lo = p.window > 0 ? max(n - p.window, 0) : 0, tile0 = lo / KT;      // first key, its tile
  const int tiles = (n + KT - 1) / KT, per = (tiles - tile0 + p.nsplit - 1) / p.nsplit;
  const int first = tile0 + split * per, last = min(tiles, first + per);
  const int vecs = p.CP / 8;
  const int* bt = p.block_tables + (long long)b * p.max_blocks;

  // cache row of the key that lane l of a warp looks up for its warp's row l (rows warp, warp + 8, ...); -1: none
  auto look_up = [&](int tile) -> int {
    const int key = tile * KT + warp + 8 * lane;
    return lane < KT / 8 && key < n ? bt[key / p.block_size] * p.block_size + key % p.block_size : -1;
  };
  auto load_tile = [&](int slots_of_lane, int buf) {
    __nv_bfloat16* dst = sKV + buf * KT * ld;
#pragma unroll
    for (int i = 0; i < KT / 8; ++i) {
      const int slot = __shfl_sync(0xffffffffu, slots_of_lane, i);
      const __nv_bfloat16* src = p.cache + (long long)max(slot, 0) * p.CP;
      for (int c = lane; c < vecs; c += 32) cp_async16(dst + (warp + 8 * i) * ld + c * 8, src + c * 8, slot >= 0);
    }
    cp_async_commit();
  };

  float o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) o[m][i][j] = 0.f;
  const int srow = threadIdx.x / TPR, spart = threadIdx.x % TPR;
  float m_run = -INFINITY, l_run = 0.f;
  const int wm = warp / WK, wk = warp % WK;                        // scores: head tile and key group of this warp
  const int col0 = warp * NT * 8;                                  // output columns of this warp

  if (first < last) {
    for (int r = warp; r < HM; r += 8) {
      const bool ok = h0 + r < p.H;
      const __nv_bfloat16* src = p.q + ((long long)b * p.H + (ok ? h0 + r : 0)) * p.CP;
      for (int c = lane; c < vecs; c += 32) cp_async16(sQ + r * ld + c * 8, src + c * 8, ok);
    }
    load_tile(look_up(first), 0);
  }
  int ahead = first + 1 < last ? look_up(first + 1) : -1;          // rows of the tile that is loaded next
  for (int tile = first; tile < last; ++tile) {
    const int buf = (tile - first) & 1;
    if (tile + 1 < last) {
      load_tile(ahead, buf ^ 1);
      if (tile + 2 < last) ahead = look_up(tile + 2);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const __nv_bfloat16* kv = sKV + buf * KT * ld;
    // scores of 16 heads x 8 * NK8 keys per warp
    float s[NK8][4], s2[NK8][4];                                   // even and odd steps of the reduction
#pragma unroll
    for (int i = 0; i < NK8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[i][j] = s2[i][j] = 0.f;
    const int key0 = wk * NK8 * 8;
    auto k_step = [&](int kk, float (&acc)[NK8][4]) {
      uint32_t a[4];
      ldmatrix_x4(a, smem_u32(sQ + (wm * 16 + (lane & 15)) * ld + kk * 16 + (lane >> 4) * 8));
      if constexpr (NK8 == 2) {
        uint32_t f[4];
        ldmatrix_x4(f, smem_u32(kv + (key0 + (lane & 7) + (lane >> 4) * 8) * ld + kk * 16 + ((lane >> 3) & 1) * 8));
        mma_16816(acc[0], a, f[0], f[1]);
        mma_16816(acc[1], a, f[2], f[3]);
      } else {
#pragma unroll
        for (int i = 0; i < NK8; ++i) {
          uint32_t f[2];
          asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];\n"
                       : "=r"(f[0]), "=r"(f[1])
                       : "r"(smem_u32(kv + (key0 + i * 8 + (lane & 7)) * ld + kk * 16 + ((lane >> 3) & 1) * 8)));
          mma_16816(acc[i], a, f[0], f[1]);
        }
      }
    };
    const int steps = p.CP / 16;
    int kk = 0;
#pragma unroll 2
    for (; kk + 1 < steps; kk += 2) {
      k_step(kk, s);
      k_step(kk + 1, s2);
    }
    if (kk < steps) k_step(kk, s);
#pragma unroll
    for (int i = 0; i < NK8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[i][j] += s2[i][j];
#pragma unroll
    for (int i = 0; i < NK8; ++i) {
      float* d = sS + (wm * 16 + (lane >> 2)) * LDS_S + key0 + i * 8 + (lane & 3) * 2;
      d[0] = s[i][0];
      d[1] = s[i][1];
      d[8 * LDS_S] = s[i][2];
      d[8 * LDS_S + 1] = s[i][3];
    }
    __syncthreads();
    // soft-max of one head row by TPR neighbouring threads
    {
      float v[KPT], mx = -INFINITY;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        const int k = spart + i * TPR;
        v[i] = tile * KT + k < n && tile * KT + k >= lo ? sS[srow * LDS_S + k] * p.scale_log2 : -INFINITY;
        mx = fmaxf(mx, v[i]);
      }
#pragma unroll
      for (int x = TPR / 2; x > 0; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
      const float m_new = fmaxf(m_run, mx);                        // finite: a tile holds at least one key
      const float corr = exp2f(m_run - m_new);
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        const float e = exp2f(v[i] - m_new);
        sum += e;
        sP[srow * LDS_P + spart + i * TPR] = __float2bfloat16_rn(e);
      }
#pragma unroll
      for (int x = TPR / 2; x > 0; x >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, x);
      l_run = l_run * corr + sum;
      m_run = m_new;
      if (spart == 0) sCorr[srow] = corr;
    }
    __syncthreads();
    // o = o * corr + P V, V = the latent columns of the same tile
    if (col0 < p.RP) {
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float ca = sCorr[m * 16 + (lane >> 2)], cb = sCorr[m * 16 + (lane >> 2) + 8];
#pragma unroll
        for (int i = 0; i < NT; ++i) {
          o[m][i][0] *= ca;
          o[m][i][1] *= ca;
          o[m][i][2] *= cb;
          o[m][i][3] *= cb;
        }
      }
#pragma unroll
      for (int kc = 0; kc < KT / 16; ++kc) {
        uint32_t a[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
          ldmatrix_x4(a[m], smem_u32(sP + (m * 16 + (lane & 15)) * LDS_P + kc * 16 + (lane >> 4) * 8));
#pragma unroll
        for (int i = 0; i < NT; ++i) {
          if (col0 + i * 8 < p.RP) {                               // uniform over the warp
            uint32_t f[2];
            asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];\n"
                         : "=r"(f[0]), "=r"(f[1])
                         : "r"(smem_u32(kv + (kc * 16 + (lane & 15)) * ld + col0 + i * 8)));
#pragma unroll
            for (int m = 0; m < MT; ++m) mma_16816(o[m][i], a[m], f[0], f[1]);
          }
        }
      }
    }
    __syncthreads();
  }
  if (spart == 0) {
    sL[srow] = p.nsplit == 1 && h0 + srow < p.H ? p.tail.scale2(b, h0 + srow, m_run, l_run) : 0.f;
    if (p.nsplit > 1 && h0 + srow < p.H) {
      float* ml = p.part_ml + (((long long)b * p.H + h0 + srow) * p.nsplit + split) * 2;
      ml[0] = m_run;
      ml[1] = l_run;
    }
  }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < MT; ++m) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = m * 16 + (lane >> 2) + half * 8;
      if (h0 + r >= p.H) continue;
      const float inv = sL[r];
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int c = col0 + i * 8 + (lane & 3) * 2;
        if (c >= p.RP) continue;
        const float x = o[m][i][2 * half], y = o[m][i][2 * half + 1];
        if (p.nsplit == 1) {
          *reinterpret_cast<__nv_bfloat162*>(p.out + ((long long)b * p.H + h0 + r) * p.RP + c) =
              __floats2bfloat162_rn(x * inv, y * inv);
        } else {
          *reinterpret_cast<float2*>(p.part_o + (((long long)b * p.H + h0 + r) * p.nsplit + split) * p.RP + c) =
              make_float2(x, y);
        }
      }
    }
  }
}

__global__ void combine_kernel(const float* part_o, const float* part_ml, int H, int nsplit, int RP,
                               const HeadTail<__nv_bfloat16> tail, __nv_bfloat16* out) {
  const long long r = blockIdx.x;
  float m = -INFINITY;
  for (int s = 0; s < nsplit; ++s) m = fmaxf(m, part_ml[(r * nsplit + s) * 2]);
  float l = 0.f;
  for (int s = 0; s < nsplit; ++s) {
    const float ls = part_ml[(r * nsplit + s) * 2 + 1];
    if (ls > 0.f) l += ls * exp2f(part_ml[(r * nsplit + s) * 2] - m);
  }
  const float inv = tail.scale2(r / H, (int)(r % H), m, l);
  for (int c = threadIdx.x; c < RP; c += blockDim.x) {
    float a = 0.f;
    for (int s = 0; s < nsplit; ++s)
      if (part_ml[(r * nsplit + s) * 2 + 1] > 0.f)
        a += part_o[(r * nsplit + s) * RP + c] * exp2f(part_ml[(r * nsplit + s) * 2] - m);
    out[r * RP + c] = __float2bfloat16_rn(a * inv);
  }
}

template <int MT, int NT, int KT>
static int launch_mma(const MmaArgs& p, int batch, cudaStream_t st) {
  constexpr int HM = 16 * MT;
  const size_t smem = sizeof(__nv_bfloat16) * (size_t)(HM + 2 * KT) * (p.CP + 8) + sizeof(float) * HM * (KT + 4) +
                      sizeof(__nv_bfloat16) * HM * (KT + 8) + sizeof(float) * 2 * HM;
  if (smem > 227 * 1024) return (int)cudaErrorNotSupported;
  cudaError_t e = cudaFuncSetAttribute(decode_mma_kernel<MT, NT, KT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  const dim3 grid((unsigned)p.nsplit, (unsigned)((p.H + HM - 1) / HM), (unsigned)batch);
  decode_mma_kernel<MT, NT, KT><<<grid, 256, smem, st>>>(p);
  if (p.nsplit > 1)
    combine_kernel<<<(unsigned)(batch * p.H), 128, 0, st>>>(p.part_o, p.part_ml, p.H, p.nsplit, p.RP, p.tail, p.out);
  return (int)cudaGetLastError();
}

template <int NT>
static int pick_mma(const MmaArgs& p, int batch, cudaStream_t st) {
  if (p.H <= 16) return launch_mma<1, NT, 64>(p, batch, st);
  if (p.H <= 32) return launch_mma<2, NT, 64>(p, batch, st);
  return launch_mma<4, NT, 32>(p, batch, st);
}

}  // namespace mla
}  // namespace msrl

using namespace msrl;

// ints: H, q_stride, dn, dr, rank, rot_dims, table_rows, RP, CP, halves, q_rank, QP, column of the queries' latent less that
// of the latent.  Without `latent` (same row stride as qkv) only queries are rotated, with H = 0 none.
MSRL_API int msrl_latent_prep(void* qkv, long long ld, const void* latent, const int* ints, const float* norm_w, float eps,
                              const float* q_norm, const float* table, const int* positions, const long long* slots,
                              void* cache, void* lat, void* cq, void* qdec, int tokens, int is_f32, cudaStream_t st) {
  if (tokens == 0) return 0;
  auto run = [&](auto tag) {
    using T = decltype(tag);
    mla::PrepArgs<T> p{};
    p.qkv = (T*)qkv;
    p.ld = ld;
    p.latent = (const T*)latent;
    p.H = ints[0];
    p.q_stride = ints[1];
    p.dn = ints[2];
    p.dr = ints[3];
    p.rank = ints[4];
    p.rot_dims = ints[5];
    p.table_rows = ints[6];
    p.RP = ints[7];
    p.CP = ints[8];
    p.halves = ints[9];
    p.q_rank = ints[10];
    p.QP = ints[11];
    p.dq = ints[12];
    p.norm_w = norm_w;
    p.eps = eps;
    p.q_norm = q_norm;
    p.table = table;
    p.positions = positions;
    p.slots = slots;
    p.cache = (T*)cache;
    p.lat = (T*)lat;
    p.cq = (T*)cq;
    p.qdec = (T*)qdec;
    bool by4 = ((p.rank | p.dr | p.dn | p.rot_dims | p.q_stride | (int)(ld & 3)) & 3) == 0 &&
               reinterpret_cast<uintptr_t>(latent) % (4 * sizeof(T)) == 0;
    if (p.cq != nullptr) by4 = by4 && ((p.q_rank | p.dq) & 3) == 0;
    if (p.halves) by4 = by4 && p.rot_dims % 8 == 0;
    if (by4) mla::prep4_kernel<T><<<tokens, 256, 0, st>>>(p);
    else mla::prep_kernel<T><<<tokens, 256, 0, st>>>(p);
    return (int)cudaGetLastError();
  };
  return is_f32 ? run(float{}) : run(__nv_bfloat16{});
}

MSRL_API int msrl_latent_spread(const void* lat, int CP, int RP, void* kv, long long ld, int H, int stride, int dn,
                                int dr, int tokens, int is_f32, cudaStream_t st) {
  if (tokens == 0 || dr == 0) return 0;
  if (is_f32)
    mla::spread_kernel<float><<<tokens, 256, 0, st>>>((const float*)lat, CP, RP, (float*)kv, ld, H, stride, dn, dr, tokens);
  else
    mla::spread_kernel<__nv_bfloat16><<<tokens, 256, 0, st>>>((const __nv_bfloat16*)lat, CP, RP, (__nv_bfloat16*)kv, ld, H,
                                                              stride, dn, dr, tokens);
  return (int)cudaGetLastError();
}

MSRL_API int msrl_latent_decode_simt(const void* q, const void* cache, const int* block_tables, int max_blocks,
                                     int block_size, const int* context_lens, float scale, int batch, int H, int CP,
                                     int RP, int window, const void* gate, long long gate_ld, const float* sink, void* out,
                                     int is_f32, cudaStream_t st) {
  if (batch == 0) return 0;
  if (RP > 256 * mla::DS_ACC || batch > 65535 || CP > 12000) return (int)cudaErrorNotSupported;
  const dim3 grid((unsigned)H, (unsigned)batch);
  if (is_f32)
    mla::decode_simt_kernel<float><<<grid, 256, CP * sizeof(float), st>>>((const float*)q, (const float*)cache, block_tables,
                                                                          max_blocks, block_size, context_lens, scale, CP, RP, window,
                                                                          HeadTail<float>{(const float*)gate, gate_ld, sink}, (float*)out);
  else
    mla::decode_simt_kernel<__nv_bfloat16><<<grid, 256, CP * sizeof(float), st>>>(
        (const __nv_bfloat16*)q, (const __nv_bfloat16*)cache, block_tables, max_blocks, block_size, context_lens, scale, CP,
        RP, window, HeadTail<__nv_bfloat16>{(const __nv_bfloat16*)gate, gate_ld, sink}, (__nv_bfloat16*)out);
  return (int)cudaGetLastError();
}

// Key ranges per (sequence, head group): the count that finishes first when whole waves of one block per SM walk
// their tiles of 64 keys and every block pays for its start, its end and the merge.
MSRL_API int msrl_latent_decode_nsplit(int batch, int H, int max_context) {
  const long long blocks = (long long)batch * (H <= 32 ? 1 : (H + 63) / 64);
  const int tiles = (max_context + 63) / 64, sms = sm_count();
  int best = 1;
  double least = 1e30;
  for (int n = 1; n <= 64 && n <= (tiles + 1) / 2 + 1; ++n) {
    const double waves = (double)((blocks * n + sms - 1) / sms);
    const double cost = waves * ((tiles + n - 1) / n + 2.5) + (n > 1 ? 1.0 : 0.0);
    if (cost < least) {
      least = cost;
      best = n;
    }
  }
  return best;
}

// merge of the key ranges that msrl_latent_decode_tcgen05 leaves in part_o / part_ml
MSRL_API int msrl_latent_decode_combine(const float* part_o, const float* part_ml, int batch, int H, int RP, int nsplit,
                                        const void* gate, long long gate_ld, const float* sink, void* out, cudaStream_t st) {
  if (batch == 0) return 0;
  mla::combine_kernel<<<(unsigned)(batch * H), 128, 0, st>>>(
      part_o, part_ml, H, nsplit, RP, HeadTail<__nv_bfloat16>{(const __nv_bfloat16*)gate, gate_ld, sink}, (__nv_bfloat16*)out);
  return (int)cudaGetLastError();
}

// part_o [B, H, nsplit, RP] and part_ml [B, H, nsplit, 2] fp32 (unused when nsplit == 1)
MSRL_API int msrl_latent_decode_mma(const void* q, const void* cache, const int* block_tables, int max_blocks,
                                    int block_size, const int* context_lens, float scale, int batch, int H, int CP,
                                    int RP, int nsplit, int window, const void* gate, long long gate_ld, const float* sink,
                                    float* part_o, float* part_ml, void* out, cudaStream_t st) {
  if (batch == 0) return 0;
  if (CP % 16 != 0 || RP % 16 != 0 || RP > 512 || batch > 65535) return (int)cudaErrorNotSupported;
  mla::MmaArgs p{(const __nv_bfloat16*)q, (const __nv_bfloat16*)cache, block_tables, max_blocks, block_size,
                 context_lens, scale * 1.4426950408889634f, H, CP, RP, nsplit, window,
                 {(const __nv_bfloat16*)gate, gate_ld, sink}, part_o, part_ml, (__nv_bfloat16*)out};
  if (RP <= 128) return mla::pick_mma<2>(p, batch, st);
  if (RP <= 256) return mla::pick_mma<4>(p, batch, st);
  return mla::pick_mma<8>(p, batch, st);
}
