// Decode step of latent attention on the 5th-generation tensor cores (tcgen05 + TMEM + TMA).
//
// One query token per sequence attends to the sequence's paged cache rows [latent (RP) | rotated key part]; all
// heads share the rows, and the latent part of a row is its value.  One CTA takes up to HB (32 or 64) heads of one
// sequence and a range of its keys, so that a row is read once for all of them.  Per tile of 64 keys:
//
//   rows      TMA boxes of [block_size rows x 64 columns] from the paged cache through the block table into a
//             two-stage ring of 128-byte-swizzled [64 keys x 64 columns] chunks;
//   S         Q K^T into one of two TMEM buffers [heads x 64]: the query's HB rows are read as the 128-row A
//             operand (the lanes past HB hold what lies behind the query in shared memory and are never looked at);
//   soft-max  two warps per 32 heads (each row's maximum by both, half of the exponentials each), P (bf16) to
//             shared memory as [heads x 64 keys];
//   O^T       [latent x heads] += V^T P^T: the SAME chunks of the ring as MN-major A operand (128 latent columns a
//             time), P as K-major B operand; O^T stays in TMEM, HB columns per 128 latents, and is rescaled by head
//             (column) only when a head's maximum moved by more than 2^8.
//
// The last tile of a sequence is ragged: blocks past its end are not loaded and the rows past its end are zeroed in
// shared memory before they are multiplied (freed pages may hold anything).
//
// Every mbarrier wait is bounded; on expiry the kernel records a code in the status word, skips the rest, frees
// TMEM and returns.
#include <cuda.h>
#include <cudaTypedefs.h>

#include "head_tail.cuh"
#include "tcgen05_utils.cuh"

namespace msrl {
namespace ld5 {

using namespace t5;

constexpr int KT = 64;                                  // keys per tile
constexpr uint32_t CHUNK = KT * 128;                    // [64 keys x 64 columns] bf16
constexpr int SM_WARPS = 8, TMA_WARP = 8, MMA_WARP = 9, THREADS = 320;

enum { ERR_SMEM = 60, ERR_Q = 61, ERR_K = 62, ERR_S = 63, ERR_P = 64, ERR_PV = 65, ERR_EMPTY = 66, ERR_FREE = 67 };

struct Params {
  const int* block_tables;
  int max_blocks, block_size;
  const int* context_lens;
  float scale_log2;
  int H, CP, RP, nsplit;
  int window;                  // keys a query sees, itself included (0: all)
  HeadTail<__nv_bfloat16> tail;
  int chunks;                  // chunks of a ring stage: enough for CP columns and for whole 128-latent blocks
  float* part_o;               // [B, H, nsplit, RP]
  float* part_ml;              // [B, H, nsplit, 2]
  __nv_bfloat16* out;          // [B, H, RP] when nsplit == 1
  int* error;
};

__device__ __forceinline__ bool mbar_test(uint64_t* bar, uint32_t parity) {       // one look, no suspension
  uint32_t ok;
  asm volatile("{\n\t.reg .pred p;\n\tmbarrier.test_wait.parity.shared::cta.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}\n"
               : "=r"(ok) : "r"(smem_u32(bar)), "r"(parity) : "memory");
  return ok != 0;
}

__host__ __device__ inline uint32_t smem_bytes(int hb, int chunks) {
  return (uint32_t)chunks * hb * 128u + 2u * chunks * CHUNK + hb * 128u;
}

constexpr uint32_t idesc_a_mn(int m, int n) { return idesc_bf16(m, n, false) | (1u << 15); }

template <int HB>
__global__ void __launch_bounds__(THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap map, const __grid_constant__ CUtensorMap map_q,
                     const __grid_constant__ Params p) {
  extern __shared__ unsigned char smem_raw[];
  unsigned char* smem = reinterpret_cast<unsigned char*>(
      (reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  __shared__ uint64_t q_full, k_full[2], k_empty[2], s_full[2], s_free[2], p_ready, pv_done;
  __shared__ uint32_t tmem_slot;
  __shared__ float corr_s[HB], l_part[2][HB];
  __shared__ int moved[SM_WARPS];
  constexpr int NQ = HB / 32;                           // TMEM lane quarters that hold heads
  constexpr uint32_t TMEM_COLS = HB == 32 ? 256 : 512;  // S0 | S1 | O^T: HB columns per 128 latents (4 at most)
  constexpr uint32_t TMEM_O = 2 * KT;

  const int split = blockIdx.x, h0 = blockIdx.y * HB, b = blockIdx.z;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n = p.context_lens[b];
  const int lo = p.window > 0 ? max(n - p.window, 0) : 0, tile0 = lo / KT;      // first key, its tile
  const int all_tiles = (n + KT - 1) / KT, per = (all_tiles - tile0 + p.nsplit - 1) / p.nsplit;
  const int first = tile0 + split * per, n_tiles = min(all_tiles, first + per) - first;
  const int heads = min(HB, p.H - h0);
  const long long row0 = (long long)b * p.H + h0;       // first (sequence, head) of this CTA
  bool fits;
  {
    uint32_t dyn;
    asm volatile("mov.u32 %0, %%dynamic_smem_size;\n" : "=r"(dyn));
    fits = (uint32_t)(smem - smem_raw) + smem_bytes(HB, p.chunks) <= dyn;
    if (!fits && threadIdx.x == 0) atomicCAS(p.error, 0, ERR_SMEM);
  }
  if (n_tiles <= 0 || !fits) {                          // uniform for the CTA: no keys in this range
    for (int i = threadIdx.x; i < heads; i += THREADS)
      if (p.nsplit > 1) {
        p.part_ml[((row0 + i) * p.nsplit + split) * 2] = -INFINITY;
        p.part_ml[((row0 + i) * p.nsplit + split) * 2 + 1] = 0.f;
      }
    if (p.nsplit == 1)
      for (int i = threadIdx.x; i < heads * p.RP; i += THREADS) p.out[row0 * p.RP + i] = __float2bfloat16_rn(0.f);
    return;
  }
  const uint32_t q_chunk = HB * 128u, stage_bytes = p.chunks * CHUNK;
  unsigned char* sQ = smem;
  unsigned char* sK = sQ + p.chunks * q_chunk;
  unsigned char* sP = sK + 2 * stage_bytes;

  if (threadIdx.x == 0) {
    mbar_init(&q_full, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&s_full[i], 1);
      mbar_init(&s_free[i], 2 * NQ);
    }
    mbar_init(&p_ready, SM_WARPS);
    mbar_init(&pv_done, 1);
    asm volatile("fence.mbarrier_init.release.cluster;\n" ::: "memory");
  }
  if (warp == MMA_WARP) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;\n" ::"r"(smem_u32(&tmem_slot)),
                 "r"(TMEM_COLS));
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;\n" ::);
  }
  fence_before();
  __syncthreads();
  fence_after();
  const uint32_t tmem = tmem_slot;
  const int m_blocks = (p.RP + 127) / 128;

  if (warp == TMA_WARP) {
    // ---------------- cache rows ----------------
    if (elect_one()) {
      const int* bt = p.block_tables + (long long)b * p.max_blocks;
      const int bs = p.block_size, per_tile = KT / bs, last_block = (n + bs - 1) / bs;
      const int boxes = (p.CP + 63) / 64;
      const uint32_t box_bytes = (uint32_t)bs * 128u;
      // HB rows from the first head on; rows past this sequence's heads belong to the next one or are zero, and
      // their scores are never used
      mbar_expect_tx(&q_full, (uint32_t)boxes * q_chunk);
      for (int c = 0; c < boxes; ++c) tma_load_2d(sQ + c * q_chunk, &map_q, &q_full, c * 64, (int)row0);
      bool ok = true;
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int st = j & 1;
        const uint32_t use = j >> 1;
        const int blk0 = (first + j) * per_tile, nb = min(per_tile, last_block - blk0);
        int rows[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) rows[i] = i < nb ? __ldg(bt + blk0 + i) * bs : 0;
        if (use > 0) ok = mbar_wait(&k_empty[st], (use - 1) & 1, p.error, ERR_EMPTY);
        if (!ok) break;
        mbar_expect_tx(&k_full[st], (uint32_t)(nb * boxes) * box_bytes);
        unsigned char* dst = sK + st * stage_bytes;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          if (i < nb)
            for (int c = 0; c < boxes; ++c) tma_load_2d(dst + c * CHUNK + i * box_bytes, &map, &k_full[st], c * 64, rows[i]);
        }
      }
    }
  } else if (warp == MMA_WARP) {
    // ---------------- products ----------------
    if (elect_one()) {
      constexpr uint32_t id_s = idesc_bf16(128, KT, false);
      constexpr uint32_t id_o = idesc_a_mn(128, HB);
      const uint32_t q_addr = smem_u32(sQ), k_base = smem_u32(sK), p_addr = smem_u32(sP);
      const int k_steps = p.CP / 16;
      auto issue_s = [&](int j) -> bool {
        const int st = j & 1;
        if (!mbar_wait(&k_full[st], (j >> 1) & 1, p.error, ERR_K)) return false;
        if (j >= 2 && !mbar_wait(&s_free[st], ((j >> 1) - 1) & 1, p.error, ERR_FREE)) return false;
        fence_after();
        const uint32_t k_addr = k_base + st * stage_bytes;
#pragma unroll 4
        for (int kk = 0; kk < k_steps; ++kk)
          umma(tmem + st * KT, desc_sw128(q_addr + (kk >> 2) * q_chunk + (kk & 3) * 32, 16, 1024),
               desc_sw128(k_addr + (kk >> 2) * CHUNK + (kk & 3) * 32, 16, 1024), id_s, kk > 0 ? 1u : 0u);
        commit(&s_full[st]);
        return true;
      };
      bool ok = mbar_wait(&q_full, 0, p.error, ERR_Q);
      if (ok) ok = issue_s(0);
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int st = j & 1;
        // The next tile's scores run during this soft-max, unless its rows are still on their way when P is ready:
        // the product comes first then, because it frees the stage that the tile after waits for.
        bool next = j + 1 < n_tiles, ahead = false;
        for (int poll = 0; next && poll < 4096; ++poll) {
          if (mbar_test(&k_full[st ^ 1], ((j + 1) >> 1) & 1)) {
            ahead = true;
            break;
          }
          if (mbar_test(&p_ready, j & 1)) break;
        }
        if (ahead) {
          ok = issue_s(j + 1);
          next = false;
        }
        if (!ok) break;
        ok = mbar_wait(&p_ready, j & 1, p.error, ERR_P);
        if (!ok) break;
        fence_after();
        const uint32_t v_addr = k_base + st * stage_bytes;
        for (int mb = 0; mb < m_blocks; ++mb) {
#pragma unroll
          for (int kk = 0; kk < KT / 16; ++kk)
            umma(tmem + TMEM_O + mb * HB, desc_sw128(v_addr + mb * 2 * CHUNK + kk * 2048, CHUNK, 1024),
                 desc_sw128(p_addr + kk * 32, 16, 1024), id_o, (j > 0 || kk > 0) ? 1u : 0u);
        }
        commit(&pv_done);
        commit(&k_empty[st]);
        if (next) ok = issue_s(j + 1);
      }
    }
  } else {
    // ---------------- soft-max, output ----------------
    const int wg = warp >> 2, quarter = warp & 3;
    const uint32_t lane_base = (uint32_t)(quarter * 32) << 16;
    const bool scores = quarter < NQ;                   // this warp's lanes hold heads
    const int row = quarter * 32 + lane;                // head inside the CTA (score warps)
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int j = 0; j < n_tiles; ++j) {
      const int sb = j & 1;
      const int valid = min(KT, n - (first + j) * KT), from = lo - (first + j) * KT;      // keys [from, valid) of the tile
      float s[32];
      float corr = 1.f;
      ok = ok && mbar_wait_warp(&s_full[sb], (j >> 1) & 1, p.error, ERR_S);
      if (ok && scores) {
        fence_after();
        float t[32];
        float mx = -INFINITY;
        tmem_ld32(tmem + lane_base + sb * KT + (wg ^ 1) * 32, t);
#pragma unroll
        for (int i = 0; i < 32; ++i) mx = fmaxf(mx, (wg ^ 1) * 32 + i < valid && (wg ^ 1) * 32 + i >= from ? t[i] : -INFINITY);
        tmem_ld32(tmem + lane_base + sb * KT + wg * 32, s);
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          s[i] = wg * 32 + i < valid && wg * 32 + i >= from ? s[i] : -INFINITY;
          mx = fmaxf(mx, s[i]);
        }
        fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&s_free[sb]);        // the score buffer may be overwritten
        mx *= p.scale_log2;                             // scale > 0; finite: a tile holds at least one key
        float m_new = fmaxf(m_run, mx);
        if (m_run != -INFINITY && m_new - m_run <= 8.f) m_new = m_run;
        corr = exp2f(m_run - m_new);
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < 32; ++i) {
          s[i] = exp2f(fmaf(s[i], p.scale_log2, -m_new));
          sum += s[i];
        }
        l_run = l_run * corr + sum;
        m_run = m_new;
      }
      // the previous product must be finished before P is overwritten or O^T is rescaled
      if (ok && j > 0) ok = mbar_wait_warp(&pv_done, (j - 1) & 1, p.error, ERR_PV);
      if (ok && scores) {
#pragma unroll
        for (int c = 0; c < 4; ++c)
          *reinterpret_cast<bf16x8*>(sP + (row >> 3) * 1024 + (row & 7) * 128 + (((wg * 4 + c) ^ (row & 7)) << 4)) = pack8(&s[c * 8]);
        if (wg == 0) corr_s[row] = corr;
      }
      const bool any_moved = __any_sync(0xffffffffu, ok && scores && j > 0 && corr != 1.f);
      if (lane == 0) moved[warp] = any_moved ? 1 : 0;
      if (ok && valid < KT) {
        // rows past the end of the sequence: zero in every chunk that the product reads
        ok = mbar_wait_warp(&k_full[sb], (j >> 1) & 1, p.error, ERR_K);
        if (ok) {
          unsigned char* st = sK + sb * stage_bytes;
          const int rows = KT - valid, total = 2 * m_blocks * rows * 8;          // 16-byte pieces
          for (int i = threadIdx.x; i < total; i += SM_WARPS * 32) {
            const int piece = i & 7, rr = (i >> 3) % rows, c = (i >> 3) / rows, r = valid + rr;
            *reinterpret_cast<uint4*>(st + c * CHUNK + (r >> 3) * 1024 + (r & 7) * 128 + piece * 16) = make_uint4(0u, 0u, 0u, 0u);
          }
        }
      }
      asm volatile("fence.proxy.async.shared::cta;\n" ::: "memory");             // generic smem writes -> UMMA reads
      asm volatile("bar.sync 1, 256;\n" ::: "memory");                          // every soft-max thread, every tile
      bool rescale = false;
#pragma unroll
      for (int w = 0; w < NQ; ++w) rescale |= moved[w] != 0;                     // warps 0 .. NQ - 1 cover all heads
      if (ok && rescale) {
        fence_after();
        for (int mb = wg; mb < m_blocks; mb += 2) {
#pragma unroll
          for (int x = 0; x < NQ; ++x) {
            float t[32];
            const uint32_t at = tmem + TMEM_O + lane_base + mb * HB + x * 32;
            tmem_ld32(at, t);
#pragma unroll
            for (int i = 0; i < 32; ++i) t[i] *= corr_s[x * 32 + i];
            tmem_st32(at, t);
          }
        }
      }
      fence_before();
      __syncwarp();
      if (lane == 0 && ok) mbar_arrive(&p_ready);
      // a warp whose wait gave up stays in the loop (the others meet it in the barrier) but does nothing more
    }
    if (ok) ok = mbar_wait_warp(&pv_done, (n_tiles - 1) & 1, p.error, ERR_PV);
    if (scores) l_part[wg][row] = l_run;
    asm volatile("bar.sync 1, 256;\n" ::: "memory");
    if (scores && wg == 0 && row < heads && p.nsplit == 1)
      corr_s[row] = p.tail.scale2(b, h0 + row, m_run, l_part[0][row] + l_part[1][row]);      // its last use was before the barrier
    asm volatile("bar.sync 1, 256;\n" ::: "memory");
    if (scores && wg == 0 && row < heads && p.nsplit > 1) {
      float* ml = p.part_ml + ((row0 + row) * p.nsplit + split) * 2;
      ml[0] = ok ? m_run : -INFINITY;
      ml[1] = ok ? l_part[0][row] + l_part[1][row] : 0.f;
    }
    ok = __all_sync(0xffffffffu, ok);
    if (ok) {
      fence_after();
      for (int mb = wg; mb < m_blocks; mb += 2) {
        const int c = mb * 128 + quarter * 32 + lane;                            // latent column of this lane
#pragma unroll
        for (int x = 0; x < NQ; ++x) {
          float v[32];
          tmem_ld32(tmem + TMEM_O + lane_base + mb * HB + x * 32, v);
          if (c < p.RP) {
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              const int h = x * 32 + i;
              if (h < heads) {
                if (p.nsplit == 1) {
                  p.out[(row0 + h) * p.RP + c] = __float2bfloat16_rn(v[i] * corr_s[h]);
                } else {
                  p.part_o[((row0 + h) * p.nsplit + split) * p.RP + c] = v[i];
                }
              }
            }
          }
        }
      }
    }
  }
  fence_before();
  __syncthreads();
  if (warp == MMA_WARP)
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;\n" ::"r"(tmem), "r"(TMEM_COLS));
}

static PFN_cuTensorMapEncodeTiled_v12000 encode_fn() {
  static PFN_cuTensorMapEncodeTiled_v12000 fn = nullptr;
  if (fn == nullptr) {
    void* ptr = nullptr;
    cudaDriverEntryPointQueryResult qres;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &ptr, cudaEnableDefault, &qres) == cudaSuccess &&
        qres == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<PFN_cuTensorMapEncodeTiled_v12000>(ptr);
  }
  return fn;
}

// a [rows, CP] bf16 matrix (the paged cache, all query heads); box = `box_rows` rows x 64 columns
static bool make_map(CUtensorMap* map, const void* base, long long rows, int CP, int box_rows) {
  auto fn = encode_fn();
  if (fn == nullptr || (reinterpret_cast<uintptr_t>(base) & 15) != 0 || CP % 8 != 0) return false;
  cuuint64_t dims[2] = {(cuuint64_t)CP, (cuuint64_t)rows};
  cuuint64_t strides[1] = {(cuuint64_t)CP * 2};
  cuuint32_t box[2] = {64u, (cuuint32_t)box_rows};
  cuuint32_t estr[2] = {1, 1};
  return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base), dims, strides, box, estr,
            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int HB>
static int launch(const CUtensorMap& map, const void* q, const Params& p, int batch, cudaStream_t st) {
  CUtensorMap map_q;
  if (!make_map(&map_q, q, (long long)batch * p.H, p.CP, HB)) return (int)cudaErrorNotSupported;
  const int smem = (int)smem_bytes(HB, p.chunks) + 1024;
  if (smem > 231 * 1000) return (int)cudaErrorNotSupported;      // static shared memory shares the 227 KiB
  static int allowed = 0;
  if (smem > allowed) {
    const cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<HB>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return (int)e;
    allowed = smem;
  }
  const dim3 grid((unsigned)p.nsplit, (unsigned)((p.H + HB - 1) / HB), (unsigned)batch);
  latent_decode_kernel<HB><<<grid, THREADS, smem, st>>>(map, map_q, p);
  return (int)cudaGetLastError();
}

}  // namespace ld5
}  // namespace msrl

using namespace msrl;

// The arguments of msrl_latent_decode_mma (latent_attention.cu) plus the number of cache blocks and a status word; key
// ranges are left in part_o / part_ml for msrl_latent_decode_combine.  Returns cudaErrorNotSupported for shapes it does not cover.
MSRL_API int msrl_latent_decode_tcgen05(const void* q, const void* cache, long long num_blocks, const int* block_tables,
                                        int max_blocks, int block_size, const int* context_lens, float scale, int batch,
                                        int H, int CP, int RP, int nsplit, int window, const void* gate, long long gate_ld,
                                        const float* sink, float* part_o, float* part_ml, void* out, int* error,
                                        cudaStream_t st) {
  if (batch == 0) return 0;
  if (CP % 16 != 0 || RP % 16 != 0 || RP > 512 || batch > 65535 || !(scale > 0.f) || block_size < 8 ||
      ld5::KT % block_size != 0 || (reinterpret_cast<uintptr_t>(q) & 15) != 0)
    return (int)cudaErrorNotSupported;
  CUtensorMap map;
  if (!ld5::make_map(&map, cache, num_blocks * block_size, CP, block_size)) return (int)cudaErrorNotSupported;
  const int boxes = (CP + 63) / 64, blocks = 2 * ((RP + 127) / 128);
  ld5::Params p{block_tables, max_blocks, block_size, context_lens,
                scale * 1.4426950408889634f, H, CP, RP, nsplit, window, {(const __nv_bfloat16*)gate, gate_ld, sink}, boxes > blocks ? boxes : blocks, part_o, part_ml,
                (__nv_bfloat16*)out, error};
  return H <= 32 ? ld5::launch<32>(map, q, p, batch, st) : ld5::launch<64>(map, q, p, batch, st);
}
