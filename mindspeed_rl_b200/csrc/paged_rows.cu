// Cache rows of given (sequence, position) pairs in order, for prompt portions that look at what earlier ones left.
#include "common.cuh"

namespace msrl {

// rows of 16-byte vectors
__global__ void gather_kernel(const uint4* cache, const int* block_tables, int max_blocks, int block_size,
                              const int* token_seq, const int* token_pos, uint4* out, long long rows, int vecs) {
  const long long r = (long long)blockIdx.x * (blockDim.x / 32) + (threadIdx.x >> 5);
  if (r >= rows) return;
  const int pos = token_pos[r];
  const long long slot = (long long)block_tables[(long long)token_seq[r] * max_blocks + pos / block_size] * block_size +
                         pos % block_size;
  for (int c = threadIdx.x & 31; c < vecs; c += 32) out[r * vecs + c] = cache[slot * vecs + c];
}

}  // namespace msrl

using namespace msrl;

MSRL_API int msrl_rows_gather(const void* cache, const int* block_tables, int max_blocks, int block_size,
                                const int* token_seq, const int* token_pos, void* out, long long rows, int row_bytes,
                                cudaStream_t st) {
  if (rows == 0) return 0;
  if (row_bytes % 16 != 0) return (int)cudaErrorInvalidValue;
  gather_kernel<<<(unsigned)((rows + 7) / 8), 256, 0, st>>>((const uint4*)cache, block_tables, max_blocks,
                                                                 block_size, token_seq, token_pos, (uint4*)out, rows,
                                                                 row_bytes / 16);
  return (int)cudaGetLastError();
}

