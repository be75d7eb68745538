// Where pooled rows live: row b is the mean of tokens b P .. b P + P - 1 of a sequence.  Eight neighbours are one group, kept together in the page of
// the first token of the group's first block, one group behind the other where several start in a page.
#pragma once

namespace ne {

__host__ __device__ __forceinline__ void pooled_group(int g, int pool, int block_size, int& page, int& row) {
  if (block_size == 64) {                     // in 32 bits: g * pool is an eighth of a position
    page = (g * pool) >> 3;
    row = pool >= 8 ? 0 : (g - (page * 8 + pool - 1) / pool) * 8;
    return;
  }
  page = (int)((8ll * g * pool) / block_size);
  const long long first = ((long long)page * block_size + 8ll * pool - 1) / (8ll * pool);       // first group of that page
  row = (int)(g - first) * 8;
}
__host__ __device__ __forceinline__ void pooled_place(int b, int pool, int block_size, int& page, int& row) {
  pooled_group(b >> 3, pool, block_size, page, row);
  row += b & 7;
}
// pooled rows a token at position i sees behind a window of `window` tokens
__host__ __device__ __forceinline__ int pooled_visible(int i, int window, int pool) { return i - window + 1 >= pool ? (i - window + 1) / pool : 0; }

}  // namespace ne
