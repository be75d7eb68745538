// Which sequence, and which of its tiles of `tile` tokens, does a CTA work on?  Tiles never straddle sequences.
#pragma once

namespace ne {

// Whole warp.  seq = -1 when there are fewer than idx + 1 tiles; tok = first token (global index) of the tile.  32 sequences per round with a
// prefix sum of their tile counts.
__device__ __forceinline__ void find_seq_tile(const int* cu, int num_seqs, int tile, int idx, int& seq, int& tok) {
  const int lane = threadIdx.x & 31;
  int rem = idx;
  seq = -1; tok = 0;
  for (int s0 = 0; s0 < num_seqs && seq < 0; s0 += 32) {
    const int s = s0 + lane;
    int q0 = 0, nt = 0;
    if (s < num_seqs) { q0 = cu[s]; nt = (cu[s + 1] - q0 + tile - 1) / tile; }
    int incl = nt;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const int v = __shfl_up_sync(0xffffffffu, incl, o); if (lane >= o) incl += v; }
    const unsigned hit = __ballot_sync(0xffffffffu, rem < incl);
    if (hit) {
      const int l = __ffs(hit) - 1;
      const int before = __shfl_sync(0xffffffffu, incl - nt, l);
      seq = s0 + l;
      tok = __shfl_sync(0xffffffffu, q0, l) + (rem - before) * tile;
    } else {
      rem -= __shfl_sync(0xffffffffu, incl, 31);
    }
  }
}

}  // namespace ne
