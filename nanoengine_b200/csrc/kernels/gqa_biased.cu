// Grouped-query paged attention on tcgen05 tensor cores with per-layer options: any head sizes up to 256 in multiples of 8 (query / key and
// value sizes may differ), any group of query heads per key / value head up to 128, a window of the last keys, capped scores
// cap tanh(s / cap), a distance bias -slope[head] (query position - key position) taken off after the cap, and an output gate: a head's
// output times sigmoid(gate[token, head]) and a constant.  bf16, 64-token pages; decode and prompt portions alike.
//
// One CTA = one KV head x one tile of (token, head of the group) rows of ONE sequence x one slice of the pages its rows can see: pages in
// front of the tile's window are never touched.  r = token_in_tile * g + head_in_group, at most 128 rows.
//
// Per 64-key page:  S = Q K^T   (nc chunks x 4 tcgen05.mma kind::f16, M=128 N=64 K=16; both K-major, 128B swizzle)
//                   cap, bias, mask and online softmax in 32-bit by 128 threads reading S from TMEM; P -> bf16 -> shared memory
//                   O += P V    (4 x tcgen05.mma, N = 64 nv; V read MN-major)
// A head size that is not a multiple of 64 ends in a chunk whose missing columns TMA fills with zeros.  M = 128 rows are always multiplied;
// rows past the tile's own read whatever shared memory follows and feed accumulator rows nobody reads.
// Tiles of at most 32 rows (decode steps) with capped scores, where the softmax is the longer part, are laid out four times (kRep), rows 32 w .. of the products for softmax warp w, and warp w takes only
// keys 16 w .. 16 w + 15 of every page: a quarter of the softmax work each, at no cost in products.  The four partial results of a row
// (own maximum, sum and accumulator) are folded at the end.
// Warp 0: TMA producer, warp 1: MMA issuer, warps 2-5: softmax / rescale / epilogue (those that own rows of the tile).  All waits are
// bounded.  Two CTAs share an SM where the tiles are small enough: one's softmax runs beside the other's products and copies.
// kExt: (1) beside the window a row sees the pooled rows (pooled.cuh) of blocks wholly in front of it: tiles of 64 pooled rows, fetched as eight
// groups of eight, come before the window's pages, in one softmax; (2) a row's output is rotated back by its position (pairs of columns m, m + Dv / 2)
// on its way out, through shared memory.
// keep: the first tokens of a sequence stay visible behind the window; their pages come in front of the window's.
// kDiff: differential attention.  A head has two query vectors and a key / value head two key vectors side by side; the two maps of a (token, head) pair
// are two rows of the tile (the maps in halves of the rows), with zeros where the other map's query would be, so that one pass over keys and values
// serves both.  A pair's rows meet in shared memory (or in the merge kernel): o = a1 - mixing a2, divided by its root mean square, scaled, gated element
// by element.
// With more than one slice the CTA writes a normalised partial result and its log2-sum-exp; gqa_biased_merge folds them and applies the gate.
#include "ptx.cuh"
#include "pooled.cuh"
#include "seq_tile.cuh"
#include "tma_host.h"

namespace ne {

constexpr int kGbThreads = 192;
constexpr int kKernelGb = 13;
constexpr int kBPage = 64;                     // keys per page
constexpr int kBChunk = kBPage * 128;          // one 64-column chunk of a page tile: 64 rows x 128 B
constexpr float kLog2e = 1.4426950408889634f;

struct GbArgs {
  const int* block_tables; int bt_stride;
  const int* cu_seqlens_q; const int* context_lens; int num_seqs;
  int T, H, Dv, g, tq, splits;
  int nc, nv, rows8, stages, pbufs, window;      // kRep: rows8 = 128
  uint32_t tmem_cols;
  float scale, softcap;
  const float* slopes;                         // [H] or null
  const __nv_bfloat16* gate; long long gate_ld; float out_scale;
  __nv_bfloat16* out; long long o_ld;          // row t, head h: out + t o_ld + h Dv (splits == 1)
  float* part; float* lse2;                    // [splits, T, H, Dv], [splits, T, H] (splits > 1)
  int pool;                                    // kExt: tokens per pooled row (0: none)
  const float* turn; int n_pos;                // kExt: [n_pos, Dv] cos | sin, or null
  int bar_off;                                 // where the barriers lie in shared memory
  int keep;                                    // first keys that stay visible behind the window
  const float* mixing; float eps; const __nv_bfloat16* egate; long long egate_ld;      // kDiff; out_scale is part of it
};

__device__ __forceinline__ float gate_of(const __nv_bfloat16* gate, long long ld, long long t, int h, float scale) {
  return gate ? scale / (1.f + __expf(-__bfloat162float(gate[t * ld + h]))) : scale;
}

__device__ __forceinline__ float sigmoid_of(float x) { return 1.f / (1.f + __expf(-x)); }

template <bool kCap, bool kRep, bool kExt, bool kDiff = false>
__global__ void __launch_bounds__(kGbThreads, 2)
gqa_biased_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap v_map,
                  const __grid_constant__ CUtensorMap kp_map, const __grid_constant__ CUtensorMap vp_map, const GbArgs a) {
  pdl_wait();                     // dependent launch: nothing above this line touches global memory
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = smem_raw;      // swizzled tiles need 1024-byte alignment: the dynamic allocation starts on such a boundary
  if (smem_u32(smem) & 1023) { if (threadIdx.x == 0) report(ST_BAD_ARG, kKernelGb, 1, 0); return; }
  const int q_chunk = a.rows8 * 128, p_bytes = a.rows8 * 128, stage_bytes = (a.nc + a.nv) * kBChunk;
  uint8_t* sQ = smem;                                    // nc chunks of rows8 x 128 B
  uint8_t* sP = sQ + a.nc * q_chunk;
  uint8_t* sKV = sP + a.pbufs * p_bytes;                 // MMA reads of rows past rows8 end inside the page tiles
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + a.bar_off);
  // q_full | kv_full[4] | kv_empty[4] | s_full[2] | s_empty[2] | p_full[2] | p_empty[2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 17);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* s_tile = reinterpret_cast<int*>(tmem_slot + 2);
  const uint32_t b_qfull = smem_u32(bars), b_kvfull = smem_u32(bars + 1), b_kvempty = smem_u32(bars + 5);
  const uint32_t b_sfull = smem_u32(bars + 9), b_sempty = smem_u32(bars + 11), b_pfull = smem_u32(bars + 13), b_pempty = smem_u32(bars + 15);

  const int warp = threadIdx.x >> 5;
  const int hkv = blockIdx.y, split = blockIdx.z;
  const int pairs = a.g * a.tq, half_rows = a.rows8 >> 1;           // kDiff: rows [0, pairs) are the first maps, [half_rows, half_rows + pairs) the second
  const int live_warps = kRep ? 4 : ((kDiff ? half_rows + pairs : pairs) + 31) / 32;         // softmax warps with rows of the tile
  if constexpr (kDiff) {
    for (int i = threadIdx.x; i < a.nc * half_rows * 8; i += kGbThreads) {
      const int c = i / (half_rows * 8), r = i - c * half_rows * 8;
      reinterpret_cast<uint4*>(sQ + c * q_chunk + (c < a.nc >> 1 ? half_rows * 128 : 0))[r] = make_uint4(0, 0, 0, 0);      // the other map's rows
    }
    fence_proxy_async_smem();
  }
  if (warp == 0) {
    int seq, tok;
    find_seq_tile(a.cu_seqlens_q, a.num_seqs, a.tq, blockIdx.x, seq, tok);
    if (lane_id() == 0) { s_tile[0] = seq; s_tile[1] = tok; }
  }
  if (threadIdx.x == 0) {
    mbar_init(b_qfull, 1);
    for (int i = 0; i < 4; i++) { mbar_init(b_kvfull + 8 * i, 1); mbar_init(b_kvempty + 8 * i, 1); }
    for (int i = 0; i < 2; i++) {
      mbar_init(b_sfull + 8 * i, 1); mbar_init(b_sempty + 8 * i, live_warps); mbar_init(b_pfull + 8 * i, live_warps); mbar_init(b_pempty + 8 * i, 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(smem_u32(tmem_slot), a.tmem_cols); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  pdl_trigger();                  // behind the TMEM allocation: a CTA of the next grid never holds columns this grid waits for
  const uint32_t tmem_base = *tmem_slot, tmem_o = tmem_base + 128;
  const int seq = s_tile[0], tok0 = s_tile[1];

  int n_tiles = 0, pg0 = 0, kept = 0, skip = 0, n_tok = 0, base_limit = -1;       // tile i that is no tile of pooled rows: page_of(i)
  int n_pt = 0, n_pool = 0, pt_first = 0;                // tiles of pooled rows in front of the pages, pooled rows visible to the tile's last token
  const int* bt = a.block_tables;
  if (seq >= 0) {
    const int q_beg = a.cu_seqlens_q[seq], q_len = a.cu_seqlens_q[seq + 1] - q_beg;
    n_tok = min(a.tq, q_beg + q_len - tok0);
    base_limit = a.context_lens[seq] - q_len + (tok0 - q_beg);              // last key visible to the tile's first token
    const int max_limit = base_limit + n_tok - 1;
    const int first = a.window > 0 ? max(0, base_limit - a.window + 1) / kBPage : 0;
    if (kExt && a.pool) { n_pool = pooled_visible(max_limit, a.window, a.pool); n_pt = (n_pool + kBPage - 1) / kBPage; }
    kept = min((a.keep + kBPage - 1) / kBPage, first);                      // pages of kept keys in front of the window's
    skip = first - kept;
    const int pages = max_limit >= 0 ? max_limit / kBPage + 1 - skip : 0, total = pages + n_pt;
    const int per_split = (total + a.splits - 1) / a.splits;
    pt_first = split * per_split;
    n_tiles = max(0, min(total, pt_first + per_split) - pt_first);
    pg0 = pt_first - n_pt;                                                  // tiles of pooled rows come first
    n_pt = max(0, -pg0);                                                    // those of this slice
    bt = a.block_tables + (long long)seq * a.bt_stride;
  }

  auto page_of = [&](int i) { const int l = pg0 + i; return l < kept ? l : l + skip; };
  if (warp == 0) {
    if (n_tiles > 0 && elect_one()) {
      constexpr int kCopies = kRep ? 4 : 1;
      mbar_expect_tx(b_qfull, kCopies * a.nc * a.g * a.tq * 128);
      const int nc1 = a.nc >> 1;                              // kDiff: chunks per map
      if constexpr (kDiff) {
        for (int c = 0; c < a.nc; c++) {
          const int m = c >= nc1;
          tma_load_4d(smem_u32(sQ + c * q_chunk + m * half_rows * 128), &q_map, b_qfull, (c - m * nc1) * 64, m, hkv * a.g, tok0);
        }
      } else
      for (int r = 0; r < kCopies; r++)
        for (int c = 0; c < a.nc; c++) tma_load_3d(smem_u32(sQ + c * q_chunk + r * 32 * 128), &q_map, b_qfull, c * 64, hkv * a.g, tok0);
      for (int i = 0; i < n_tiles; i++) {
        const int s = i % a.stages;
        if (!mbar_wait(b_kvempty + 8 * s, ((i / a.stages) & 1) ^ 1, abort_flag, kKernelGb, 100 + s)) break;
        uint8_t* dst = sKV + s * stage_bytes;
        if (kExt && i < n_pt) {
          int page[8], prow[8];
#pragma unroll
          for (int j = 0; j < 8; j++) pooled_group(min((pt_first + i) * 8 + j, (n_pool - 1) >> 3), a.pool, kBPage, page[j], prow[j]);      // past the last: masked
#pragma unroll
          for (int j = 0; j < 8; j++) { page[j] = bt[page[j]]; if (!NE_INDEX_OK(page[j], BK_CACHE_PAGES, kKernelGb, __LINE__)) page[j] = 0; }
          mbar_expect_tx(b_kvfull + 8 * s, stage_bytes);
          for (int c = 0; c < a.nc; c++)
#pragma unroll
            for (int j = 0; j < 8; j++) tma_load_4d(smem_u32(dst + c * kBChunk + j * 1024), &kp_map, b_kvfull + 8 * s, c * 64, hkv, prow[j], page[j]);
          for (int c = 0; c < a.nv; c++)
#pragma unroll
            for (int j = 0; j < 8; j++) tma_load_4d(smem_u32(dst + (a.nc + c) * kBChunk + j * 1024), &vp_map, b_kvfull + 8 * s, c * 64, hkv, prow[j], page[j]);
          continue;
        }
        int block = bt[page_of(i)];
        if (!NE_INDEX_OK(block, BK_CACHE_PAGES, kKernelGb, __LINE__)) block = 0;      // a bad page id reads page 0
        mbar_expect_tx(b_kvfull + 8 * s, stage_bytes);
        if constexpr (kDiff) {
          for (int c = 0; c < a.nc; c++) {
            const int m = c >= nc1;
            tma_load_4d(smem_u32(dst + c * kBChunk), &k_map, b_kvfull + 8 * s, (c - m * nc1) * 64, 2 * hkv + m, 0, block);
          }
        } else
        for (int c = 0; c < a.nc; c++) tma_load_4d(smem_u32(dst + c * kBChunk), &k_map, b_kvfull + 8 * s, c * 64, hkv, 0, block);
        for (int c = 0; c < a.nv; c++) tma_load_4d(smem_u32(dst + (a.nc + c) * kBChunk), &v_map, b_kvfull + 8 * s, c * 64, hkv, 0, block);
      }
    }
  } else if (warp == 1) {
    if (n_tiles > 0 && elect_one()) {
      constexpr uint32_t kIdescQK = make_idesc(FMT_BF16, FMT_BF16, 128, kBPage);
      const uint32_t idesc_pv = make_idesc(FMT_BF16, FMT_BF16, 128, (uint32_t)a.nv * 64, 0, 1);      // B (= V) is MN-major
      bool ok = mbar_wait(b_qfull, 0, abort_flag, kKernelGb, 200);
      const uint32_t q_addr = smem_u32(sQ), p_addr = smem_u32(sP), kv_addr = smem_u32(sKV);
      auto pv = [&](int j) -> bool {
        const int pb = j % a.pbufs;
        if (!mbar_wait(b_pfull + 8 * pb, (j / a.pbufs) & 1, abort_flag, kKernelGb, 230)) return false;
        tc_fence_after();
        const int s = j % a.stages;
        const uint32_t vt = kv_addr + s * stage_bytes + a.nc * kBChunk;
#pragma unroll
        for (int ks = 0; ks < 4; ks++) {                     // 16 keys per MMA
          const uint64_t adesc = make_smem_desc(p_addr + pb * p_bytes + ks * 32, 16, 1024, SW_128B);
          const uint64_t bdesc = make_smem_desc(vt + ks * 16 * 128, kBChunk, 1024, SW_128B);
          umma_f16(tmem_o, adesc, bdesc, idesc_pv, (j | ks) != 0);
        }
        tc_commit(b_kvempty + 8 * s);
        tc_commit(b_pempty + 8 * pb);
        return true;
      };
      // barriers that gate S(i+1) are tested before the MMAs of S(i) are issued (see gqa_bf16.cu)
      bool pre_se = true, pre_kv = mbar_test(b_kvfull, 0);
      for (int i = 0; ok && i < n_tiles; i++) {
        const int sb = i & 1, s = i % a.stages;
        if (!pre_se && !mbar_wait(b_sempty + 8 * sb, ((i >> 1) & 1) ^ 1, abort_flag, kKernelGb, 210 + sb)) { ok = false; break; }
        if (!pre_kv && !mbar_wait(b_kvfull + 8 * s, (i / a.stages) & 1, abort_flag, kKernelGb, 220 + s)) { ok = false; break; }
        mbar_test2(b_sempty + 8 * ((i + 1) & 1), (((i + 1) >> 1) & 1) ^ 1, b_kvfull + 8 * ((i + 1) % a.stages), ((i + 1) / a.stages) & 1, pre_se, pre_kv);
        tc_fence_after();
        const uint32_t kt = kv_addr + s * stage_bytes, d = tmem_base + sb * kBPage;
        for (int c = 0; c < a.nc; c++) {
#pragma unroll
          for (int ks = 0; ks < 4; ks++) {
            const uint64_t adesc = make_smem_desc(q_addr + c * q_chunk + ks * 32, 16, 1024, SW_128B);
            const uint64_t bdesc = make_smem_desc(kt + c * kBChunk + ks * 32, 16, 1024, SW_128B);
            umma_f16(d, adesc, bdesc, kIdescQK, (c | ks) != 0);
          }
        }
        tc_commit(b_sfull + 8 * sb);
        if (i > 0 && !pv(i - 1)) { ok = false; break; }
      }
      if (ok) pv(n_tiles - 1);
    }
  } else if ((warp & 3) < live_warps) {
    const int wq = warp & 3;
    const int row = wq * 32 + (int)lane_id();
    const uint32_t lane_addr = (uint32_t)(wq * 32) << 16;
    const int map = kDiff && row >= half_rows;
    const int trow = kRep ? (int)lane_id() : kDiff ? row - map * half_rows : row;             // row of the tile (kDiff: pair)
    const int tl = trow / a.g, head = hkv * a.g + trow % a.g;
    const bool row_ok = trow < pairs && tl < n_tok;
    constexpr int kKeys = kRep ? 16 : 64;                     // keys of a page this thread scores, from kfirst on
    const int kfirst = kRep ? wq * 16 : 0;
    const int limit = row_ok ? base_limit + tl : -1;          // this row's last visible key
    const int lowest = (row_ok && a.window > 0) ? limit - a.window + 1 : 0;
    const int pool_last = kExt && a.pool ? pooled_visible(limit, a.window, a.pool) - 1 : -1;      // last visible pooled row
    const float slope = (row_ok && a.slopes) ? __ldg(a.slopes + head) * kLog2e : 0.f;
    const float c_in = kCap ? a.scale / a.softcap * (2.f * kLog2e) : a.scale * kLog2e, c_cap = a.softcap * kLog2e;
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true, s_ready = false;
    if constexpr (kRep)                                       // the columns of the other warps' keys stay zero
      for (int i = 0; i < a.pbufs * 8; i++) *reinterpret_cast<uint4*>(sP + (i >> 3) * p_bytes + row * 128 + (i & 7) * 16) = make_uint4(0, 0, 0, 0);
    for (int i = 0; ok && i < n_tiles; i++) {
      const int sb = i & 1, pb = i % a.pbufs;
      if (!s_ready && !mbar_wait(b_sfull + 8 * sb, (i >> 1) & 1, abort_flag, kKernelGb, 300 + sb)) { ok = false; break; }
      tc_fence_after();
      uint32_t r[kKeys];
      if constexpr (kRep) {
        tmem_ld_32x32b_x16(tmem_base + lane_addr + sb * kBPage + kfirst, r);
      } else {
        tmem_ld_32x32b_x32(tmem_base + lane_addr + sb * kBPage, *reinterpret_cast<uint32_t(*)[32]>(r));
        tmem_ld_32x32b_x32(tmem_base + lane_addr + sb * kBPage + 32, *reinterpret_cast<uint32_t(*)[32]>(r + 32));
      }
      tc_wait_ld();
      tc_fence_before();
      __syncwarp();
      if (lane_id() == 0) mbar_arrive(b_sempty + 8 * sb);
      const bool pooled = kExt && i < n_pt;
      const int key0 = (pooled ? pt_first + i : page_of(i)) * kBPage + kfirst;
      const int hi = pooled ? pool_last : limit, lo = pooled ? 0 : lowest;
      const bool p_free = i < a.pbufs || mbar_test(b_pempty + 8 * pb, ((i - a.pbufs) / a.pbufs) & 1);     // needed only after the math
      // score in the log2 domain: cap and bias
      const float b0 = slope * (float)(key0 - limit);
      auto score4 = [&](uint32_t* rr4, int j0) {
        float s[4];
#pragma unroll
        for (int e = 0; e < 4; e++) s[e] = __uint_as_float(rr4[e]) * c_in;
        if (kCap) {
          // cap tanh(x) = cap - 2 cap / (e^(2x) + 1); one reciprocal for four: 1/a = bcd / abcd.  e^(2x) up to 2^30, where tanh has long been one.
#pragma unroll
          for (int e = 0; e < 4; e++) s[e] = 1.f + exp2f(fminf(s[e], 30.f));
          const float ab = s[0] * s[1], cd = s[2] * s[3], rr = -2.f * c_cap * __fdividef(1.f, ab * cd);
          const float rab = rr * cd, rcd = rr * ab;
          const float t0 = fmaf(rab, s[1], c_cap), t1 = fmaf(rab, s[0], c_cap), t2 = fmaf(rcd, s[3], c_cap), t3 = fmaf(rcd, s[2], c_cap);
          s[0] = t0; s[1] = t1; s[2] = t2; s[3] = t3;
        }
#pragma unroll
        for (int e = 0; e < 4; e++) rr4[e] = __float_as_uint(s[e] + fmaf(slope, (float)(j0 + e), b0));
      };
#pragma unroll
      for (int j = 0; j < kKeys; j += 4) score4(r + j, j);
      if (key0 + kKeys - 1 > hi || key0 < lo) {
#pragma unroll
        for (int j = 0; j < kKeys; j++)
          if (key0 + j > hi || (key0 + j < lo && key0 + j >= a.keep)) r[j] = 0xff800000u;
      }
      float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int j = 0; j < kKeys; j++) mx[j & 3] = fmaxf(mx[j & 3], __uint_as_float(r[j]));
      const float m_tile = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
      // lazy rescaling: the reference maximum only moves when the page's maximum exceeds it by more than 2^8
      const bool first_valid = (m_run == -INFINITY);
      const float m_new = (first_valid || m_tile > m_run + 8.f) ? fmaxf(m_run, m_tile) : m_run;
      const float alpha = (m_new == -INFINITY || first_valid) ? 1.f : exp2f(m_run - m_new);
      const float neg_m = (m_new == -INFINITY) ? 0.f : -m_new;
      float psum = 0.f;
      uint32_t pk[kKeys / 2];
#pragma unroll
      for (int j = 0; j < kKeys / 2; j++) {
        pk[j] = pack_bf16x2(exp2f(__uint_as_float(r[2 * j]) + neg_m), exp2f(__uint_as_float(r[2 * j + 1]) + neg_m));
        // sum what the MMA will see (bf16-rounded probabilities), so numerator and denominator stay consistent
        const float2 q = unpack_bf16x2(pk[j]);
        psum += q.x + q.y;
      }
      l_run = l_run * alpha + psum;
      m_run = m_new;
      if (i > 0 && __any_sync(0xffffffffu, alpha < 1.f)) {
        if (!mbar_wait(b_pempty + 8 * ((i - 1) % a.pbufs), ((i - 1) / a.pbufs) & 1, abort_flag, kKernelGb, 310)) { ok = false; break; }
        tc_fence_after();
#pragma unroll 1
        for (int cblk = 0; cblk < a.nv * 4; cblk++) {
          uint32_t o[16];
          tmem_ld_32x32b_x16(tmem_o + lane_addr + cblk * 16, o);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 16; j++) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
          tmem_st_32x32b_x16(tmem_o + lane_addr + cblk * 16, o);
        }
        tc_wait_st();
      }
      if (!p_free && !mbar_wait(b_pempty + 8 * pb, ((i - a.pbufs) / a.pbufs) & 1, abort_flag, kKernelGb, 311)) { ok = false; break; }
      s_ready = mbar_test(b_sfull + 8 * ((i + 1) & 1), ((i + 1) >> 1) & 1);
      if (row < a.rows8) {       // P row (64 bf16 = 8 chunks of 16 bytes) into the 128B-swizzled K-major layout the MMA reads
        uint8_t* prow = sP + pb * p_bytes + row * 128;
        const int sw = row & 7;
#pragma unroll
        for (int cch = 0; cch < kKeys / 8; cch++)
          *reinterpret_cast<uint4*>(prow + (((kfirst / 8 + cch) ^ sw) << 4)) = make_uint4(pk[4 * cch], pk[4 * cch + 1], pk[4 * cch + 2], pk[4 * cch + 3]);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane_id() == 0) mbar_arrive(b_pfull + 8 * pb);
    }
    if (ok && n_tiles > 0) ok = mbar_wait(b_pempty + 8 * ((n_tiles - 1) % a.pbufs), ((n_tiles - 1) / a.pbufs) & 1, abort_flag, kKernelGb, 320);
    const long long all_rows = (long long)a.T * a.H * (kDiff ? 2 : 1);
    const long long tok = tok0 + tl, orow = row_ok ? (kDiff ? (tok * a.H + head) * 2 + map : tok * a.H + head) : 0;
    const bool have = ok && n_tiles > 0;
    if (have) tc_fence_after();
    if constexpr (kRep) {
      // fold the four partial results of every row: accumulators through shared memory (nothing else uses it any more)
      float* fold = reinterpret_cast<float*>(smem);
      const int ld = a.Dv + 4, rows = a.g * a.tq;
#pragma unroll 1
      for (int cblk = 0; cblk < a.nv * 2; cblk++) {
        uint32_t o[32];
        __syncwarp();                          // the lanes of rows outside the tile skip the stores below
        if (have) {
          tmem_ld_32x32b_x32(tmem_o + lane_addr + cblk * 32, o);
          tc_wait_ld();
        }
        if (!row_ok) continue;
#pragma unroll
        for (int v = 0; v < 8; v++) {
          const int col = cblk * 32 + v * 4;
          if (col >= a.Dv) continue;
          *reinterpret_cast<float4*>(fold + (wq * rows + trow) * ld + 4 + col) =
              have ? make_float4(__uint_as_float(o[4 * v]), __uint_as_float(o[4 * v + 1]), __uint_as_float(o[4 * v + 2]), __uint_as_float(o[4 * v + 3]))
                   : make_float4(0.f, 0.f, 0.f, 0.f);
        }
      }
      if (row_ok) { fold[(wq * rows + trow) * ld] = have ? m_run : -INFINITY; fold[(wq * rows + trow) * ld + 1] = have ? l_run : 0.f; }
      named_bar_sync(1, 128);
      const int groups = a.Dv / 8;
      for (int i = (int)threadIdx.x - 64; i < n_tok * a.g * groups; i += 128) {
        const int rr = i / groups, col = (i - rr * groups) * 8, hd = hkv * a.g + rr % a.g;
        const long long tk = tok0 + rr / a.g;
        float m = -INFINITY, den = 0.f, f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int w = 0; w < 4; w++) m = fmaxf(m, fold[(w * rows + rr) * ld]);
#pragma unroll
        for (int w = 0; w < 4; w++) {
          const float* src = fold + (w * rows + rr) * ld;
          if (src[0] == -INFINITY) continue;
          const float e = exp2f(src[0] - m);
          den += e * src[1];
#pragma unroll
          for (int j = 0; j < 8; j++) f[j] = fmaf(e, src[4 + col + j], f[j]);
        }
        const float inv = (den > 0.f ? 1.f / den : 0.f) * (a.splits == 1 ? gate_of(a.gate, a.gate_ld, tk, hd, a.out_scale) : 1.f);
        if (a.splits == 1) {
          *reinterpret_cast<uint4*>(a.out + tk * a.o_ld + (long long)hd * a.Dv + col) =
              make_uint4(pack_bf16x2(f[0] * inv, f[1] * inv), pack_bf16x2(f[2] * inv, f[3] * inv), pack_bf16x2(f[4] * inv, f[5] * inv), pack_bf16x2(f[6] * inv, f[7] * inv));
        } else {
          const long long o = (long long)split * a.T * a.H + tk * a.H + hd;
          float* dst = a.part + o * a.Dv + col;
          *reinterpret_cast<float4*>(dst) = make_float4(f[0] * inv, f[1] * inv, f[2] * inv, f[3] * inv);
          *reinterpret_cast<float4*>(dst + 4) = make_float4(f[4] * inv, f[5] * inv, f[6] * inv, f[7] * inv);
          if (col == 0) a.lse2[o] = den > 0.f ? m + log2f(den) : -INFINITY;
        }
      }
    } else if (kDiff && a.splits == 1) {
      // rows into shared memory (nothing else uses it any more); one warp per pair from there
      float* fold = reinterpret_cast<float*>(smem);
      const int ld = a.Dv + 4;
      const float inv = (have && l_run > 0.f) ? 1.f / l_run : 0.f;
#pragma unroll 1
      for (int cblk = 0; cblk < a.nv * 2; cblk++) {
        uint32_t o[32];
        __syncwarp();                          // the lanes of rows outside the tile skip the stores below
        if (have) {
          tmem_ld_32x32b_x32(tmem_o + lane_addr + cblk * 32, o);
          tc_wait_ld();
        }
        if (!row_ok) continue;
#pragma unroll
        for (int v = 0; v < 8; v++) {
          const int col = cblk * 32 + v * 4;
          if (col >= a.Dv) continue;
          *reinterpret_cast<float4*>(fold + (map * pairs + trow) * ld + col) =
              have ? make_float4(__uint_as_float(o[4 * v]) * inv, __uint_as_float(o[4 * v + 1]) * inv, __uint_as_float(o[4 * v + 2]) * inv, __uint_as_float(o[4 * v + 3]) * inv)
                   : make_float4(0.f, 0.f, 0.f, 0.f);
        }
      }
      named_bar_sync(1, live_warps * 32);
      const float lam = *a.mixing;
      const int lane = (int)lane_id();
      for (int p = wq; p < n_tok * a.g; p += live_warps) {
        const long long tk = tok0 + p / a.g;
        const int hd = hkv * a.g + p % a.g;
        float f[8], ss = 0.f;
        uint2 gv[2];
#pragma unroll
        for (int it = 0; it < 2; it++) {
          const int col = lane * 4 + it * 128;
          f[4 * it] = f[4 * it + 1] = f[4 * it + 2] = f[4 * it + 3] = 0.f;
          gv[it] = make_uint2(0, 0);
          if (col >= a.Dv) continue;
          gv[it] = *reinterpret_cast<const uint2*>(a.egate + tk * a.egate_ld + (long long)hd * a.Dv + col);
          const float4 x = *reinterpret_cast<const float4*>(fold + p * ld + col), y = *reinterpret_cast<const float4*>(fold + (pairs + p) * ld + col);
          f[4 * it] = x.x - lam * y.x; f[4 * it + 1] = x.y - lam * y.y; f[4 * it + 2] = x.z - lam * y.z; f[4 * it + 3] = x.w - lam * y.w;
          ss += f[4 * it] * f[4 * it] + f[4 * it + 1] * f[4 * it + 1] + f[4 * it + 2] * f[4 * it + 2] + f[4 * it + 3] * f[4 * it + 3];
        }
        const float r = rsqrtf(warp_sum(ss) / (float)a.Dv + a.eps) * a.out_scale;
#pragma unroll
        for (int it = 0; it < 2; it++) {
          const int col = lane * 4 + it * 128;
          if (col >= a.Dv) continue;
          const float2 g0 = unpack_bf16x2(gv[it].x), g1 = unpack_bf16x2(gv[it].y);
          *reinterpret_cast<uint2*>(a.out + tk * a.o_ld + (long long)hd * a.Dv + col) =
              make_uint2(pack_bf16x2(f[4 * it] * r * sigmoid_of(g0.x), f[4 * it + 1] * r * sigmoid_of(g0.y)),
                         pack_bf16x2(f[4 * it + 2] * r * sigmoid_of(g1.x), f[4 * it + 3] * r * sigmoid_of(g1.y)));
        }
      }
    } else if (kExt && a.turn && a.splits == 1) {
      // rows into shared memory (nothing else uses it any more), pairs of columns from there
      float* fold = reinterpret_cast<float*>(smem);
      const int ld = a.Dv + 4, half = a.Dv >> 1;
      const float inv = ((have && l_run > 0.f) ? 1.f / l_run : 0.f) * (row_ok ? gate_of(a.gate, a.gate_ld, tok, head, a.out_scale) : 0.f);
#pragma unroll 1
      for (int cblk = 0; cblk < a.nv * 2; cblk++) {
        uint32_t o[32];
        __syncwarp();                          // the lanes of rows outside the tile skip the stores below
        if (have) {
          tmem_ld_32x32b_x32(tmem_o + lane_addr + cblk * 32, o);
          tc_wait_ld();
        }
        if (!row_ok) continue;
#pragma unroll
        for (int v = 0; v < 8; v++) {
          const int col = cblk * 32 + v * 4;
          if (col >= a.Dv) continue;
          *reinterpret_cast<float4*>(fold + trow * ld + col) =
              have ? make_float4(__uint_as_float(o[4 * v]) * inv, __uint_as_float(o[4 * v + 1]) * inv, __uint_as_float(o[4 * v + 2]) * inv, __uint_as_float(o[4 * v + 3]) * inv)
                   : make_float4(0.f, 0.f, 0.f, 0.f);
        }
      }
      named_bar_sync(1, live_warps * 32);
      const int groups = half / 4, me = wq * 32 + (int)lane_id();      // Dv is a multiple of 8: groups of four pairs
      for (int i = me; i < n_tok * a.g * groups; i += live_warps * 32) {
        const int rr = i / groups, m = (i - rr * groups) * 4, tk = rr / a.g;
        const float* src = fold + rr * ld + m;
        const float* tab = a.turn + (long long)min(base_limit + tk, a.n_pos - 1) * a.Dv + m;
        const float4 x = *reinterpret_cast<const float4*>(src), y = *reinterpret_cast<const float4*>(src + half);
        const float4 c = __ldg(reinterpret_cast<const float4*>(tab)), s = __ldg(reinterpret_cast<const float4*>(tab + half));
        __nv_bfloat16* dst = a.out + (long long)(tok0 + tk) * a.o_ld + (long long)(hkv * a.g + rr % a.g) * a.Dv + m;
        *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16x2(x.x * c.x + y.x * s.x, x.y * c.y + y.y * s.y), pack_bf16x2(x.z * c.z + y.z * s.z, x.w * c.w + y.w * s.w));
        *reinterpret_cast<uint2*>(dst + half) =
            make_uint2(pack_bf16x2(y.x * c.x - x.x * s.x, y.y * c.y - x.y * s.y), pack_bf16x2(y.z * c.z - x.z * s.z, y.w * c.w - x.w * s.w));
      }
    } else {
      float inv = (have && l_run > 0.f) ? 1.f / l_run : 0.f;
      if (a.splits == 1 && row_ok) inv *= gate_of(a.gate, a.gate_ld, tok, head, a.out_scale);
#pragma unroll 1
      for (int cblk = 0; cblk < a.nv * 2; cblk++) {
        uint32_t o[32];
        __syncwarp();                          // the lanes of rows outside the tile skip the stores below
        if (have) {
          tmem_ld_32x32b_x32(tmem_o + lane_addr + cblk * 32, o);
          tc_wait_ld();
        }
        if (!row_ok) continue;
#pragma unroll
        for (int v = 0; v < 4; v++) {                            // Dv is a multiple of 8: whole groups of 8 columns
          const int col = cblk * 32 + v * 8;
          if (col >= a.Dv) continue;
          float f[8];
#pragma unroll
          for (int j = 0; j < 8; j++) f[j] = have ? __uint_as_float(o[v * 8 + j]) * inv : 0.f;
          if (a.splits == 1) {
            *reinterpret_cast<uint4*>(a.out + tok * a.o_ld + (long long)head * a.Dv + col) =
                make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
          } else {
            float* dst = a.part + (split * all_rows + orow) * a.Dv + col;
            *reinterpret_cast<float4*>(dst) = make_float4(f[0], f[1], f[2], f[3]);
            *reinterpret_cast<float4*>(dst + 4) = make_float4(f[4], f[5], f[6], f[7]);
          }
        }
      }
      if (a.splits > 1 && row_ok)
        a.lse2[split * all_rows + orow] = (have && l_run > 0.f) ? m_run + log2f(l_run) : -INFINITY;
    }
  }

  tc_fence_before();
  __syncthreads();
  if (*abort_flag && threadIdx.x == 0) for (int i = 0; i < 2000; i++) __nanosleep(1000);      // copies in flight land before the CTA goes
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, a.tmem_cols); }
}

// out[t, h] = gate * sum_s softmax_s(lse2) part[s, t, h]; one CTA per (token, head)
__global__ void __launch_bounds__(128) gqa_biased_merge_kernel(const GbArgs a) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const long long row = blockIdx.x, rows = (long long)a.T * a.H, t = row / a.H;
  const int h = (int)(row - t * a.H);
  float m = -INFINITY;
  for (int s = 0; s < a.splits; s++) m = fmaxf(m, a.lse2[s * rows + row]);
  float den = 0.f;
  for (int s = 0; s < a.splits; s++) { const float l = a.lse2[s * rows + row]; den += l == -INFINITY ? 0.f : exp2f(l - m); }
  const float inv = den > 0.f ? gate_of(a.gate, a.gate_ld, t, h, a.out_scale) / den : 0.f;
  auto column = [&](int d) {
    float acc = 0.f;
    for (int s = 0; s < a.splits; s++) {
      const float l = a.lse2[s * rows + row];
      if (l != -INFINITY) acc += exp2f(l - m) * a.part[(s * rows + row) * a.Dv + d];
    }
    return acc * inv;
  };
  __nv_bfloat16* out = a.out + t * a.o_ld + (long long)h * a.Dv;
  if (a.turn) {
    int lo = 0, hi = a.num_seqs - 1;          // last sequence whose first token is <= t
    while (lo < hi) { const int mid = (lo + hi + 1) >> 1; if (a.cu_seqlens_q[mid] <= t) lo = mid; else hi = mid - 1; }
    const int pos = min(max(a.context_lens[lo] - a.cu_seqlens_q[lo + 1] + (int)t, 0), a.n_pos - 1), half = a.Dv >> 1;
    const float* tab = a.turn + (long long)pos * a.Dv;
    for (int d = threadIdx.x; d < half; d += blockDim.x) {
      const float x = column(d), y = column(d + half), c = tab[d], s = tab[half + d];
      out[d] = __float2bfloat16(x * c + y * s);
      out[d + half] = __float2bfloat16(y * c - x * s);
    }
    return;
  }
  for (int d = threadIdx.x; d < a.Dv; d += blockDim.x) out[d] = __float2bfloat16(column(d));
}

// kDiff: the slices of both maps, their difference, norm and gate; one warp per (token, head), at most 32 slices
__global__ void __launch_bounds__(128) gqa_diff_merge_kernel(const GbArgs a) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const long long pair = (long long)blockIdx.x * 4 + (threadIdx.x >> 5), rows = (long long)a.T * a.H * 2;
  const int lane = (int)lane_id();
  if (pair >= (long long)a.T * a.H) return;
  const long long t = pair / a.H;
  const int h = (int)(pair - t * a.H);
  const float lam = *a.mixing;
  float f[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int m = 0; m < 2; m++) {
    const long long row = pair * 2 + m;
    const float l = lane < a.splits ? a.lse2[lane * rows + row] : -INFINITY, mx = warp_max(l);
    const float e = l == -INFINITY ? 0.f : exp2f(l - mx), den = warp_sum(e), w = den > 0.f ? (m ? -lam : 1.f) * e / den : 0.f;
#pragma unroll 4
    for (int s = 0; s < a.splits; s++) {
      const float ws = __shfl_sync(0xffffffffu, w, s);
#pragma unroll
      for (int it = 0; it < 2; it++) {
        const int col = lane * 4 + it * 128;
        if (col >= a.Dv || ws == 0.f) continue;
        const float4 v = *reinterpret_cast<const float4*>(a.part + (s * rows + row) * a.Dv + col);
        f[4 * it] = fmaf(ws, v.x, f[4 * it]); f[4 * it + 1] = fmaf(ws, v.y, f[4 * it + 1]);
        f[4 * it + 2] = fmaf(ws, v.z, f[4 * it + 2]); f[4 * it + 3] = fmaf(ws, v.w, f[4 * it + 3]);
      }
    }
  }
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < 8; e++) ss += f[e] * f[e];
  const float r = rsqrtf(warp_sum(ss) / (float)a.Dv + a.eps) * a.out_scale;
#pragma unroll
  for (int it = 0; it < 2; it++) {
    const int col = lane * 4 + it * 128;
    if (col >= a.Dv) continue;
    const uint2 gv = *reinterpret_cast<const uint2*>(a.egate + t * a.egate_ld + (long long)h * a.Dv + col);
    const float2 g0 = unpack_bf16x2(gv.x), g1 = unpack_bf16x2(gv.y);
    *reinterpret_cast<uint2*>(a.out + t * a.o_ld + (long long)h * a.Dv + col) =
        make_uint2(pack_bf16x2(f[4 * it] * r * sigmoid_of(g0.x), f[4 * it + 1] * r * sigmoid_of(g0.y)),
                   pack_bf16x2(f[4 * it + 2] * r * sigmoid_of(g1.x), f[4 * it + 3] * r * sigmoid_of(g1.y)));
  }
}

struct GbPlan { int nc, nv, tq, rep, rows8, stages, pbufs, bar_off, smem; };

// Tile geometry for groups of g heads, head sizes D / Dv and sequences of at most max_q new tokens; false: not covered.
// maps = 2: kDiff, D the size of one map.
static bool gb_plan(int g, int D, int Dv, int max_q, bool rep, bool ext, GbPlan* p, int maps = 1) {
  if (g < 1 || g * maps > 128 || D < 8 || D % 8 || D * maps > 256 || Dv < 8 || Dv % 8 || Dv > 256 || max_q < 1) return false;
  p->nc = (D + 63) / 64 * maps; p->nv = (Dv + 63) / 64;
  p->tq = 128 / (g * maps) < max_q ? 128 / (g * maps) : max_q;
  p->rep = rep && g * p->tq <= 32;
  p->rows8 = p->rep ? 128 : (g * p->tq + 7) / 8 * 8 * maps;
  const int kv = (p->nc + p->nv) * kBChunk, pb = p->rows8 * 128, q = p->nc * pb;
  // two CTAs per SM where half of its shared memory (and of its TMEM columns) holds a tile and two stages, else one with more stages
  const int half = (233472 / 2 - 1024) - 256, whole = 232448 - 256;
  const int limit = p->nv <= 2 && q + pb + 2 * kv <= half ? half : whole;
  p->pbufs = q + 2 * pb + 2 * kv <= limit ? 2 : 1;
  p->stages = (limit - q - p->pbufs * pb) / kv;
  if (p->stages > 4) p->stages = 4;
  if (p->stages < 2) return false;
  const int used = q + p->pbufs * pb + p->stages * kv;
  const int rows_out = ext || maps == 2 ? g * maps * p->tq * (Dv + 4) * 4 : 0;              // the way out of kExt and kDiff
  p->bar_off = ((rows_out > used ? rows_out : used) + 15) / 16 * 16;
  p->smem = p->bar_off + 256;
  if (p->smem > 232448) return false;
  if (p->rep && 4 * g * p->tq * (Dv + 4) * 4 > used) return false;      // the fold's buffer
  // an MMA reads 128 rows from each chunk of Q and from each P buffer: those reads must end inside the allocation
  const int last_q = (p->nc - 1) * p->rows8 * 128 + 16384, last_p = q + (p->pbufs - 1) * p->rows8 * 128 + 16384;
  return (last_q > last_p ? last_q : last_p) <= used;
}

}  // namespace ne

using namespace ne;

// Tokens per tile (0: the shape is not covered)
extern "C" int ne_gqa_biased_plan(int H, int Hkv, int D, int Dv, int max_q, int ext) {
  GbPlan p;
  return Hkv >= 1 && H % Hkv == 0 && gb_plan(H / Hkv, D, Dv, max_q, false, ext != 0, &p) ? p.tq : 0;
}

// q bf16 [T, H, D] (row stride q_ld elements), k_cache bf16 [num_blocks, 64, Hkv, D], v_cache bf16 [num_blocks, 64, Hkv, Dv];
// max_tiles >= sum over sequences of ceil(q_len / tokens per tile).  softcap 0 / slopes null / window 0 / gate null: without.  out bf16, row
// stride o_ld, heads Dv apart.  pool > 0: pooled rows k_pool [num_blocks, pool_rows, Hkv, D], v_pool [.., Dv] (a window, no cap, no slopes); turn:
// [n_pos, Dv] or null.  splits > 1: part fp32 [splits, T, H, Dv], lse2 [splits, T, H]; the merge kernel is launched too.
extern "C" int ne_gqa_biased(const void* q, long long q_ld, const void* k_cache, const void* v_cache, int num_blocks, const int* block_tables, int bt_stride,
                             const int* cu_seqlens_q, const int* context_lens, int num_seqs, int T, int H, int Hkv, int D, int Dv, int max_q, int max_tiles,
                             int splits, float scale, float softcap, const float* slopes, int window, const void* gate, long long gate_ld, float out_scale,
                             void* out, long long o_ld, float* part, float* lse2, const void* k_pool, const void* v_pool, int pool, int pool_rows,
                             const float* turn, int n_pos, int keep, cudaStream_t st) {
  if (T <= 0) return 0;
  if (keep > 0 && pool > 0) return 1004;
  GbPlan p;
  const bool ext = pool > 0 || turn;
  if (ext && (softcap > 0.f || slopes || (turn && n_pos < 1))) return 1003;
  if (pool > 0 && (window < 1 || !k_pool || !v_pool || pool_rows < (kBPage + 8 * pool - 1) / (8 * pool) * 8)) return 1004;
  if (Hkv < 1 || H % Hkv || splits < 1 || (splits > 1 && (!part || !lse2)) || max_tiles < 1) return 1001;
  if (!gb_plan(H / Hkv, D, Dv, max_q, softcap > 0.f, ext, &p) && !gb_plan(H / Hkv, D, Dv, max_q, false, ext, &p)) return 1001;
  if (q_ld % 8 || o_ld % 8 || q_ld < (long long)H * D || (((uintptr_t)q | (uintptr_t)out) & 15)) return 1002;
  const int g = H / Hkv;
  CUtensorMap mq, mk, mv;
  int rc;
  {
    uint64_t dims[3] = {(uint64_t)D, (uint64_t)H, (uint64_t)T}; uint64_t strides[2] = {(uint64_t)D * 2, (uint64_t)q_ld * 2};
    uint32_t box[3] = {64, (uint32_t)g, (uint32_t)p.tq};
    rc = make_tmap(&mq, q, TMA_BF16, 3, dims, strides, box, TMA_SW_128); if (rc) return 2000 + rc;
  }
  for (int which = 0; which < 2; which++) {
    const uint64_t w = which ? Dv : D;
    uint64_t dims[4] = {w, (uint64_t)Hkv, (uint64_t)kBPage, (uint64_t)num_blocks};
    uint64_t strides[3] = {w * 2, (uint64_t)Hkv * w * 2, (uint64_t)kBPage * Hkv * w * 2};
    uint32_t box[4] = {64, 1, kBPage, 1};
    rc = make_tmap(which ? &mv : &mk, which ? v_cache : k_cache, TMA_BF16, 4, dims, strides, box, TMA_SW_128); if (rc) return 2100 + rc;
  }
  CUtensorMap mkp = mk, mvp = mv;
  for (int which = 0; which < 2 && pool > 0; which++) {
    const uint64_t w = which ? Dv : D;
    uint64_t dims[4] = {w, (uint64_t)Hkv, (uint64_t)pool_rows, (uint64_t)num_blocks};
    uint64_t strides[3] = {w * 2, (uint64_t)Hkv * w * 2, (uint64_t)pool_rows * Hkv * w * 2};
    uint32_t box[4] = {64, 1, 8, 1};
    rc = make_tmap(which ? &mvp : &mkp, which ? v_pool : k_pool, TMA_BF16, 4, dims, strides, box, TMA_SW_128); if (rc) return 2200 + rc;
  }
  const int variant = ext ? 4 : (softcap > 0.f ? 2 : 0) + p.rep;
  auto kern = variant == 4 ? gqa_biased_kernel<false, false, true> : variant == 3 ? gqa_biased_kernel<true, true, false> : variant == 2 ? gqa_biased_kernel<true, false, false>
              : variant == 1 ? gqa_biased_kernel<false, true, false> : gqa_biased_kernel<false, false, false>;
  static bool configured[5] = {false, false, false, false, false};
  if (!configured[variant]) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 232448);
    if (e != cudaSuccess) return (int)e;
    configured[variant] = true;
  }
  GbArgs a;
  a.block_tables = block_tables; a.bt_stride = bt_stride; a.cu_seqlens_q = cu_seqlens_q; a.context_lens = context_lens; a.num_seqs = num_seqs;
  a.T = T; a.H = H; a.Dv = Dv; a.g = g; a.tq = p.tq; a.splits = splits; a.nc = p.nc; a.nv = p.nv; a.rows8 = p.rows8; a.stages = p.stages; a.pbufs = p.pbufs;
  a.window = window; a.tmem_cols = p.nv <= 2 ? 256 : 512; a.scale = scale; a.softcap = softcap; a.slopes = slopes; a.gate = (const __nv_bfloat16*)gate;
  a.gate_ld = gate_ld; a.out_scale = out_scale; a.out = (__nv_bfloat16*)out; a.o_ld = o_ld; a.part = part; a.lse2 = lse2;
  a.pool = pool > 0 ? pool : 0; a.turn = turn; a.n_pos = n_pos; a.bar_off = p.bar_off; a.keep = window > 0 && keep > 0 ? keep : 0;
  a.mixing = nullptr; a.eps = 0.f; a.egate = nullptr; a.egate_ld = 0;
  cudaError_t e = launch_pdl(kern, dim3((unsigned)max_tiles, (unsigned)Hkv, (unsigned)splits), dim3(kGbThreads), (size_t)p.smem, st, mq, mk, mv, mkp, mvp, a);
  if (e != cudaSuccess || splits == 1) return (int)e;
  return (int)launch_pdl(gqa_biased_merge_kernel, dim3((unsigned)((long long)T * H)), dim3(128), 0, st, a);
}

// Pairs of (token, head) tokens per tile of the differential form (0: the shape is not covered); D: size of one map
extern "C" int ne_gqa_diff_plan(int H, int Hkv, int D, int Dv, int max_q) {
  GbPlan p;
  return Hkv >= 1 && H % Hkv == 0 && gb_plan(H / Hkv, D, Dv, max_q, false, false, &p, 2) ? p.tq : 0;
}

// q bf16 [T, H, 2, D] (row stride q_ld elements), k_cache bf16 [num_blocks, 64, Hkv, 2 D], v_cache bf16 [num_blocks, 64, Hkv, Dv]; mixing fp32 [1], gate bf16
// [T, H Dv] (row stride gate_ld), out bf16 [T, H Dv] (row stride o_ld).  window 0: all earlier keys; keep: the first keys stay visible behind the window.
// splits > 1 (at most 32): part fp32 [splits, T, H, 2, Dv], lse2 [splits, T, H, 2]; the merge kernel is launched too.
extern "C" int ne_gqa_diff(const void* q, long long q_ld, const void* k_cache, const void* v_cache, int num_blocks, const int* block_tables, int bt_stride,
                           const int* cu_seqlens_q, const int* context_lens, int num_seqs, int T, int H, int Hkv, int D, int Dv, int max_q, int max_tiles, int splits,
                           float scale, int window, int keep, const float* mixing, float out_scale, float eps, const void* gate, long long gate_ld, void* out,
                           long long o_ld, float* part, float* lse2, cudaStream_t st) {
  if (T <= 0) return 0;
  GbPlan p;
  if (Hkv < 1 || H % Hkv || splits < 1 || splits > 32 || (splits > 1 && (!part || !lse2)) || max_tiles < 1 || !mixing || !gate) return 1001;
  if (!gb_plan(H / Hkv, D, Dv, max_q, false, false, &p, 2)) return 1001;
  if (q_ld % 8 || o_ld % 4 || gate_ld % 4 || q_ld < (long long)H * 2 * D || ((uintptr_t)q & 15) || (((uintptr_t)out | (uintptr_t)gate) & 7)) return 1002;
  const int g = H / Hkv;
  CUtensorMap mq, mk, mv;
  int rc;
  {
    uint64_t dims[4] = {(uint64_t)D, 2, (uint64_t)H, (uint64_t)T}; uint64_t strides[3] = {(uint64_t)D * 2, (uint64_t)D * 4, (uint64_t)q_ld * 2};
    uint32_t box[4] = {64, 1, (uint32_t)g, (uint32_t)p.tq};
    rc = make_tmap(&mq, q, TMA_BF16, 4, dims, strides, box, TMA_SW_128); if (rc) return 2000 + rc;
  }
  for (int which = 0; which < 2; which++) {
    const uint64_t w = which ? Dv : D, heads = which ? Hkv : 2 * Hkv;
    uint64_t dims[4] = {w, heads, (uint64_t)kBPage, (uint64_t)num_blocks};
    uint64_t strides[3] = {w * 2, heads * w * 2, (uint64_t)kBPage * heads * w * 2};
    uint32_t box[4] = {64, 1, kBPage, 1};
    rc = make_tmap(which ? &mv : &mk, which ? v_cache : k_cache, TMA_BF16, 4, dims, strides, box, TMA_SW_128); if (rc) return 2100 + rc;
  }
  auto kern = gqa_biased_kernel<false, false, false, true>;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 232448);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  GbArgs a = {};
  a.block_tables = block_tables; a.bt_stride = bt_stride; a.cu_seqlens_q = cu_seqlens_q; a.context_lens = context_lens; a.num_seqs = num_seqs;
  a.T = T; a.H = H; a.Dv = Dv; a.g = g; a.tq = p.tq; a.splits = splits; a.nc = p.nc; a.nv = p.nv; a.rows8 = p.rows8; a.stages = p.stages; a.pbufs = p.pbufs;
  a.window = window; a.tmem_cols = p.nv <= 2 ? 256 : 512; a.scale = scale; a.out_scale = out_scale; a.out = (__nv_bfloat16*)out; a.o_ld = o_ld; a.part = part;
  a.lse2 = lse2; a.bar_off = p.bar_off; a.keep = window > 0 && keep > 0 ? keep : 0; a.mixing = mixing; a.eps = eps; a.egate = (const __nv_bfloat16*)gate;
  a.egate_ld = gate_ld;
  cudaError_t e = launch_pdl(kern, dim3((unsigned)max_tiles, (unsigned)Hkv, (unsigned)splits), dim3(kGbThreads), (size_t)p.smem, st, mq, mk, mv, mk, mv, a);
  if (e != cudaSuccess || splits == 1) return (int)e;
  return (int)launch_pdl(gqa_diff_merge_kernel, dim3((unsigned)(((long long)T * H + 3) / 4)), dim3(128), 0, st, a);
}
