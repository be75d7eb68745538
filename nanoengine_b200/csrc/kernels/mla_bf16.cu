// Paged latent attention (absorbed MLA) on tcgen05 tensor cores over bf16 pages: queries [T, H, D], one shared key row [D = R + rope]
// per cached token whose first R values are the value row, 64-token pages, any R <= 512 and D <= 576 in multiples of 8.  Decode and
// prompt portions alike; every row has its own causal limit.
//
// One CTA = one tile of (token, head) rows of ONE sequence x one part of the output width x one slice of its key pages.  A tile holds
// `tq` consecutive tokens x `g` heads (all heads, or a group of them), at most 128 rows (64 when the row is wider than 320, so that
// two page tiles fit beside the queries); r = token_in_tile * g + head_in_group.
//
// Per 64-key page:  S = Q K^T   (nc chunks x 4 tcgen05.mma kind::f16, M=128 N=64 K=16; both K-major, 128B swizzle)
//                   online softmax by 128 threads reading S from TMEM; P -> bf16 -> shared memory
//                   O += P V    (4 x tcgen05.mma, N = 64 nv; V = the first chunks of the same page tile, read MN-major)
// A row width that is not a multiple of 64 ends in a chunk whose missing columns TMA fills with zeros.  TMEM: S twice 64 columns,
// O up to 256, so an output wider than 256 is split over two CTAs which both compute S.  M = 128 rows are always multiplied; rows past
// the tile's own read whatever shared memory follows and feed accumulator rows nobody reads.
// Warp 0: TMA producer, warp 1: MMA issuer, warps 2-5: softmax / rescale / epilogue.  All waits are bounded.
// With more than one key slice the CTA writes a normalised partial result and its log2-sum-exp; ne_attn_merge folds them.
#include "ptx.cuh"
#include "tma_host.h"

namespace ne {

constexpr int kLatThreads = 192;
constexpr int kKernelLat = 12;
constexpr int kLPage = 64;                     // keys per page
constexpr int kLChunk = kLPage * 128;          // one 64-column chunk of a page tile: 64 rows x 128 B

struct LatArgs {
  const int* block_tables; int bt_stride;
  const int* cu_seqlens_q; const int* context_lens; int num_seqs;
  int T, H, R, g, tq, splits;                  // g heads x tq tokens per tile
  int nc, nfull, nv, parts;                    // chunks of a row (of which nfull come as one box), value chunks per output part, output parts
  int rows8, stages, pbufs;                    // tile rows rounded up to 8, page tiles in flight, P buffers
  int q_boxed;                                 // 1: the query tile is one box, 0: one per chunk
  uint32_t tmem_cols;
  float scale_log2;
  __nv_bfloat16* out;                          // [T, H, R] (splits == 1)
  float* part; float* lse2;                    // [splits, T, H, R], [splits, T, H] (splits > 1)
};

__global__ void __launch_bounds__(kLatThreads, 1)
mla_bf16_kernel(const __grid_constant__ CUtensorMap q_map, const __grid_constant__ CUtensorMap k_map, const __grid_constant__ CUtensorMap kt_map,
                const LatArgs a) {
  pdl_wait();                     // dependent launch: nothing above this line touches global memory
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int q_chunk = a.rows8 * 128, p_bytes = a.rows8 * 128, k_stage = a.nc * kLChunk;
  uint8_t* sQ = smem;                                    // nc chunks of rows8 x 128 B
  uint8_t* sP = sQ + a.nc * q_chunk;
  uint8_t* sK = sP + a.pbufs * p_bytes;                  // MMA reads of rows past rows8 end inside the page tiles
  uint64_t* bars = reinterpret_cast<uint64_t*>(sK + a.stages * k_stage);
  // q_full | kv_full[4] | kv_empty[4] | s_full[2] | s_empty[2] | p_full[2] | p_empty[2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 17);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* s_tile = reinterpret_cast<int*>(tmem_slot + 2);
  const uint32_t b_qfull = smem_u32(bars), b_kvfull = smem_u32(bars + 1), b_kvempty = smem_u32(bars + 5);
  const uint32_t b_sfull = smem_u32(bars + 9), b_sempty = smem_u32(bars + 11), b_pfull = smem_u32(bars + 13), b_pempty = smem_u32(bars + 15);

  const int warp = threadIdx.x >> 5;
  const int opart = blockIdx.y % a.parts, h0 = (blockIdx.y / a.parts) * a.g, split = blockIdx.z;
  const int vc0 = opart * a.nv, nv = min(a.nv, (a.R + 63) / 64 - vc0);       // value chunks of this CTA

  if (warp == 0) {          // which sequence and which of its token tiles: 32 sequences per round, prefix sum of their tile counts
    const int lane = (int)lane_id();
    int rem = blockIdx.x, seq = -1, tok0 = 0;
    for (int s0 = 0; s0 < a.num_seqs && seq < 0; s0 += 32) {
      const int s = s0 + lane;
      int q0 = 0, nt = 0;
      if (s < a.num_seqs) { q0 = a.cu_seqlens_q[s]; nt = (a.cu_seqlens_q[s + 1] - q0 + a.tq - 1) / a.tq; }
      int incl = nt;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) { const int v = __shfl_up_sync(0xffffffffu, incl, o); if (lane >= o) incl += v; }
      const unsigned hit = __ballot_sync(0xffffffffu, rem < incl);
      if (hit) {
        const int l = __ffs(hit) - 1;
        const int before = __shfl_sync(0xffffffffu, incl - nt, l);
        seq = s0 + l;
        tok0 = __shfl_sync(0xffffffffu, q0, l) + (rem - before) * a.tq;
      } else {
        rem -= __shfl_sync(0xffffffffu, incl, 31);
      }
    }
    if (lane == 0) { s_tile[0] = seq; s_tile[1] = tok0; }
  }
  if (threadIdx.x == 0) {
    mbar_init(b_qfull, 1);
    for (int i = 0; i < 4; i++) { mbar_init(b_kvfull + 8 * i, 1); mbar_init(b_kvempty + 8 * i, 1); }
    for (int i = 0; i < 2; i++) {
      mbar_init(b_sfull + 8 * i, 1); mbar_init(b_sempty + 8 * i, 4); mbar_init(b_pfull + 8 * i, 4); mbar_init(b_pempty + 8 * i, 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == 1) { tmem_alloc(smem_u32(tmem_slot), a.tmem_cols); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  // Only now may the next kernel's CTAs come in: every CTA of this grid holds its TMEM, so none can be left waiting for columns
  // that a CTA waiting for this grid holds.
  pdl_trigger();
  const uint32_t tmem_base = *tmem_slot, tmem_o = tmem_base + 128;
  const int seq = s_tile[0], tok0 = s_tile[1];

  int n_tiles = 0, pg_begin = 0, n_tok = 0, base_limit = -1;
  const int* bt = a.block_tables;
  if (seq >= 0) {
    const int q_beg = a.cu_seqlens_q[seq], q_len = a.cu_seqlens_q[seq + 1] - q_beg;
    n_tok = min(a.tq, q_beg + q_len - tok0);
    base_limit = a.context_lens[seq] - q_len + (tok0 - q_beg);              // last key visible to the tile's first token
    const int max_limit = base_limit + n_tok - 1;
    const int total_pages = max_limit >= 0 ? max_limit / kLPage + 1 : 0;
    const int per_split = (total_pages + a.splits - 1) / a.splits;
    pg_begin = split * per_split;
    n_tiles = max(0, min(total_pages, pg_begin + per_split) - pg_begin);
    bt = a.block_tables + (long long)seq * a.bt_stride;
  }

  if (warp == 0) {
    if (n_tiles > 0 && elect_one()) {
      mbar_expect_tx(b_qfull, a.nc * a.g * a.tq * 128);
      if (a.q_boxed) tma_load_4d(smem_u32(sQ), &q_map, b_qfull, 0, h0, tok0, 0);
      else for (int c = 0; c < a.nc; c++) tma_load_3d(smem_u32(sQ + c * q_chunk), &q_map, b_qfull, c * 64, h0, tok0);
      for (int i = 0; i < n_tiles; i++) {
        const int s = i % a.stages;
        if (!mbar_wait(b_kvempty + 8 * s, ((i / a.stages) & 1) ^ 1, abort_flag, kKernelLat, 100 + s)) break;
        uint8_t* dst = sK + s * k_stage;
        int block = bt[pg_begin + i];
        if (!NE_INDEX_OK(block, BK_CACHE_PAGES, kKernelLat, __LINE__)) block = 0;      // a bad page id reads page 0
        mbar_expect_tx(b_kvfull + 8 * s, k_stage);
        tma_load_4d(smem_u32(dst), &k_map, b_kvfull + 8 * s, 0, 0, block, 0);
        if (a.nfull < a.nc) tma_load_3d(smem_u32(dst + a.nfull * kLChunk), &kt_map, b_kvfull + 8 * s, a.nfull * 64, 0, block);
      }
    }
  } else if (warp == 1) {
    if (n_tiles > 0 && elect_one()) {
      constexpr uint32_t kIdescQK = make_idesc(FMT_BF16, FMT_BF16, 128, kLPage);
      const uint32_t idesc_pv = make_idesc(FMT_BF16, FMT_BF16, 128, (uint32_t)nv * 64, 0, 1);      // B (= V) is MN-major
      bool ok = mbar_wait(b_qfull, 0, abort_flag, kKernelLat, 200);
      const uint32_t q_addr = smem_u32(sQ), p_addr = smem_u32(sP), k_addr = smem_u32(sK);
      auto pv = [&](int j) -> bool {
        const int pb = j % a.pbufs;
        if (!mbar_wait(b_pfull + 8 * pb, (j / a.pbufs) & 1, abort_flag, kKernelLat, 230)) return false;
        tc_fence_after();
        const int s = j % a.stages;
        const uint32_t vt = k_addr + s * k_stage + vc0 * kLChunk;
#pragma unroll
        for (int ks = 0; ks < 4; ks++) {                     // 16 keys per MMA
          const uint64_t adesc = make_smem_desc(p_addr + pb * p_bytes + ks * 32, 16, 1024, SW_128B);
          const uint64_t bdesc = make_smem_desc(vt + ks * 16 * 128, kLChunk, 1024, SW_128B);
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
        if (!pre_se && !mbar_wait(b_sempty + 8 * sb, ((i >> 1) & 1) ^ 1, abort_flag, kKernelLat, 210 + sb)) { ok = false; break; }
        if (!pre_kv && !mbar_wait(b_kvfull + 8 * s, (i / a.stages) & 1, abort_flag, kKernelLat, 220 + s)) { ok = false; break; }
        mbar_test2(b_sempty + 8 * ((i + 1) & 1), (((i + 1) >> 1) & 1) ^ 1, b_kvfull + 8 * ((i + 1) % a.stages), ((i + 1) / a.stages) & 1, pre_se, pre_kv);
        tc_fence_after();
        const uint32_t kt = k_addr + s * k_stage, d = tmem_base + sb * kLPage;
        for (int c = 0; c < a.nc; c++) {
#pragma unroll
          for (int ks = 0; ks < 4; ks++) {
            const uint64_t adesc = make_smem_desc(q_addr + c * q_chunk + ks * 32, 16, 1024, SW_128B);
            const uint64_t bdesc = make_smem_desc(kt + c * kLChunk + ks * 32, 16, 1024, SW_128B);
            umma_f16(d, adesc, bdesc, kIdescQK, (c | ks) != 0);
          }
        }
        tc_commit(b_sfull + 8 * sb);
        if (i > 0 && !pv(i - 1)) { ok = false; break; }
      }
      if (ok) pv(n_tiles - 1);
    }
  } else {
    const int wq = warp & 3;
    const int row = wq * 32 + (int)lane_id();
    const uint32_t lane_addr = (uint32_t)(wq * 32) << 16;
    const int tl = row / a.g, head = h0 + row % a.g;
    const bool row_ok = row < a.g * a.tq && tl < n_tok && head < a.H;
    const int limit = row_ok ? base_limit + tl : -1;          // this row's last visible key
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true, s_ready = false;
    for (int i = 0; ok && i < n_tiles; i++) {
      const int sb = i & 1, pb = i % a.pbufs;
      if (!s_ready && !mbar_wait(b_sfull + 8 * sb, (i >> 1) & 1, abort_flag, kKernelLat, 300 + sb)) { ok = false; break; }
      tc_fence_after();
      uint32_t r0[32], r1[32];
      tmem_ld_32x32b_x32(tmem_base + lane_addr + sb * kLPage, r0);
      tmem_ld_32x32b_x32(tmem_base + lane_addr + sb * kLPage + 32, r1);
      tc_wait_ld();
      tc_fence_before();
      __syncwarp();
      if (lane_id() == 0) mbar_arrive(b_sempty + 8 * sb);
      const int key0 = (pg_begin + i) * kLPage;
      const bool p_free = i < a.pbufs || mbar_test(b_pempty + 8 * pb, ((i - a.pbufs) / a.pbufs) & 1);     // needed only after the math
      if (key0 + kLPage - 1 > limit) {
#pragma unroll
        for (int j = 0; j < 32; j++) {
          if (key0 + j > limit) r0[j] = 0xff800000u;
          if (key0 + 32 + j > limit) r1[j] = 0xff800000u;
        }
      }
      float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int j = 0; j < 32; j += 2) {
        mx[0] = fmaxf(mx[0], __uint_as_float(r0[j])); mx[1] = fmaxf(mx[1], __uint_as_float(r0[j + 1]));
        mx[2] = fmaxf(mx[2], __uint_as_float(r1[j])); mx[3] = fmaxf(mx[3], __uint_as_float(r1[j + 1]));
      }
      const float m_tile = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * a.scale_log2;
      // lazy rescaling: the reference maximum only moves when the page's maximum exceeds it by more than 2^8
      const bool first_valid = (m_run == -INFINITY);
      const float m_new = (first_valid || m_tile > m_run + 8.f) ? fmaxf(m_run, m_tile) : m_run;
      const float alpha = (m_new == -INFINITY || first_valid) ? 1.f : exp2f(m_run - m_new);
      const float neg_m = (m_new == -INFINITY) ? 0.f : -m_new;
      float psum = 0.f;
      uint32_t pk[32];
#pragma unroll
      for (int j = 0; j < 16; j++) {
        const float p0 = exp2f(fmaf(__uint_as_float(r0[2 * j]), a.scale_log2, neg_m)), p1 = exp2f(fmaf(__uint_as_float(r0[2 * j + 1]), a.scale_log2, neg_m));
        const float p2 = exp2f(fmaf(__uint_as_float(r1[2 * j]), a.scale_log2, neg_m)), p3 = exp2f(fmaf(__uint_as_float(r1[2 * j + 1]), a.scale_log2, neg_m));
        pk[j] = pack_bf16x2(p0, p1);
        pk[16 + j] = pack_bf16x2(p2, p3);
        // sum what the MMA will see (bf16-rounded probabilities), so numerator and denominator stay consistent
        const float2 q0 = unpack_bf16x2(pk[j]), q1 = unpack_bf16x2(pk[16 + j]);
        psum += (q0.x + q0.y) + (q1.x + q1.y);
      }
      l_run = l_run * alpha + psum;
      m_run = m_new;
      if (i > 0 && __any_sync(0xffffffffu, alpha < 1.f)) {
        if (!mbar_wait(b_pempty + 8 * ((i - 1) % a.pbufs), ((i - 1) / a.pbufs) & 1, abort_flag, kKernelLat, 310)) { ok = false; break; }
        tc_fence_after();
#pragma unroll 1
        for (int cblk = 0; cblk < nv * 4; cblk++) {
          uint32_t o[16];
          tmem_ld_32x32b_x16(tmem_o + lane_addr + cblk * 16, o);
          tc_wait_ld();
#pragma unroll
          for (int j = 0; j < 16; j++) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
          tmem_st_32x32b_x16(tmem_o + lane_addr + cblk * 16, o);
        }
        tc_wait_st();
      }
      if (!p_free && !mbar_wait(b_pempty + 8 * pb, ((i - a.pbufs) / a.pbufs) & 1, abort_flag, kKernelLat, 311)) { ok = false; break; }
      s_ready = mbar_test(b_sfull + 8 * ((i + 1) & 1), ((i + 1) >> 1) & 1);
      if (row < a.rows8) {       // P row (64 bf16 = 8 chunks of 16 bytes) into the 128B-swizzled K-major layout the MMA reads
        uint8_t* prow = sP + pb * p_bytes + row * 128;
        const int sw = row & 7;
#pragma unroll
        for (int cch = 0; cch < 8; cch++)
          *reinterpret_cast<uint4*>(prow + ((cch ^ sw) << 4)) = make_uint4(pk[4 * cch], pk[4 * cch + 1], pk[4 * cch + 2], pk[4 * cch + 3]);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      __syncwarp();
      if (lane_id() == 0) mbar_arrive(b_pfull + 8 * pb);
    }
    if (ok && n_tiles > 0) ok = mbar_wait(b_pempty + 8 * ((n_tiles - 1) % a.pbufs), ((n_tiles - 1) / a.pbufs) & 1, abort_flag, kKernelLat, 320);
    const long long orow = row_ok ? ((long long)(tok0 + tl) * a.H + head) : 0;
    const bool have = ok && n_tiles > 0;
    if (have) tc_fence_after();
    const float inv = (have && l_run > 0.f) ? 1.f / l_run : 0.f;
#pragma unroll 1
    for (int cblk = 0; cblk < nv * 2; cblk++) {
      uint32_t o[32];
      if (have) {
        tmem_ld_32x32b_x32(tmem_o + lane_addr + cblk * 32, o);
        tc_wait_ld();
      }
      const int col0 = vc0 * 64 + cblk * 32;
      if (!row_ok) continue;
#pragma unroll
      for (int v = 0; v < 4; v++) {                            // R is a multiple of 8: whole groups of 8 columns
        if (col0 + v * 8 >= a.R) continue;
        float f[8];
#pragma unroll
        for (int j = 0; j < 8; j++) f[j] = have ? __uint_as_float(o[v * 8 + j]) * inv : 0.f;
        if (a.splits == 1) {
          *reinterpret_cast<uint4*>(a.out + orow * a.R + col0 + v * 8) =
              make_uint4(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]), pack_bf16x2(f[4], f[5]), pack_bf16x2(f[6], f[7]));
        } else {
          float* dst = a.part + ((long long)split * a.T * a.H + orow) * a.R + col0 + v * 8;
          *reinterpret_cast<float4*>(dst) = make_float4(f[0], f[1], f[2], f[3]);
          *reinterpret_cast<float4*>(dst + 4) = make_float4(f[4], f[5], f[6], f[7]);
        }
      }
    }
    if (a.splits > 1 && opart == 0 && row_ok)
      a.lse2[(long long)split * a.T * a.H + orow] = (have && l_run > 0.f) ? m_run + log2f(l_run) : -INFINITY;
  }

  tc_fence_before();
  __syncthreads();
  if (*abort_flag && threadIdx.x == 0) for (int i = 0; i < 2000; i++) __nanosleep(1000);      // copies in flight land before the CTA goes
  __syncthreads();
  if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, a.tmem_cols); }
}

struct LatPlan { int nc, nfull, nv, parts, g, tq, rows8, stages, pbufs, smem; };

// Tile geometry for H heads, row D = R + rope, sequences of at most max_q new tokens; false when the kernel does not cover it.
static bool lat_plan(int H, int R, int D, int max_q, LatPlan* p) {
  if (R < 8 || R % 8 || D % 8 || D < 64 || D > 576 || R > 512 || R > D || H < 1 || max_q < 1) return false;
  p->nc = (D + 63) / 64; p->nfull = D / 64;
  const int nvt = (R + 63) / 64;
  p->parts = nvt > 4 ? 2 : 1;
  p->nv = (nvt + p->parts - 1) / p->parts;
  const int cap = p->nc <= 5 ? 128 : 64;
  const int groups = (H + cap - 1) / cap;
  p->g = (H + groups - 1) / groups;
  p->tq = cap / p->g < max_q ? cap / p->g : max_q;
  p->rows8 = (p->g * p->tq + 7) / 8 * 8;
  const int limit = 232448 - 1024 - 256, k = p->nc * kLChunk, q = p->nc * p->rows8 * 128;
  p->pbufs = q + 2 * p->rows8 * 128 + 2 * k <= limit ? 2 : 1;
  p->stages = (limit - q - p->pbufs * p->rows8 * 128) / k;
  if (p->stages > 4) p->stages = 4;
  if (p->stages < 2) return false;
  p->smem = q + p->pbufs * p->rows8 * 128 + p->stages * k + 1024 + 256;
  // an MMA reads 128 rows from each chunk of Q and from each P buffer: those reads must end inside the allocation
  const int last_q = (p->nc - 1) * p->rows8 * 128 + 16384, last_p = q + (p->pbufs - 1) * p->rows8 * 128 + 16384;
  return (last_q > last_p ? last_q : last_p) <= q + p->pbufs * p->rows8 * 128 + p->stages * k;
}

}  // namespace ne

using namespace ne;

// Output parts x head groups of one tile (0: the shape is not covered) and tokens per tile, for the caller's choice of key slices.
extern "C" int ne_mla_bf16_plan(int H, int R, int D, int max_q, int* tq) {
  LatPlan p;
  if (!lat_plan(H, R, D, max_q, &p)) return 0;
  *tq = p.tq;
  return p.parts * ((H + p.g - 1) / p.g);
}

// q bf16 [T, H, D] contiguous, cache bf16 [num_blocks, 64, D]; max_tiles >= sum over sequences of ceil(q_len / tq).  out bf16 [T, H, R].
extern "C" int ne_mla_bf16(const void* q, const void* cache, int num_blocks, const int* block_tables, int bt_stride, const int* cu_seqlens_q,
                           const int* context_lens, int num_seqs, int T, int H, int R, int D, int max_q, int max_tiles, int splits, float scale, void* out,
                           float* part, float* lse2, cudaStream_t st) {
  if (T <= 0) return 0;
  LatPlan p;
  if (splits < 1 || (splits > 1 && (!part || !lse2)) || max_tiles < 1 || !lat_plan(H, R, D, max_q, &p)) return 1001;
  CUtensorMap mq, mk, mt;
  const bool q_boxed = D % 64 == 0 && (p.g * p.tq) % 8 == 0;
  int rc;
  if (q_boxed) {
    uint64_t dims[4] = {64, (uint64_t)H, (uint64_t)T, (uint64_t)p.nc}; uint64_t strides[3] = {(uint64_t)D * 2, (uint64_t)H * D * 2, 128};
    uint32_t box[4] = {64, (uint32_t)p.g, (uint32_t)p.tq, (uint32_t)p.nc};
    rc = make_tmap(&mq, q, TMA_BF16, 4, dims, strides, box, TMA_SW_128);
  } else {
    uint64_t dims[3] = {(uint64_t)D, (uint64_t)H, (uint64_t)T}; uint64_t strides[2] = {(uint64_t)D * 2, (uint64_t)H * D * 2};
    uint32_t box[3] = {64, (uint32_t)p.g, (uint32_t)p.tq};
    rc = make_tmap(&mq, q, TMA_BF16, 3, dims, strides, box, TMA_SW_128);
  }
  if (rc) return 2000 + rc;
  {
    uint64_t dims[4] = {64, (uint64_t)kLPage, (uint64_t)num_blocks, (uint64_t)p.nfull};
    uint64_t strides[3] = {(uint64_t)D * 2, (uint64_t)kLPage * D * 2, 128};
    uint32_t box[4] = {64, kLPage, 1, (uint32_t)p.nfull};
    rc = make_tmap(&mk, cache, TMA_BF16, 4, dims, strides, box, TMA_SW_128); if (rc) return 2100 + rc;
  }
  {
    uint64_t dims[3] = {(uint64_t)D, (uint64_t)kLPage, (uint64_t)num_blocks}; uint64_t strides[2] = {(uint64_t)D * 2, (uint64_t)kLPage * D * 2};
    uint32_t box[3] = {64, kLPage, 1};
    rc = make_tmap(&mt, cache, TMA_BF16, 3, dims, strides, box, TMA_SW_128); if (rc) return 2200 + rc;
  }
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(mla_bf16_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 232448);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  LatArgs a;
  a.block_tables = block_tables; a.bt_stride = bt_stride; a.cu_seqlens_q = cu_seqlens_q; a.context_lens = context_lens; a.num_seqs = num_seqs;
  a.T = T; a.H = H; a.R = R; a.g = p.g; a.tq = p.tq; a.splits = splits; a.nc = p.nc; a.nfull = p.nfull; a.nv = p.nv; a.parts = p.parts;
  a.rows8 = p.rows8; a.stages = p.stages; a.pbufs = p.pbufs; a.q_boxed = q_boxed ? 1 : 0; a.tmem_cols = p.nv <= 2 ? 256 : 512;
  a.scale_log2 = scale * 1.4426950408889634f; a.out = (__nv_bfloat16*)out; a.part = part; a.lse2 = lse2;
  const int groups = (H + p.g - 1) / p.g;
  return (int)launch_pdl(mla_bf16_kernel, dim3((unsigned)max_tiles, (unsigned)(groups * p.parts), (unsigned)splits), dim3(kLatThreads), (size_t)p.smem, st, mq, mk,
                         mt, a);
}
