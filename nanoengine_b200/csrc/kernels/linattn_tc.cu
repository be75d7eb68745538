// Chunked tensor-core form of the recurrence of linattn.cu for long portions:  S_t = a_t S_(t-1) + b_t k_t v_t^T,  o_t = S_t^T q_t (+ d v_t).
// bf16 q, k, v (the values that enter the products are bf16 anyway), everything else in 32-bit: fp32 accumulators, decays and step sizes in
// fp32, and each fp32 operand of a product (decayed scores, decayed values, the state) is split into a bf16 head and a bf16 remainder, two
// products that add up to about 2^-16 of relative accuracy.  The state itself never leaves fp32: it lives in TMEM as an accumulator.
//
// One CTA = one (sequence, head) x 64 columns of Dv, walking chunks of 128 tokens (Dk <= 128, tcgen05.mma kind::f16, M = 128):
//     G  = Q K^T                     [128 tokens x 128 tokens]
//     Yi = Q (S_hi + S_lo)           [128 x 64]     the state in front of the chunk
//     S  = e^(C_end) S + K^T (V'_hi + V'_lo)        V'_j = b_j e^(C_end - C_j) v_j      [Dk x 64]
//     P  = G_ij b_j e^(C_i - C_j), j <= i           -> P_hi, P_lo in shared memory
//     Y  = (P_hi + P_lo) V           [128 x 64]
//     o  = e^(C_i) Yi + Y + d v
// C: running sum of the log-decays, kept per block of 32 tokens so that no difference of large sums is taken: a factor between blocks is the
// product of two exponentials of at most one, only the diagonal blocks take an exponential per element.
// 512 threads: all of them load, convert and store; thread 0 issues the products.  All waits are bounded.
#include "ptx.cuh"

namespace ne {

constexpr int kCtThreads = 512;
constexpr int kKernelCt = 14;
constexpr int kCL = 128;                        // tokens per chunk
constexpr int kCTile = kCL * 128;               // 128 rows x 64 bf16 columns, 128-byte swizzled
constexpr float kMinLog2 = -100.f;              // a decay below 2^-100 counts as 2^-100

struct ChunkArgs {
  const __nv_bfloat16* q; const __nv_bfloat16* k; const __nv_bfloat16* v; long long q_ld, k_ld, v_ld;
  const float2* gates; const float* decay; const float* skip;
  float* state; const int* slots; const int* cu; const int* fresh;
  float* raw;
  int H, Hk, Dk, Dv, act, min_n, tiles;
};

__device__ __forceinline__ int swz(int row, int piece) { return row * 128 + ((piece ^ (row & 7)) << 4); }      // byte offset of a 16-byte piece
__device__ __forceinline__ uint32_t silu2(uint32_t u) {
  const float2 f = unpack_bf16x2(u);
  // one reciprocal for two; below -40 the result is zero in bf16 next to anything
  const float a = 1.f + __expf(fminf(-f.x, 40.f)), b = 1.f + __expf(fminf(-f.y, 40.f)), r = __fdividef(1.f, a * b);
  return pack_bf16x2(f.x * b * r, f.y * a * r);
}
// fp32 pair -> bf16 heads and bf16 remainders
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(a, b);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(a - h.x, b - h.y);
}

// NK: tiles of 64 columns of Dk.  smem: Q nk tiles | K nk tiles | V | V'_hi | V'_lo | P_hi 2 tiles | P_lo 2 tiles | S_hi | S_lo
template <int NK>
__global__ void __launch_bounds__(kCtThreads, 1) decay_chunk_kernel(const ChunkArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  __shared__ __align__(16) float s_lc[kCL], s_b[kCL], s_w[kCL], s_bt[4];
  __shared__ uint64_t s_bar[2];
  __shared__ uint32_t s_tmem;
  __shared__ int s_abort;
  const int seq = blockIdx.y, h = blockIdx.x / a.tiles, dv0 = (blockIdx.x % a.tiles) * 64, hk = h / (a.H / a.Hk);
  const int start = a.cu[seq], n = a.cu[seq + 1] - start;
  const int slot = a.slots[seq];
  if (n < a.min_n || n <= 0 || !NE_INDEX_OK(slot, BK_STATE_SLOTS, kKernelCt, __LINE__)) return;
  constexpr int nk = NK, kShift = NK == 2 ? 4 : 3;
  const int Dk = a.Dk, Dv = a.Dv, vcols = min(64, Dv - dv0);
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + nk * kCTile;
  uint8_t* sV = sK + nk * kCTile;
  uint8_t* sVh = sV + kCTile;
  uint8_t* sVl = sVh + kCTile;
  uint8_t* sPh = sVl + kCTile;
  uint8_t* sPl = sPh + 2 * kCTile;
  uint8_t* sSh = sPl + 2 * kCTile;
  uint8_t* sSl = sSh + kCTile;
  float* sY = reinterpret_cast<float*>(sPh);     // [128][68]: the output tile, once P has been multiplied
  constexpr int kYld = 68;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, wq = warp & 3, hf = warp >> 2;
  const int row = wq * 32 + lane;                // TMEM lane of this thread
  volatile int* abort_flag = &s_abort;
  const uint32_t bar_g = smem_u32(&s_bar[0]), bar_y = smem_u32(&s_bar[1]);
  if (tid == 0) { mbar_init(bar_g, 1); mbar_init(bar_y, 1); s_abort = 0; mbar_fence_init(); }
  if (warp == 0) { tmem_alloc(smem_u32(&s_tmem), 512); tmem_relinquish(); }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t t_g = s_tmem, t_yi = t_g + 128, t_y = t_yi + 64, t_s = t_y + 64;
  const uint32_t lane_addr = (uint32_t)(wq * 32) << 16;
  const bool s_row = wq * 32 < nk * 64;          // whole warps: rows of the state tile

  float* Sg = a.state + ((long long)slot * a.H + h) * Dv * Dk;
  {                                              // the carried state: lane = column of Dk, 16 columns of Dv per thread
    const bool have = a.fresh[seq] == 0 && row < Dk;
    uint32_t r[16];
#pragma unroll
    for (int c = 0; c < 16; c++) {
      const int d = hf * 16 + c;
      r[c] = (have && d < vcols) ? __float_as_uint(Sg[(long long)(dv0 + d) * Dk + row]) : 0u;
    }
    tmem_st_32x32b_x16(t_s + lane_addr + hf * 16, r);
    tc_wait_st();
  }
  const float skip = a.skip ? a.skip[h] : 0.f;
  const float fixed = a.gates ? 0.f : fmaxf(log2f(a.decay[h]), kMinLog2);
  const __nv_bfloat16* qg = a.q + (long long)hk * Dk;
  const __nv_bfloat16* kg = a.k + (long long)hk * Dk;
  const __nv_bfloat16* vg = a.v + (long long)h * Dv + dv0;

  constexpr uint32_t kIdG = make_idesc(FMT_BF16, FMT_BF16, 128, 128);
  constexpr uint32_t kIdY = make_idesc(FMT_BF16, FMT_BF16, 128, 64, 0, 1);       // B read MN-major: rows are tokens or columns of Dk
  constexpr uint32_t kIdS = make_idesc(FMT_BF16, FMT_BF16, 128, 64, 1, 1);
  // the next chunk's rows are fetched into registers while this one's products run
  uint4 rq[2 * NK], rk[2 * NK], rv[2];
  float2 rg = make_float2(0.f, 0.f);
  auto fetch = [&](int i0) {
    const int m = min(kCL, n - i0);
    const long long t0 = start + i0;
#pragma unroll
    for (int e = 0; e < 2 * NK; e++) {
      const int j = tid + e * kCtThreads, r = j >> kShift, c = (j & (8 * NK - 1)) * 8;
      const bool in = r < m && c < Dk;
      rq[e] = in ? *reinterpret_cast<const uint4*>(qg + (t0 + r) * a.q_ld + c) : make_uint4(0, 0, 0, 0);
      rk[e] = in ? *reinterpret_cast<const uint4*>(kg + (t0 + r) * a.k_ld + c) : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int e = 0; e < 2; e++) {
      const int j = tid + e * kCtThreads, r = j >> 3, c = (j & 7) * 8;
      rv[e] = r < m && c < vcols ? *reinterpret_cast<const uint4*>(vg + (t0 + r) * a.v_ld + c) : make_uint4(0, 0, 0, 0);
    }
    if (hf == 0 && a.gates) rg = row < m ? a.gates[(t0 + row) * a.H + h] : make_float2(0.f, 0.f);
  };
  auto put = [&](uint8_t* dst, int r, int p, uint4 u) {
    if (a.act) { u.x = silu2(u.x); u.y = silu2(u.y); u.z = silu2(u.z); u.w = silu2(u.w); }
    *reinterpret_cast<uint4*>(dst + (p >> 3) * kCTile + swz(r, p & 7)) = u;
  };
  fetch(0);
  bool ok = true;
  uint32_t phase = 0;
  for (int i0 = 0; i0 < n && ok; i0 += kCL, phase ^= 1) {
    const int m = min(kCL, n - i0);
    const long long t0 = start + i0;
    // ---- decays: inclusive sums within blocks of 32 tokens
    if (hf == 0) {
      float la = 0.f, b = 0.f;
      if (row < m) {
        if (a.gates) { la = fmaxf(rg.x * 1.4426950408889634f, kMinLog2); b = rg.y; }
        else { la = fixed; b = 1.f; }
      }
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) { const float x = __shfl_up_sync(0xffffffffu, la, o); if (lane >= o) la += x; }
      const float tot = __shfl_sync(0xffffffffu, la, 31);
      s_lc[row] = la; s_b[row] = b; s_w[row] = b * exp2f(tot - la);
      if (lane == 31) s_bt[wq] = tot;
    }
    // ---- q, k, v tiles
#pragma unroll
    for (int e = 0; e < 2 * NK; e++) {
      const int j = tid + e * kCtThreads, r = j >> kShift, p = j & (8 * NK - 1);
      put(sQ, r, p, rq[e]);
      put(sK, r, p, rk[e]);
    }
#pragma unroll
    for (int e = 0; e < 2; e++) { const int j = tid + e * kCtThreads; put(sV, j >> 3, j & 7, rv[e]); }
    __syncthreads();
    const float bt0 = s_bt[0], bt1 = s_bt[1], bt2 = s_bt[2], bt3 = s_bt[3];
    const float after[4] = {bt1 + bt2 + bt3, bt2 + bt3, bt3, 0.f};
    // ---- decayed values, head and remainder
    for (int i = tid; i < kCL * 8; i += kCtThreads) {
      const int r = i >> 3, o = swz(r, i & 7);
      const uint4 u = *reinterpret_cast<const uint4*>(sV + o);
      const int blk = r >> 5;
      const float w = s_w[r] * exp2f(blk == 0 ? after[0] : blk == 1 ? after[1] : blk == 2 ? after[2] : 0.f);
      uint4 hi, lo;
      float2 f = unpack_bf16x2(u.x); split2(f.x * w, f.y * w, hi.x, lo.x);
      f = unpack_bf16x2(u.y); split2(f.x * w, f.y * w, hi.y, lo.y);
      f = unpack_bf16x2(u.z); split2(f.x * w, f.y * w, hi.z, lo.z);
      f = unpack_bf16x2(u.w); split2(f.x * w, f.y * w, hi.w, lo.w);
      *reinterpret_cast<uint4*>(sVh + o) = hi;
      *reinterpret_cast<uint4*>(sVl + o) = lo;
    }
    // ---- the state: head and remainder as it is, the accumulator scaled by the whole chunk's decay
    if (s_row) {
      const float dec = exp2f(bt0 + after[0]);
      uint32_t r[16];
      tmem_ld_32x32b_x16(t_s + lane_addr + hf * 16, r);
      tc_wait_ld();
      uint32_t hi[8], lo[8];
#pragma unroll
      for (int c = 0; c < 8; c++) split2(__uint_as_float(r[2 * c]), __uint_as_float(r[2 * c + 1]), hi[c], lo[c]);
#pragma unroll
      for (int p = 0; p < 2; p++) {
        const int o = swz(row, hf * 2 + p);
        *reinterpret_cast<uint4*>(sSh + o) = make_uint4(hi[4 * p], hi[4 * p + 1], hi[4 * p + 2], hi[4 * p + 3]);
        *reinterpret_cast<uint4*>(sSl + o) = make_uint4(lo[4 * p], lo[4 * p + 1], lo[4 * p + 2], lo[4 * p + 3]);
      }
#pragma unroll
      for (int c = 0; c < 16; c++) r[c] = __float_as_uint(__uint_as_float(r[c]) * dec);
      tmem_st_32x32b_x16(t_s + lane_addr + hf * 16, r);
      tc_wait_st();
    }
    fence_proxy_async_smem();
    tc_fence_before();
    __syncthreads();
    if (tid == 0) {
      tc_fence_after();
      const uint32_t aq = smem_u32(sQ), ak = smem_u32(sK), vh = smem_u32(sVh), vl = smem_u32(sVl), sh = smem_u32(sSh), sl = smem_u32(sSl);
      for (int c = 0; c < nk; c++)
#pragma unroll
        for (int ks = 0; ks < 4; ks++)
          umma_f16(t_g, make_smem_desc(aq + c * kCTile + ks * 32, 16, 1024, SW_128B), make_smem_desc(ak + c * kCTile + ks * 32, 16, 1024, SW_128B), kIdG, (c | ks) != 0);
      tc_commit(bar_g);
      for (int x = 0; x < 2; x++)
        for (int ks = 0; ks < nk * 4; ks++)
          umma_f16(t_yi, make_smem_desc(aq + (ks >> 2) * kCTile + (ks & 3) * 32, 16, 1024, SW_128B), make_smem_desc((x ? sl : sh) + ks * 16 * 128, kCTile, 1024, SW_128B), kIdY,
                   (x | ks) != 0);
      for (int x = 0; x < 2; x++)
#pragma unroll
        for (int ks = 0; ks < 8; ks++)
          umma_f16(t_s, make_smem_desc(ak + ks * 16 * 128, kCTile, 1024, SW_128B), make_smem_desc((x ? vl : vh) + ks * 16 * 128, kCTile, 1024, SW_128B), kIdS, 1);
    }
    ok = mbar_wait(bar_g, phase, abort_flag, kKernelCt, 100);
    tc_fence_after();
    // ---- decayed scores: this thread's row, block hf of 32 columns
    if (ok) {
      const float li = s_lc[row];
      {
        const int jb = hf;                       // whole warps take the same branch: a warp's rows are one block
        uint32_t hi[16], lo[16];
        if (jb > wq) {
#pragma unroll
          for (int c = 0; c < 16; c++) hi[c] = lo[c] = 0u;
        } else {
          uint32_t r[32];
          tmem_ld_32x32b_x32(t_g + lane_addr + jb * 32, r);
          tc_wait_ld();
          if (jb < wq) {
            float between = 0.f;
            if (jb < 1 && wq > 1) between += bt1;
            if (jb < 2 && wq > 2) between += bt2;
            const float f = exp2f(li + between);
#pragma unroll
            for (int c = 0; c < 16; c += 2) {
              const float4 w = *reinterpret_cast<const float4*>(s_w + jb * 32 + 2 * c);
              split2(__uint_as_float(r[2 * c]) * (f * w.x), __uint_as_float(r[2 * c + 1]) * (f * w.y), hi[c], lo[c]);
              split2(__uint_as_float(r[2 * c + 2]) * (f * w.z), __uint_as_float(r[2 * c + 3]) * (f * w.w), hi[c + 1], lo[c + 1]);
            }
          } else {
#pragma unroll
            for (int c = 0; c < 16; c += 2) {
              const float4 b4 = *reinterpret_cast<const float4*>(s_b + jb * 32 + 2 * c), l4 = *reinterpret_cast<const float4*>(s_lc + jb * 32 + 2 * c);
              const float bb[4] = {b4.x, b4.y, b4.z, b4.w}, ll[4] = {l4.x, l4.y, l4.z, l4.w};
              float p4[4];
#pragma unroll
              for (int e = 0; e < 4; e++) p4[e] = 2 * c + e <= lane ? __uint_as_float(r[2 * c + e]) * bb[e] * exp2f(li - ll[e]) : 0.f;
              split2(p4[0], p4[1], hi[c], lo[c]);
              split2(p4[2], p4[3], hi[c + 1], lo[c + 1]);
            }
          }
        }
#pragma unroll
        for (int p = 0; p < 4; p++) {
          const int o = (hf >> 1) * kCTile + swz(row, (hf & 1) * 4 + p);
          *reinterpret_cast<uint4*>(sPh + o) = make_uint4(hi[4 * p], hi[4 * p + 1], hi[4 * p + 2], hi[4 * p + 3]);
          *reinterpret_cast<uint4*>(sPl + o) = make_uint4(lo[4 * p], lo[4 * p + 1], lo[4 * p + 2], lo[4 * p + 3]);
        }
      }
    }
    fence_proxy_async_smem();
    tc_fence_before();
    if (!__syncthreads_and(ok)) { ok = false; break; }
    if (tid == 0) {
      tc_fence_after();
      const uint32_t av = smem_u32(sV), ph = smem_u32(sPh), pl = smem_u32(sPl);
      for (int x = 0; x < 2; x++)
#pragma unroll
        for (int ks = 0; ks < 8; ks++)
          umma_f16(t_y, make_smem_desc((x ? pl : ph) + (ks >> 2) * kCTile + (ks & 3) * 32, 16, 1024, SW_128B), make_smem_desc(av + ks * 16 * 128, kCTile, 1024, SW_128B), kIdY,
                   (x | ks) != 0);
      tc_commit(bar_y);                          // covers every product issued so far
    }
    if (i0 + kCL < n) fetch(i0 + kCL);
    ok = mbar_wait(bar_y, phase, abort_flag, kKernelCt, 200);
    tc_fence_after();
    // ---- outputs: 16 columns of this thread's row
    if (ok) {
      const float before = (wq > 0 ? bt0 : 0.f) + (wq > 1 ? bt1 : 0.f) + (wq > 2 ? bt2 : 0.f);
      const float f = exp2f(s_lc[row] + before);
      {
        uint32_t yi[16], y[16];
        tmem_ld_32x32b_x16(t_yi + lane_addr + hf * 16, yi);
        tmem_ld_32x32b_x16(t_y + lane_addr + hf * 16, y);
        tc_wait_ld();
#pragma unroll
        for (int p = 0; p < 2; p++) {
          const uint4 u = *reinterpret_cast<const uint4*>(sV + swz(row, hf * 2 + p));
          const float2 v0 = unpack_bf16x2(u.x), v1 = unpack_bf16x2(u.y), v2 = unpack_bf16x2(u.z), v3 = unpack_bf16x2(u.w);
          const float vv[8] = {v0.x, v0.y, v1.x, v1.y, v2.x, v2.y, v3.x, v3.y};
          float o[8];
#pragma unroll
          for (int e = 0; e < 8; e++) o[e] = fmaf(skip, vv[e], fmaf(f, __uint_as_float(yi[p * 8 + e]), __uint_as_float(y[p * 8 + e])));
          float* dst = sY + row * kYld + hf * 16 + p * 8;
          *reinterpret_cast<float4*>(dst) = make_float4(o[0], o[1], o[2], o[3]);
          *reinterpret_cast<float4*>(dst + 4) = make_float4(o[4], o[5], o[6], o[7]);
        }
      }
    }
    tc_fence_before();
    if (!__syncthreads_and(ok)) { ok = false; break; }
    tc_fence_after();
    for (int i = tid; i < m * 16; i += kCtThreads) {
      const int r = i >> 4, c = (i & 15) * 4;
      if (c < vcols)
        *reinterpret_cast<float4*>(a.raw + ((t0 + r) * a.H + h) * Dv + dv0 + c) = *reinterpret_cast<const float4*>(sY + r * kYld + c);
    }
  }
  if (ok) {
    if (s_row) {
      uint32_t r[16];
      tmem_ld_32x32b_x16(t_s + lane_addr + hf * 16, r);
      tc_wait_ld();
#pragma unroll
      for (int c = 0; c < 16; c++) {
        const int d = hf * 16 + c;
        if (row < Dk && d < vcols) Sg[(long long)(dv0 + d) * Dk + row] = __uint_as_float(r[c]);
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) { tc_fence_after(); tmem_dealloc(t_g, 512); }
}

static size_t chunk_smem(int Dk) {
  const int nk = (Dk + 63) / 64;
  return (size_t)(2 * nk + 3 + 4 + 2) * kCTile + 1024;
}

}  // namespace ne

using namespace ne;

extern "C" int ne_decay_chunk_covers(int Dk, int Dv) { return Dk >= 8 && Dk <= 128 && Dk % 8 == 0 && Dv >= 8 && Dv % 8 == 0 ? 1 : 0; }

// As ne_decay_scan, for the sequences of at least min_n tokens in this call (the others are left alone): bf16, rows of 16-byte aligned pieces.
extern "C" int ne_decay_chunk(const void* q, long long q_ld, const void* k, long long k_ld, const void* v, long long v_ld, const float* gates, const float* decay,
                              const float* skip, float* state, const int* slots, const int* cu, const int* fresh, float* raw, int B, int H, int Hk, int Dk, int Dv,
                              int act, int min_n, cudaStream_t st) {
  if (B <= 0) return 0;
  if (Hk < 1 || H % Hk || !ne_decay_chunk_covers(Dk, Dv) || B > 65535 || (!gates && !decay)) return 1001;
  if (q_ld % 8 || k_ld % 8 || v_ld % 8 || (((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)raw) & 15)) return 1002;
  ChunkArgs a;
  a.q = (const __nv_bfloat16*)q; a.k = (const __nv_bfloat16*)k; a.v = (const __nv_bfloat16*)v; a.q_ld = q_ld; a.k_ld = k_ld; a.v_ld = v_ld;
  a.gates = reinterpret_cast<const float2*>(gates); a.decay = decay; a.skip = skip; a.state = state; a.slots = slots; a.cu = cu; a.fresh = fresh; a.raw = raw;
  a.H = H; a.Hk = Hk; a.Dk = Dk; a.Dv = Dv; a.act = act; a.min_n = min_n; a.tiles = (Dv + 63) / 64;
  const size_t smem = chunk_smem(Dk);
  auto kern = Dk > 64 ? decay_chunk_kernel<2> : decay_chunk_kernel<1>;
  static bool configured[2] = {false, false};
  if (!configured[Dk > 64]) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured[Dk > 64] = true;
  }
  // an ordinary launch: a few long CTAs spread over the machine
  kern<<<dim3((unsigned)(H * a.tiles), (unsigned)B), kCtThreads, smem, st>>>(a);
  return (int)cudaGetLastError();
}
