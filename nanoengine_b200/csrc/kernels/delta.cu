// Gated delta-rule mixer with everything between its projections in 32-bit: any head sizes (Dk <= 512), bf16 or fp32 activations,
// any mix of prompt portions and single tokens in one call.
//   1. delta_prepare: short causal convolution + silu over [q | k | v] with the carried window, unit q and k (q scaled by Dk^-0.5), q.k,
//      decay exp(-exp(A_log) softplus(a + dt_bias)) and write strength sigmoid(b) - one warp per (token, head).
//   2. delta_scan: the recurrence.  Rows of a head's [Dv, Dk] state are independent of each other, so a CTA owns some rows of one
//      (sequence, head) in registers: 8 lanes share a row (each CPL of its columns), a warp holds 4 R rows.  Per token two dot
//      products with the old state (k and q) are reduced over the 8 lanes; then u = beta (v - g S.k), S <- g S + u k^T,
//      o = g S.q + u (q.k).  Inputs of the next tokens are copied to shared memory (cp.async) while a chunk is computed.  The carried
//      convolution window is moved on here too: the kernel before has read it.
//      Single-token steps keep a whole head in one CTA and apply the output norm and gate before the row leaves (kFuse).
//   3. delta_out_norm: o / rms(o) * w * silu(z) for the calls whose heads are spread over several CTAs.
// The same arithmetic in the same order runs whatever the portions are, so a sequence cut differently gives the same state.
#include "ptx.cuh"

namespace ne {

__device__ __forceinline__ float ldd(const float* p) { return *p; }
__device__ __forceinline__ float ldd(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void std_(float* p, float v) { *p = v; }
__device__ __forceinline__ void std_(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float silu_exact(float x) { return x / (1.f + expf(-x)); }

struct DeltaArgs {
  const void* proj; long long proj_ld;       // [T, q | k | v | z]
  const float* ab; long long ab_ld;          // [T, a (Hv) | b (Hv)]
  const void* conv_w;                        // [C, K]
  const float* A_log; const float* dt_bias;
  const void* norm_w; float eps;
  void* window;                              // [S, K - 1, C]
  float* state;                              // [S, Hv, Dv, Dk]
  const int* slots; const int* cu; const int* fresh;
  float* qn; float* kn; float* vn; float* gates;   // [T, Hk, Dk] x 2, [T, Hv, Dv], [T, 2 Hv + Hk]: decay, beta, q.k
  void* out; float* raw;                     // [T, Hv, Dv] in the activation dtype / fp32 before the norm
  int T, B, Hk, Hv, Dk, Dv, K, C;
};

__device__ __forceinline__ int seq_of(const int* cu, int B, int t) {
  int lo = 0, hi = B - 1;                     // last sequence whose start is <= t
  while (lo < hi) { const int mid = (lo + hi + 1) >> 1; if (cu[mid] <= t) lo = mid; else hi = mid - 1; }
  return lo;
}

__device__ __forceinline__ float2 ldd2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ldd2(const __nv_bfloat16* p) { return unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p)); }
__device__ __forceinline__ void ldd4(const float* p, float* o) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
}
__device__ __forceinline__ void ldd4(const __nv_bfloat16* p, float* o) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 x = unpack_bf16x2(u.x), y = unpack_bf16x2(u.y);
  o[0] = x.x; o[1] = x.y; o[2] = y.x; o[3] = y.y;
}

// One warp per (token, unit): units [0, Hk) are key heads (q and k), [Hk, Hk + Hv) value heads.  KT: taps (0 = any number).
// V = 2 (four taps, even head sizes and strides): a lane takes two neighbouring channels at a time.
template <typename T, int KT, int V>
__global__ void __launch_bounds__(256) delta_prepare_kernel(const DeltaArgs a) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const int units = a.Hk + a.Hv, lane = threadIdx.x & 31, K = KT ? KT : a.K, C = a.C;
  const long long wid = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (wid >= (long long)a.T * units) return;
  const int t = (int)(wid / units), u = (int)(wid - (long long)t * units);
  const int seq = seq_of(a.cu, a.B, t), p = t - a.cu[seq];
  const int slot = a.slots[seq];
  const bool carried = a.fresh[seq] == 0 && NE_INDEX_OK(slot, BK_STATE_SLOTS, 43, __LINE__);
  const T* x = reinterpret_cast<const T*>(a.proj) + (long long)t * a.proj_ld;
  const T* win = reinterpret_cast<const T*>(a.window) + (long long)(carried ? slot : 0) * (K - 1) * C;
  const T* w = reinterpret_cast<const T*>(a.conv_w);
  auto conv = [&](int c) {
    float acc = 0.f;
#pragma unroll
    for (int j = 0; j < (KT ? KT : 1); j++) {
      for (int jj = KT ? j : 0; jj < (KT ? j + 1 : K); jj++) {
        const int back = K - 1 - jj;           // how many tokens before this one
        float v = 0.f;
        if (back <= p) v = ldd(x - back * a.proj_ld + c);
        else if (carried) v = ldd(win + (long long)(p + jj) * C + c);
        acc += v * ldd(w + (long long)c * K + jj);
      }
    }
    return silu_exact(acc);
  };
  auto conv2 = [&](int c) {                  // channels c and c + 1, four taps
    float w0[4], w1[4];
    ldd4(w + (long long)c * 4, w0); ldd4(w + (long long)c * 4 + 4, w1);
    float a0 = 0.f, a1 = 0.f;
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int back = 3 - j;
      float2 v = make_float2(0.f, 0.f);
      if (back <= p) v = ldd2(x - back * a.proj_ld + c);
      else if (carried) v = ldd2(win + (long long)(p + j) * C + c);
      a0 += v.x * w0[j]; a1 += v.y * w1[j];
    }
    return make_float2(silu_exact(a0), silu_exact(a1));
  };
  if (u < a.Hk) {
    const int Dk = a.Dk, q0 = u * Dk, k0 = a.Hk * Dk + u * Dk;
    float* qo = a.qn + ((long long)t * a.Hk + u) * Dk;
    float* ko = a.kn + ((long long)t * a.Hk + u) * Dk;
    float qq = 0.f, kk = 0.f, qk = 0.f;
    if constexpr (V == 2) {
      for (int c = lane * 2; c < Dk; c += 64) {
        const float2 qv = conv2(q0 + c), kv = conv2(k0 + c);
        *reinterpret_cast<float2*>(qo + c) = qv; *reinterpret_cast<float2*>(ko + c) = kv;
        qq += qv.x * qv.x + qv.y * qv.y; kk += kv.x * kv.x + kv.y * kv.y; qk += qv.x * kv.x + qv.y * kv.y;
      }
    } else {
      for (int c = lane; c < Dk; c += 32) {
        const float qv = conv(q0 + c), kv = conv(k0 + c);
        qo[c] = qv; ko[c] = kv;
        qq += qv * qv; kk += kv * kv; qk += qv * kv;
      }
    }
    qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
    const float qr = rsqrtf(qq + 1e-6f) * rsqrtf((float)Dk), kr = rsqrtf(kk + 1e-6f);
    if constexpr (V == 2) {                                                  // a lane rereads its own stores
      for (int c = lane * 2; c < Dk; c += 64) {
        float2 *q2 = reinterpret_cast<float2*>(qo + c), *k2 = reinterpret_cast<float2*>(ko + c);
        const float2 qv = *q2, kv = *k2;
        *q2 = make_float2(qv.x * qr, qv.y * qr); *k2 = make_float2(kv.x * kr, kv.y * kr);
      }
    } else {
      for (int c = lane; c < Dk; c += 32) { qo[c] *= qr; ko[c] *= kr; }
    }
    if (lane == 0) a.gates[(long long)t * (2 * a.Hv + a.Hk) + 2 * a.Hv + u] = qk * qr * kr;
  } else {
    const int h = u - a.Hk, Dv = a.Dv, v0 = 2 * a.Hk * a.Dk + h * Dv;
    float* vo = a.vn + ((long long)t * a.Hv + h) * Dv;
    if constexpr (V == 2) { for (int c = lane * 2; c < Dv; c += 64) *reinterpret_cast<float2*>(vo + c) = conv2(v0 + c); }
    else { for (int c = lane; c < Dv; c += 32) vo[c] = conv(v0 + c); }
    if (lane == 0) {
      const float av = a.ab[(long long)t * a.ab_ld + h] + a.dt_bias[h], bv = a.ab[(long long)t * a.ab_ld + a.Hv + h];
      const float sp = av > 20.f ? av : log1pf(expf(av));
      float* g = a.gates + (long long)t * (2 * a.Hv + a.Hk);
      g[h] = expf(-expf(a.A_log[h]) * sp);
      g[a.Hv + h] = 1.f / (1.f + expf(-bv));
    }
  }
}

__device__ __forceinline__ void cp_async4(uint32_t dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(dst), "l"(src) : "memory");
}

constexpr int kScanChunk = 16;     // tokens staged at a time (two chunks in flight)

// grid = (Hv * splits, B), NW = blockDim.x / 32 warps of 4 R rows each; `splits` CTAs share a head's Dv rows.
template <int CPL, int R, bool kFuse, typename T>
__global__ void __launch_bounds__(kFuse ? 256 : 128, kFuse ? (CPL * R >= 40 ? 2 : CPL * R >= 32 ? 3 : 4) : (CPL * R >= 40 ? 4 : CPL * R >= 24 ? 6 : 8))
delta_scan_kernel(const DeltaArgs a) {
  constexpr int DKP = CPL * 8;                 // columns a row is padded to
  extern __shared__ float sm[];
  const int nw = blockDim.x >> 5, rows = nw * 4 * R;
  const int splits = gridDim.x / a.Hv, h = blockIdx.x / splits, row0 = (blockIdx.x % splits) * rows, hk = h / (a.Hv / a.Hk);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, cg = lane & 7, rg = lane >> 3;
  const int Dk = a.Dk, Dv = a.Dv, seq = blockIdx.y;
  // per buffer (n = kScanChunk tokens): k [n][DKP] | q [n][DKP] | v [n][rows] | gates [n][4]
  const int buf_floats = kScanChunk * (2 * DKP + rows + 4);
  // columns past Dk stay zero: the copies below never touch them
  if (Dk < DKP)
    for (int i = threadIdx.x; i < 2 * kScanChunk * 2 * (DKP - Dk); i += blockDim.x) {
      const int c = i % (DKP - Dk), r = i / (DKP - Dk);            // r: (buffer, k or q, token)
      sm[(r / (2 * kScanChunk)) * buf_floats + (r % (2 * kScanChunk)) * DKP + Dk + c] = 0.f;
    }
  // The step's tables and the state were written before delta_prepare began (it triggers behind its own wait and writes none of
  // them), so they are fetched while it still runs; only what it produces waits for it below.
  const int start = a.cu[seq], n = a.cu[seq + 1] - start;
  const int slot = a.slots[seq];
  if (n <= 0 || !NE_INDEX_OK(slot, BK_STATE_SLOTS, 44, __LINE__)) { pdl_wait(); return; }
  const bool is_fresh = a.fresh[seq] != 0;

  const bool vec = (Dk & 3) == 0;
  auto stage = [&](int buf, int i0) {
    const int m = min(kScanChunk, n - i0);
    float* base = sm + buf * buf_floats;
    const long long t0 = start + i0;
    if (vec) {
      const int per = Dk >> 2;
      for (int i = threadIdx.x; i < m * 2 * per; i += blockDim.x) {
        const int c = i % per, r = i / per, tok = r >> 1, which = r & 1;
        const float* src = (which ? a.qn : a.kn) + ((t0 + tok) * a.Hk + hk) * Dk + c * 4;
        cp_async16(smem_u32(base + which * kScanChunk * DKP + tok * DKP + c * 4), src, 16);
      }
    } else {
      for (int i = threadIdx.x; i < m * 2 * Dk; i += blockDim.x) {
        const int c = i % Dk, r = i / Dk, tok = r >> 1, which = r & 1;
        cp_async4(smem_u32(base + which * kScanChunk * DKP + tok * DKP + c), (which ? a.qn : a.kn) + ((t0 + tok) * a.Hk + hk) * Dk + c);
      }
    }
    float* sv = base + 2 * kScanChunk * DKP;
    for (int i = threadIdx.x; i < m * rows; i += blockDim.x) {
      const int r = i % rows, tok = i / rows;
      if (row0 + r < Dv) cp_async4(smem_u32(sv + tok * rows + r), a.vn + ((t0 + tok) * a.Hv + h) * Dv + row0 + r);
    }
    float* sg = sv + kScanChunk * rows;
    for (int i = threadIdx.x; i < m * 3; i += blockDim.x) {
      const int which = i % 3, tok = i / 3;
      cp_async4(smem_u32(sg + tok * 4 + which), a.gates + (t0 + tok) * (2 * a.Hv + a.Hk) + (which == 0 ? h : which == 1 ? a.Hv + h : 2 * a.Hv + hk));
    }
    cp_async_commit();
  };

  // state rows of this thread: row0 + warp * 4R + r * 4 + rg; columns j * 32 + cg * 4 + {0..3}
  float* Sg = a.state + (((long long)slot * a.Hv + h) * Dv) * Dk;
  float S[R][CPL];
#pragma unroll
  for (int r = 0; r < R; r++) {
    const int row = row0 + warp * 4 * R + r * 4 + rg;
#pragma unroll
    for (int j = 0; j < CPL / 4; j++) {
      const int c = j * 32 + cg * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!is_fresh && row < Dv) {
        const float* src = Sg + (long long)row * Dk + c;
        if (vec) { if (c < Dk) v = *reinterpret_cast<const float4*>(src); }
        else { if (c < Dk) v.x = src[0]; if (c + 1 < Dk) v.y = src[1]; if (c + 2 < Dk) v.z = src[2]; if (c + 3 < Dk) v.w = src[3]; }
      }
      S[r][4 * j] = v.x; S[r][4 * j + 1] = v.y; S[r][4 * j + 2] = v.z; S[r][4 * j + 3] = v.w;
    }
  }
  pdl_wait();
  if (kFuse) pdl_trigger();       // a long scan triggers at its end
  stage(0, 0);
  // the convolution window after this call: the last K - 1 inputs (older entries move up where the call is shorter)
  {
    const int K = a.K, C = a.C;
    const T* x = reinterpret_cast<const T*>(a.proj) + (long long)start * a.proj_ld;
    T* win = reinterpret_cast<T*>(a.window) + (long long)slot * (K - 1) * C;
    for (int c = blockIdx.x * blockDim.x + threadIdx.x; c < C; c += gridDim.x * blockDim.x)
      for (int j = 0; j < K - 1; j++) {                      // ascending: an entry is read before it is overwritten
        const int src = n - (K - 1) + j;
        T v;
        if (src >= 0) v = x[(long long)src * a.proj_ld + c];
        else if (is_fresh) std_(&v, 0.f);
        else v = win[(long long)(src + K - 1) * C + c];
        win[(long long)j * C + c] = v;
      }
  }

  for (int i0 = 0, buf = 0; i0 < n; i0 += kScanChunk, buf ^= 1) {
    const int m = min(kScanChunk, n - i0);
    if (i0 + kScanChunk < n) { stage(buf ^ 1, i0 + kScanChunk); cp_async_wait<1>(); } else cp_async_wait<0>();
    __syncthreads();
    const float* sk = sm + buf * buf_floats;
    const float* sq = sk + kScanChunk * DKP;
    const float* sv = sq + kScanChunk * DKP;
    const float* sg = sv + kScanChunk * rows;
    for (int i = 0; i < m; i++) {
      const float4 gt = *reinterpret_cast<const float4*>(sg + i * 4);      // decay, beta, q.k
      float pk[R], pq[R];
#pragma unroll
      for (int r = 0; r < R; r++) pk[r] = pq[r] = 0.f;
#pragma unroll
      for (int j = 0; j < CPL / 4; j++) {
        const float4 k4 = *reinterpret_cast<const float4*>(sk + i * DKP + j * 32 + cg * 4), q4 = *reinterpret_cast<const float4*>(sq + i * DKP + j * 32 + cg * 4);
#pragma unroll
        for (int r = 0; r < R; r++) {
          pk[r] = fmaf(S[r][4 * j], k4.x, pk[r]); pq[r] = fmaf(S[r][4 * j], q4.x, pq[r]);
          pk[r] = fmaf(S[r][4 * j + 1], k4.y, pk[r]); pq[r] = fmaf(S[r][4 * j + 1], q4.y, pq[r]);
          pk[r] = fmaf(S[r][4 * j + 2], k4.z, pk[r]); pq[r] = fmaf(S[r][4 * j + 2], q4.z, pq[r]);
          pk[r] = fmaf(S[r][4 * j + 3], k4.w, pk[r]); pq[r] = fmaf(S[r][4 * j + 3], q4.w, pq[r]);
        }
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1)
#pragma unroll
        for (int r = 0; r < R; r++) {
          pk[r] += __shfl_xor_sync(0xffffffffu, pk[r], o);
          pq[r] += __shfl_xor_sync(0xffffffffu, pq[r], o);
        }
      float o_sel = 0.f, u[R];
#pragma unroll
      for (int r = 0; r < R; r++) {
        u[r] = gt.y * (sv[i * rows + warp * 4 * R + r * 4 + rg] - gt.x * pk[r]);
        const float o = fmaf(u[r], gt.z, gt.x * pq[r]);
        if (cg == r) o_sel = o;
      }
#pragma unroll
      for (int j = 0; j < CPL / 4; j++) {
        const float4 k4 = *reinterpret_cast<const float4*>(sk + i * DKP + j * 32 + cg * 4);
#pragma unroll
        for (int r = 0; r < R; r++) {
          S[r][4 * j] = fmaf(u[r], k4.x, gt.x * S[r][4 * j]);
          S[r][4 * j + 1] = fmaf(u[r], k4.y, gt.x * S[r][4 * j + 1]);
          S[r][4 * j + 2] = fmaf(u[r], k4.z, gt.x * S[r][4 * j + 2]);
          S[r][4 * j + 3] = fmaf(u[r], k4.w, gt.x * S[r][4 * j + 3]);
        }
      }
      const int lrow = warp * 4 * R + cg * 4 + rg;             // the row whose output this lane holds (cg < R)
      const long long t = start + i0 + i;
      if constexpr (!kFuse) {
        if (cg < R && row0 + lrow < Dv) a.raw[(t * a.Hv + h) * Dv + row0 + lrow] = o_sel;
      } else {
        // the CTA holds the whole head: norm over Dv, weight, gate, one rounding
        __shared__ float s_red[8];
        const bool mine = cg < R && lrow < Dv;
        const float ss = warp_sum(mine ? o_sel * o_sel : 0.f);
        if (lane == 0) s_red[warp] = ss;
        __syncthreads();
        float tot = 0.f;
        for (int w = 0; w < nw; w++) tot += s_red[w];
        if (mine) {
          const float z = ldd(reinterpret_cast<const T*>(a.proj) + t * a.proj_ld + a.C + h * Dv + lrow);
          std_(reinterpret_cast<T*>(a.out) + (t * a.Hv + h) * Dv + lrow,
               o_sel * rsqrtf(tot / (float)Dv + a.eps) * ldd(reinterpret_cast<const T*>(a.norm_w) + lrow) * silu_exact(z));
        }
        __syncthreads();
      }
    }
    __syncthreads();          // everyone is done with this buffer before the next-but-one chunk is copied into it
  }
  if (!kFuse) pdl_trigger();
#pragma unroll
  for (int r = 0; r < R; r++) {
    const int row = row0 + warp * 4 * R + r * 4 + rg;
    if (row >= Dv) continue;
#pragma unroll
    for (int j = 0; j < CPL / 4; j++) {
      const int c = j * 32 + cg * 4;
      float* dst = Sg + (long long)row * Dk + c;
      if (vec) { if (c < Dk) *reinterpret_cast<float4*>(dst) = make_float4(S[r][4 * j], S[r][4 * j + 1], S[r][4 * j + 2], S[r][4 * j + 3]); }
      else { for (int e = 0; e < 4; e++) if (c + e < Dk) dst[e] = S[r][4 * j + e]; }
    }
  }
}

// one warp per (token, head); V = 4: head size, strides and addresses allow groups of four
template <typename T, int V>
__global__ void __launch_bounds__(256) delta_out_norm_kernel(const DeltaArgs a) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const long long row = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (row >= (long long)a.T * a.Hv) return;
  const int lane = threadIdx.x & 31, h = (int)(row % a.Hv), Dv = a.Dv;
  const long long t = row / a.Hv;
  const float* o = a.raw + row * Dv;
  const T* z = reinterpret_cast<const T*>(a.proj) + t * a.proj_ld + a.C + h * Dv;
  float ss = 0.f;
  if (V == 4 && Dv <= 128) {                 // one group of four per lane, held in registers
    const bool on = lane * 4 < Dv;
    const float4 f = on ? *reinterpret_cast<const float4*>(o + lane * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float r = rsqrtf(warp_sum(f.x * f.x + f.y * f.y + f.z * f.z + f.w * f.w) / (float)Dv + a.eps);
    if (on) {
      float zz[4], ww[4];
      ldd4(z + lane * 4, zz); ldd4(reinterpret_cast<const T*>(a.norm_w) + lane * 4, ww);
      T y[4];
      std_(y, f.x * r * ww[0] * silu_exact(zz[0])); std_(y + 1, f.y * r * ww[1] * silu_exact(zz[1]));
      std_(y + 2, f.z * r * ww[2] * silu_exact(zz[2])); std_(y + 3, f.w * r * ww[3] * silu_exact(zz[3]));
      T* dst = reinterpret_cast<T*>(a.out) + row * Dv + lane * 4;
      if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(dst) = *reinterpret_cast<uint2*>(y);
      else *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<uint4*>(y);
    }
    return;
  }
  for (int d = lane; d < Dv; d += 32) { const float f = o[d]; ss += f * f; }
  const float r = rsqrtf(warp_sum(ss) / (float)Dv + a.eps);
  for (int d = lane; d < Dv; d += 32)
    std_(reinterpret_cast<T*>(a.out) + row * Dv + d, o[d] * r * ldd(reinterpret_cast<const T*>(a.norm_w) + d) * silu_exact(ldd(z + d)));
}

template <int CPL, int R, bool kFuse, typename T>
static int scan(const DeltaArgs& a, int warps, cudaStream_t st) {
  const int rows = warps * 4 * R, splits = (a.Dv + rows - 1) / rows;
  const size_t smem = sizeof(float) * 2 * kScanChunk * (2 * CPL * 8 + rows + 4);
  auto k = delta_scan_kernel<CPL, R, kFuse, T>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  const dim3 grid((unsigned)(a.Hv * splits), (unsigned)a.B), block((unsigned)(warps * 32));
  if (kFuse) return (int)launch_pdl(k, grid, block, smem, st, a);
  // A prompt's scan is a few long CTAs.  A dependent launch would place them while delta_prepare drains, several on the first SMs that
  // have room, and leave the others empty for the whole scan (2.5 times as long for one 8192-token prompt); an ordinary launch
  // spreads them over the machine.
  k<<<grid, block, smem, st>>>(a);
  return (int)cudaGetLastError();
}

template <typename T>
static int delta_t(const DeltaArgs& a, int max_q, cudaStream_t st) {
  const long long warps = (long long)a.T * (a.Hk + a.Hv);
  const dim3 pgrid((unsigned)((warps + 7) / 8));
  const bool pairs = a.K == 4 && a.Dk % 2 == 0 && a.Dv % 2 == 0 && a.proj_ld % 2 == 0 && ((uintptr_t)a.proj | (uintptr_t)a.window | (uintptr_t)a.conv_w) % 16 == 0;
  auto prep = pairs ? delta_prepare_kernel<T, 4, 2> : a.K == 4 ? delta_prepare_kernel<T, 4, 1> : delta_prepare_kernel<T, 0, 1>;
  cudaError_t e = launch_pdl(prep, pgrid, dim3(256), 0, st, a);
  if (e != cudaSuccess) return (int)e;
  int rc;
  // whole heads per CTA (norm and gate in the same kernel) for single-token steps whose state fits the registers of 8 warps
  const int whole4 = (a.Dv + 15) / 16;
  if (max_q <= 2 && a.Dk <= 128 && whole4 <= 8) {
    if (a.Dk <= 32) rc = scan<4, 4, true, T>(a, whole4, st);
    else if (a.Dk <= 64) rc = scan<8, 4, true, T>(a, whole4, st);
    else if (a.Dk <= 96) rc = scan<12, 4, true, T>(a, whole4, st);
    else rc = scan<16, 4, true, T>(a, whole4, st);
    return rc;
  }
  // rows spread over the machine: two rows per thread while that leaves warp schedulers idle, four otherwise
  const bool wide = (long long)a.Hv * a.Dv * a.B >= 148ll * 4 * 16 * 2;
#define NE_SCAN(CPL_) (wide ? scan<CPL_, 4, false, T>(a, 4, st) : scan<CPL_, 2, false, T>(a, 4, st))
  if (a.Dk <= 32) rc = NE_SCAN(4);
  else if (a.Dk <= 64) rc = NE_SCAN(8);
  else if (a.Dk <= 96) rc = NE_SCAN(12);
  else if (a.Dk <= 128) rc = NE_SCAN(16);
  else if (a.Dk <= 192) rc = scan<24, 2, false, T>(a, 4, st);
  else if (a.Dk <= 256) rc = scan<32, 2, false, T>(a, 4, st);
  else rc = scan<64, 1, false, T>(a, 4, st);
#undef NE_SCAN
  if (rc) return rc;
  const long long orows = (long long)a.T * a.Hv;
  const bool fours = a.Dv % 4 == 0 && a.C % 4 == 0 && a.proj_ld % 4 == 0 && ((uintptr_t)a.proj | (uintptr_t)a.norm_w | (uintptr_t)a.out) % 16 == 0;
  return (int)launch_pdl(fours ? delta_out_norm_kernel<T, 4> : delta_out_norm_kernel<T, 1>, dim3((unsigned)((orows + 7) / 8)), dim3(256), 0, st, a);
}

}  // namespace ne

using namespace ne;

// scratch: fp32, ne_delta_scratch_floats(...) elements.  Returns 0 or an error code; *launches receives the kernels launched.
extern "C" long long ne_delta_scratch_floats(int T, int Hk, int Hv, int Dk, int Dv) {
  const long long al = 4;      // keep every part 16-byte aligned
  auto up = [&](long long n) { return (n + al - 1) / al * al; };
  return 2 * up((long long)T * Hk * Dk) + 2 * up((long long)T * Hv * Dv) + up((long long)T * (2 * Hv + Hk));
}

extern "C" int ne_gated_delta(const void* proj, long long proj_ld, const float* ab, long long ab_ld, const void* conv_w, const float* A_log,
                              const float* dt_bias, const void* norm_w, float eps, void* window, float* state, const int* slots, const int* cu,
                              const int* fresh, float* scratch, void* out, int T, int B, int Hk, int Hv, int Dk, int Dv, int K, int max_q, int fp32,
                              int* launches, cudaStream_t st) {
  if (T <= 0 || B <= 0) return 0;
  if (Hk < 1 || Hv % Hk || Dk < 1 || Dk > 512 || Dv < 1 || K < 1 || B > 65535) return 1001;
  DeltaArgs a;
  a.proj = proj; a.proj_ld = proj_ld; a.ab = ab; a.ab_ld = ab_ld; a.conv_w = conv_w; a.A_log = A_log; a.dt_bias = dt_bias; a.norm_w = norm_w;
  a.eps = eps; a.window = window; a.state = state; a.slots = slots; a.cu = cu; a.fresh = fresh; a.out = out;
  a.T = T; a.B = B; a.Hk = Hk; a.Hv = Hv; a.Dk = Dk; a.Dv = Dv; a.K = K; a.C = 2 * Hk * Dk + Hv * Dv;
  auto up = [](long long n) { return (n + 3) / 4 * 4; };
  a.qn = scratch; a.kn = a.qn + up((long long)T * Hk * Dk); a.vn = a.kn + up((long long)T * Hk * Dk);
  a.raw = a.vn + up((long long)T * Hv * Dv); a.gates = a.raw + up((long long)T * Hv * Dv);
  *launches = (max_q <= 2 && Dk <= 128 && (Dv + 15) / 16 <= 8) ? 2 : 3;
  return fp32 ? delta_t<float>(a, max_q, st) : delta_t<__nv_bfloat16>(a, max_q, st);
}
