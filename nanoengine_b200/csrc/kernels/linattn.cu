// Linear attention with a scalar decay per head, everything past the projections and short convolutions in 32-bit:
//     S_t = a_t S_(t-1) + b_t k_t v_t^T       o_t = S_t^T q_t (+ d v_t)          (S: Dk x Dv, stored [Dv][Dk])
// in two uses.  Mamba-2 (state-space duality): k, q, v are B, C, x behind a short causal convolution, a = exp(-exp(A_log) dt), b = dt.
// Decayed attention (Lightning): k, q, v = silu of their projections, a a constant per head, b = 1.
//   1. ssm_prepare (Mamba-2): convolution + bias + silu over [x | B | C] with the carried window, dt = softplus(raw + bias) and the
//      log-decay -exp(A_log) dt; moves the window on.  A thread walks a run of tokens of one channel.
//   2. decay_scan: the recurrence token by token, any sizes, any mix of prompt portions and single tokens.  Rows of S are independent: a CTA
//      owns some rows of one (sequence, head) in registers, 8 lanes share a row (each CPL of its columns).  Long portions of bf16 models take
//      the chunked tensor-core form instead (linattn_tc.cu).
//   3. gated_norm: rows of heads, RMS-normed in equal parts, with the gate before (silu) or behind (sigmoid) the norm.
// Whatever the portions are, the scan does the same arithmetic in the same order.
#include "ptx.cuh"
#include "seq_tile.cuh"

namespace ne {

__device__ __forceinline__ float lda(const float* p) { return *p; }
__device__ __forceinline__ float lda(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void sta(float* p, float v) { *p = v; }
__device__ __forceinline__ void sta(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void lda4(const float* p, float* o) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
}
__device__ __forceinline__ void lda4(const __nv_bfloat16* p, float* o) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 x = unpack_bf16x2(u.x), y = unpack_bf16x2(u.y);
  o[0] = x.x; o[1] = x.y; o[2] = y.x; o[3] = y.y;
}
__device__ __forceinline__ void sta4(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void sta4(__nv_bfloat16* p, const float* v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3])); }
template <int V, typename T> __device__ __forceinline__ void ldv(const T* p, float* o) { if constexpr (V == 4) lda4(p, o); else o[0] = lda(p); }
template <int V, typename T> __device__ __forceinline__ void stv(T* p, const float* v) { if constexpr (V == 4) sta4(p, v); else sta(p, v[0]); }
// silu and sigmoid in the accuracy of the values they meet: exact functions for fp32, hardware exponentials (2^-21) where the result is rounded
// to bf16
__device__ __forceinline__ float sigm(float x, const float*) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float sigm(float x, const __nv_bfloat16*) { return __fdividef(1.f, 1.f + __expf(-x)); }
template <typename T> __device__ __forceinline__ float silu_t(float x) { return x * sigm(x, (const T*)nullptr); }
__device__ __forceinline__ float round_as(float x, const float*) { return x; }
__device__ __forceinline__ float round_as(float x, const __nv_bfloat16*) { return __bfloat162float(__float2bfloat16(x)); }

// ---- Mamba-2: convolution, step sizes, log-decays ---------------------------------------------------------------------------
constexpr int kRun = 16;              // tokens a thread walks
constexpr int kMaxTaps = 16;          // <= kRun: only a sequence's first run reads the carried window

struct SsmArgs {
  const void* xbc; long long ld;                   // [T, C] raw projections of x | B | C (row stride ld)
  const float* dt_raw; long long dt_ld;            // [T, H]
  const void* w; const void* b;                    // [C, K], [C]
  const float* A_log; const float* dt_bias;        // [H]
  void* window; const int* slots; const int* cu; const int* fresh;      // window [S, K - 1, C]
  void* out; float2* gates;                        // [T, C], [T, H]: (log-decay, dt)
  int T, B, H, C, K;
};

// grid = (channel groups, runs); channel groups past C hold the heads' step sizes.  KT: taps (0 = any number).
template <typename T, int KT, int V>
__global__ void __launch_bounds__(128) ssm_prepare_kernel(const SsmArgs a) {
  constexpr int KM = KT ? KT : kMaxTaps;
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const int K = KT ? KT : a.K, C = a.C;
  __shared__ int s_run[2];
  if (threadIdx.x < 32) {
    int seq, tok;
    find_seq_tile(a.cu, a.B, kRun, blockIdx.y, seq, tok);
    if (threadIdx.x == 0) { s_run[0] = seq; s_run[1] = tok; }
  }
  __syncthreads();
  const int seq = s_run[0], t0 = s_run[1];
  if (seq < 0) return;
  const int beg = a.cu[seq], end = a.cu[seq + 1], t1 = min(t0 + kRun, end);
  const int unit = blockIdx.x * blockDim.x + threadIdx.x, cunits = (C + V - 1) / V;
  if (unit >= cunits) {
    const int h = unit - cunits;
    if (h >= a.H) return;
    const float e = -expf(a.A_log[h]), bias = a.dt_bias[h];
    for (int t = t0; t < t1; t++) {
      const float v = a.dt_raw[(long long)t * a.dt_ld + h] + bias;
      const float dt = v > 20.f ? v : log1pf(expf(v));
      a.gates[(long long)t * a.H + h] = make_float2(e * dt, dt);
    }
    return;
  }
  const int c = unit * V;
  const int slot = a.slots[seq];
  if (!NE_INDEX_OK(slot, BK_STATE_SLOTS, 47, __LINE__)) return;
  const bool is_fresh = a.fresh[seq] != 0;
  const T* x = reinterpret_cast<const T*>(a.xbc) + c;
  T* win = reinterpret_cast<T*>(a.window) + (long long)slot * (K - 1) * C + c;
  float w[KM][V], bias[V], h[KM][V];               // h[K - 1 - i]: the input i tokens back
#pragma unroll
  for (int e = 0; e < V; e++)
#pragma unroll
    for (int j = 0; j < KM; j++) if (KT || j < K) w[j][e] = lda(reinterpret_cast<const T*>(a.w) + (long long)(c + e) * K + j);
  ldv<V>(reinterpret_cast<const T*>(a.b) + c, bias);
  // the K - 1 inputs before t0 in h[1 .. K - 1]: the first token shifts them down by one
#pragma unroll
  for (int j = 1; j < KM; j++) {
    if (!KT && j >= K) break;
    const int p = t0 - beg - (K - j);              // its position in this call
    if (p >= 0) ldv<V>(x + (long long)(beg + p) * a.ld, h[j]);
    else if (!is_fresh) ldv<V>(win + (long long)(p + K - 1) * C, h[j]);
    else {
#pragma unroll
      for (int e = 0; e < V; e++) h[j][e] = 0.f;
    }
  }
  if (t0 == beg) {                                 // this thread has read what it needs of its channels' window and nobody else reads it
    const int n = end - beg;
    for (int j = 0; j < K - 1; j++) {
      const int p = n - (K - 1) + j;
      float v[V];
      if (p >= 0) ldv<V>(x + (long long)(beg + p) * a.ld, v);
      else {
#pragma unroll
        for (int e = 0; e < V; e++) v[e] = 0.f;
#pragma unroll
        for (int jj = 1; jj < KM; jj++)            // h[jj] is window entry jj - 1; entry p + K - 1 moves to j
          if ((KT || jj < K) && jj == p + K) {
#pragma unroll
            for (int e = 0; e < V; e++) v[e] = h[jj][e];
          }
      }
      stv<V>(win + (long long)j * C, v);
    }
  }
  T* out = reinterpret_cast<T*>(a.out) + c;
  for (int tb = t0; tb < t1; tb += 4) {            // four tokens' loads in flight
    float cur4[4][V];
#pragma unroll
    for (int u = 0; u < 4; u++) if (tb + u < t1) ldv<V>(x + (long long)(tb + u) * a.ld, cur4[u]);
#pragma unroll
    for (int u = 0; u < 4; u++) {
      if (tb + u >= t1) break;
#pragma unroll
      for (int j = 1; j < KM; j++)
#pragma unroll
        for (int e = 0; e < V; e++) if (KT || j < K) h[j - 1][e] = h[j][e];
      float acc[V];
#pragma unroll
      for (int e = 0; e < V; e++) {
        acc[e] = bias[e];
#pragma unroll
        for (int j = 0; j < KM; j++) {
          if (!KT && j >= K) break;
          if (j == K - 1) h[j][e] = cur4[u][e];
          acc[e] = fmaf(h[j][e], w[j][e], acc[e]);
        }
        acc[e] = silu_t<T>(acc[e]);
      }
      stv<V>(out + (long long)(tb + u) * C, acc);
    }
  }
}

// ---- the recurrence ---------------------------------------------------------------------------------------------------------
struct ScanArgs {
  const void* q; const void* k; const void* v; long long q_ld, k_ld, v_ld;     // [T, Hk, Dk] x 2, [T, H, Dv], heads packed
  const float2* gates;                        // [T, H] (log a, b), or null: a = decay[head], b = 1
  const float* decay; const float* skip;      // [H]; skip null: no d v term
  float* state; const int* slots; const int* cu; const int* fresh;
  float* raw;                                 // [T, H, Dv] fp32
  int T, B, H, Hk, Dk, Dv, act;               // act 1: silu on q, k and v, rounded to their type
  int below;                                  // > 0: only sequences of fewer tokens (the others take the chunked form)
};

constexpr int kScanTok = 16;                  // tokens staged at a time

// grid = (H * splits, B); NW = blockDim.x / 32 warps of 4 R rows each, `splits` CTAs share a head's Dv rows.
template <int CPL, int R, typename T, bool kVec>
__global__ void __launch_bounds__(256, CPL * R >= 64 ? 2 : CPL * R >= 32 ? 3 : 4) decay_scan_kernel(const ScanArgs a) {
  constexpr int DKP = CPL * 8;
  extern __shared__ float sm[];
  const int rows = (blockDim.x >> 5) * 4 * R;
  const int splits = gridDim.x / a.H, h = blockIdx.x / splits, row0 = (blockIdx.x % splits) * rows, hk = h / (a.H / a.Hk);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, cg = lane & 7, rg = lane >> 3;
  const int Dk = a.Dk, Dv = a.Dv, seq = blockIdx.y;
  float* sk = sm;                             // [kScanTok][DKP] x 2, [kScanTok][rows], [kScanTok][2]
  float* sq = sk + kScanTok * DKP;
  float* sv = sq + kScanTok * DKP;
  float* sg = sv + kScanTok * rows;
  if (Dk < DKP)                               // columns past Dk stay zero
    for (int i = threadIdx.x; i < 2 * kScanTok * (DKP - Dk); i += blockDim.x) sm[(i / (DKP - Dk)) * DKP + Dk + i % (DKP - Dk)] = 0.f;
  // The step's tables and the state were written before the kernel in front of this one began (every kernel triggers behind its own
  // wait, and that kernel writes none of these), so they are fetched while it still runs.
  const int start = a.cu[seq], n = a.cu[seq + 1] - start;
  const int slot = a.slots[seq];
  if (n <= 0 || (a.below > 0 && n >= a.below) || !NE_INDEX_OK(slot, BK_STATE_SLOTS, 48, __LINE__)) { pdl_wait(); return; }
  const bool is_fresh = a.fresh[seq] != 0, vec = (Dk & 3) == 0;
  float* Sg = a.state + (((long long)slot * a.H + h) * Dv) * Dk;
  float S[R][CPL];                            // rows row0 + warp * 4R + r * 4 + rg, columns j * 32 + cg * 4 + {0..3}
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
  const float fixed = a.gates ? 0.f : a.decay[h], skip = a.skip ? a.skip[h] : 0.f;
  pdl_wait();
  pdl_trigger();
  const T* qg = reinterpret_cast<const T*>(a.q) + (long long)hk * Dk;
  const T* kg = reinterpret_cast<const T*>(a.k) + (long long)hk * Dk;
  const T* vg = reinterpret_cast<const T*>(a.v) + (long long)h * Dv + row0;
  constexpr int V = kVec ? 4 : 1;
  const int per = Dk / V, vper = rows / V;
  for (int i0 = 0; i0 < n; i0 += kScanTok) {
    const int m = min(kScanTok, n - i0);
    const long long t0 = start + i0;
    for (int i = threadIdx.x; i < m * 2 * per; i += blockDim.x) {
      const int c = (i % per) * V, tok = (i / per) >> 1, which = (i / per) & 1;
      float f[V];
      ldv<V>(which ? qg + (t0 + tok) * a.q_ld + c : kg + (t0 + tok) * a.k_ld + c, f);
#pragma unroll
      for (int e = 0; e < V; e++) (which ? sq : sk)[tok * DKP + c + e] = a.act ? round_as(silu_t<T>(f[e]), qg) : f[e];
    }
    for (int i = threadIdx.x; i < m * vper; i += blockDim.x) {
      const int r = (i % vper) * V, tok = i / vper;
      if (row0 + r >= Dv) continue;             // kVec: Dv is a multiple of 4
      float f[V];
      ldv<V>(vg + (t0 + tok) * a.v_ld + r, f);
#pragma unroll
      for (int e = 0; e < V; e++) sv[tok * rows + r + e] = a.act ? round_as(silu_t<T>(f[e]), qg) : f[e];
    }
    for (int i = threadIdx.x; i < m; i += blockDim.x) {
      if (a.gates) {
        const float2 g = a.gates[(t0 + i) * a.H + h];
        sg[2 * i] = expf(g.x); sg[2 * i + 1] = g.y;
      } else { sg[2 * i] = fixed; sg[2 * i + 1] = 1.f; }
    }
    __syncthreads();
    for (int i = 0; i < m; i++) {
      const float dec = sg[2 * i], b = sg[2 * i + 1];
      float u[R], o[R], vv[R];
#pragma unroll
      for (int r = 0; r < R; r++) { vv[r] = sv[i * rows + warp * 4 * R + r * 4 + rg]; u[r] = b * vv[r]; o[r] = 0.f; }
#pragma unroll
      for (int j = 0; j < CPL / 4; j++) {
        const float4 k4 = *reinterpret_cast<const float4*>(sk + i * DKP + j * 32 + cg * 4), q4 = *reinterpret_cast<const float4*>(sq + i * DKP + j * 32 + cg * 4);
#pragma unroll
        for (int r = 0; r < R; r++) {
          S[r][4 * j] = fmaf(u[r], k4.x, dec * S[r][4 * j]); o[r] = fmaf(S[r][4 * j], q4.x, o[r]);
          S[r][4 * j + 1] = fmaf(u[r], k4.y, dec * S[r][4 * j + 1]); o[r] = fmaf(S[r][4 * j + 1], q4.y, o[r]);
          S[r][4 * j + 2] = fmaf(u[r], k4.z, dec * S[r][4 * j + 2]); o[r] = fmaf(S[r][4 * j + 2], q4.z, o[r]);
          S[r][4 * j + 3] = fmaf(u[r], k4.w, dec * S[r][4 * j + 3]); o[r] = fmaf(S[r][4 * j + 3], q4.w, o[r]);
        }
      }
#pragma unroll
      for (int x = 4; x > 0; x >>= 1)
#pragma unroll
        for (int r = 0; r < R; r++) o[r] += __shfl_xor_sync(0xffffffffu, o[r], x);
      float o_sel = 0.f;
#pragma unroll
      for (int r = 0; r < R; r++) if (cg == r) o_sel = fmaf(skip, vv[r], o[r]);
      const int lrow = warp * 4 * R + cg * 4 + rg;             // the row whose output this lane holds (cg < R)
      if (cg < R && row0 + lrow < Dv) a.raw[((t0 + i) * a.H + h) * Dv + row0 + lrow] = o_sel;
    }
    __syncthreads();
  }
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

template <int CPL, int R, typename T>
static int scan(const ScanArgs& a, int warps, bool spread, cudaStream_t st) {
  const int rows = warps * 4 * R, splits = (a.Dv + rows - 1) / rows;
  const size_t smem = sizeof(float) * kScanTok * (2 * CPL * 8 + rows + 2);
  const bool vec = a.Dk % 4 == 0 && a.Dv % 4 == 0 && a.q_ld % 4 == 0 && a.k_ld % 4 == 0 && a.v_ld % 4 == 0 &&
                   ((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v) % 16 == 0;
  auto k = vec ? decay_scan_kernel<CPL, R, T, true> : decay_scan_kernel<CPL, R, T, false>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  const dim3 grid((unsigned)(a.H * splits), (unsigned)a.B), block((unsigned)(warps * 32));
  if (!spread) return (int)launch_pdl(k, grid, block, smem, st, a);
  // few long CTAs: an ordinary launch spreads them over the machine, a dependent one packs them onto the SMs that drain first
  k<<<grid, block, smem, st>>>(a);
  return (int)cudaGetLastError();
}

template <typename T>
static int scan_t(const ScanArgs& a, int max_q, cudaStream_t st) {
  const int whole4 = (a.Dv + 15) / 16;
  if (max_q <= 4 && a.Dk <= 128) {              // short steps: the state streams once, as many rows per CTA as 8 warps hold
    const int w = whole4 < 8 ? whole4 : 8;
    if (a.Dk <= 32) return scan<4, 4, T>(a, w, false, st);
    if (a.Dk <= 64) return scan<8, 4, T>(a, w, false, st);
    if (a.Dk <= 96) return scan<12, 4, T>(a, w, false, st);
    return scan<16, 4, T>(a, w, false, st);
  }
  const bool spread = max_q > 64, wide = (long long)a.H * a.Dv * a.B >= 148ll * 4 * 16 * 2;
#define NE_SCAN(CPL_) (wide ? scan<CPL_, 4, T>(a, 4, spread, st) : scan<CPL_, 2, T>(a, 4, spread, st))
  if (a.Dk <= 32) return NE_SCAN(4);
  if (a.Dk <= 64) return NE_SCAN(8);
  if (a.Dk <= 96) return NE_SCAN(12);
  if (a.Dk <= 128) return NE_SCAN(16);
#undef NE_SCAN
  if (a.Dk <= 256) return scan<32, 2, T>(a, 4, spread, st);
  return scan<64, 1, T>(a, 4, spread, st);
}

// ---- gated norm of rows -----------------------------------------------------------------------------------------------------
// raw [T, W] fp32, gate [T, W] (row stride g_ld), w [W]; grid = (T, parts), one CTA per part of a row.
//   before = 1: y = raw silu(gate), out = y / rms(y) w scale          before = 0: out = raw / rms(raw) w sigmoid(gate) scale
template <typename T, int V>
__global__ void __launch_bounds__(512) gated_norm_kernel(const float* __restrict__ raw, const T* __restrict__ gate, long long g_ld, const T* __restrict__ w,
                                                        T* __restrict__ out, long long o_ld, int W, int P, int before, float eps, float scale) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  extern __shared__ float srow[];            // P floats
  __shared__ float red[16];
  const long long t = blockIdx.x;
  const int c0 = blockIdx.y * P;
  const float* rr = raw + t * W + c0;
  const T* gr = gate + t * g_ld + c0;
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < P; i += blockDim.x * V) {
    float f[V], g[V];
    ldv<V>(rr + i, f);
    if (before) {
      ldv<V>(gr + i, g);
#pragma unroll
      for (int e = 0; e < V; e++) f[e] *= silu_t<T>(g[e]);
    }
#pragma unroll
    for (int e = 0; e < V; e++) ss += f[e] * f[e];
    stv<V>(srow + i, f);                     // a thread rereads only what it stored itself
  }
  ss = warp_sum(ss);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (nw > 1) {
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = warp_sum(lane < nw ? red[lane] : 0.f);
  }
  const float r = rsqrtf(ss / (float)P + eps) * scale;
  for (int i = threadIdx.x * V; i < P; i += blockDim.x * V) {
    float f[V], g[V], ww[V];
    ldv<V>(srow + i, f); ldv<V>(w + c0 + i, ww);
    if (!before) ldv<V>(gr + i, g);
#pragma unroll
    for (int e = 0; e < V; e++) {
      f[e] *= r * ww[e];
      if (!before) f[e] *= sigm(g[e], gr);
    }
    stv<V>(out + t * o_ld + c0 + i, f);
  }
}

// The same for parts of up to IT * 8 elements per thread, held in registers: all of a thread's loads are in flight before the reduction.
template <typename T, int IT>
__global__ void __launch_bounds__(512) gated_norm_regs_kernel(const float* __restrict__ raw, const T* __restrict__ gate, long long g_ld, const T* __restrict__ w,
                                                             T* __restrict__ out, long long o_ld, int W, int P, int before, float eps, float scale) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  __shared__ float red[16];
  const long long t = blockIdx.x;
  const int c0 = blockIdx.y * P;
  const float* rr = raw + t * W + c0;
  const T* gr = gate + t * g_ld + c0;
  float f[IT][8], g[IT][8], ww[IT][8], ss = 0.f;
#pragma unroll
  for (int it = 0; it < IT; it++) {
    const int i = (it * blockDim.x + threadIdx.x) * 8;
    if (i < P) { lda4(rr + i, f[it]); lda4(rr + i + 4, f[it] + 4); lda4(gr + i, g[it]); lda4(gr + i + 4, g[it] + 4); lda4(w + c0 + i, ww[it]); lda4(w + c0 + i + 4, ww[it] + 4); }
    else {
#pragma unroll
      for (int e = 0; e < 8; e++) f[it][e] = g[it][e] = ww[it][e] = 0.f;
    }
  }
#pragma unroll
  for (int it = 0; it < IT; it++)
#pragma unroll
    for (int e = 0; e < 8; e++) {
      if (before) f[it][e] *= silu_t<T>(g[it][e]);
      ss += f[it][e] * f[it][e];
    }
  ss = warp_sum(ss);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (nw > 1) {
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = warp_sum(lane < nw ? red[lane] : 0.f);
  }
  const float r = rsqrtf(ss / (float)P + eps) * scale;
#pragma unroll
  for (int it = 0; it < IT; it++) {
    const int i = (it * blockDim.x + threadIdx.x) * 8;
    if (i >= P) continue;
#pragma unroll
    for (int e = 0; e < 8; e++) {
      f[it][e] *= r * ww[it][e];
      if (!before) f[it][e] *= sigm(g[it][e], gr);
    }
    sta4(out + t * o_ld + c0 + i, f[it]); sta4(out + t * o_ld + c0 + i + 4, f[it] + 4);
  }
}

template <typename T>
static int gated_norm_t(const float* raw, const void* gate, long long g_ld, const void* w, void* out, long long o_ld, int T_, int W, int parts, int before,
                        float eps, float scale, cudaStream_t st) {
  const int P = W / parts;
  const bool vec = P % 4 == 0 && g_ld % 4 == 0 && o_ld % 4 == 0 && ((uintptr_t)raw | (uintptr_t)gate | (uintptr_t)w | (uintptr_t)out) % 16 == 0;
  if (vec && P % 8 == 0 && P <= 8 * 512 * 2) {
    const int units = P / 8, two = units > 512;
    const int th = ((two ? (units + 1) / 2 : units) + 31) / 32 * 32;
    return (int)launch_pdl(two ? gated_norm_regs_kernel<T, 2> : gated_norm_regs_kernel<T, 1>, dim3((unsigned)T_, (unsigned)parts), dim3((unsigned)th), 0, st, raw,
                           (const T*)gate, g_ld, (const T*)w, (T*)out, o_ld, W, P, before, eps, scale);
  }
  const int per = vec ? 4 : 1;
  int threads = ((P + per - 1) / per + 31) / 32 * 32;
  threads = threads > 512 ? 512 : threads;
  const size_t smem = (size_t)P * sizeof(float);
  auto k = vec ? gated_norm_kernel<T, 4> : gated_norm_kernel<T, 1>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)launch_pdl(k, dim3((unsigned)T_, (unsigned)parts), dim3((unsigned)threads), smem, st, raw, (const T*)gate, g_ld, (const T*)w, (T*)out, o_ld, W, P, before,
                         eps, scale);
}

template <typename T>
static int ssm_prepare_t(const SsmArgs& a, cudaStream_t st) {
  const bool vec = a.K >= 2 && a.K <= 4 && a.C % 4 == 0 && a.ld % 4 == 0 && ((uintptr_t)a.xbc | (uintptr_t)a.window | (uintptr_t)a.out | (uintptr_t)a.b) % 16 == 0;
  const int units = (vec ? a.C / 4 : a.C) + a.H;
  const long long most = (long long)a.T / kRun + a.B, runs = most < a.T ? most : a.T;
  void (*k)(const SsmArgs) = nullptr;
  switch (a.K) {
    case 2: k = vec ? ssm_prepare_kernel<T, 2, 4> : ssm_prepare_kernel<T, 2, 1>; break;
    case 3: k = vec ? ssm_prepare_kernel<T, 3, 4> : ssm_prepare_kernel<T, 3, 1>; break;
    case 4: k = vec ? ssm_prepare_kernel<T, 4, 4> : ssm_prepare_kernel<T, 4, 1>; break;
    default: k = ssm_prepare_kernel<T, 0, 1>; break;
  }
  if (runs > 65535) return 1002;
  return (int)launch_pdl(k, dim3((unsigned)((units + 127) / 128), (unsigned)runs), dim3(128), 0, st, a);
}

}  // namespace ne

using namespace ne;

// Convolution + bias + silu of xbc [T, C] (row stride ld, activation dtype) into out [T, C], gates [T, H, 2] fp32 = (-exp(A_log) dt, dt) with
// dt = softplus(dt_raw + dt_bias); window [S, K - 1, C] moves on.
extern "C" int ne_ssm_prepare(const void* xbc, long long ld, const float* dt_raw, long long dt_ld, const void* w, const void* b, const float* A_log,
                              const float* dt_bias, void* window, const int* slots, const int* cu, const int* fresh, void* out, float* gates, int T, int B, int H,
                              int C, int K, int fp32, cudaStream_t st) {
  if (T <= 0 || B <= 0) return 0;
  if (K < 1 || K > kMaxTaps || H < 1 || C < 1) return 1001;
  SsmArgs a;
  a.xbc = xbc; a.ld = ld; a.dt_raw = dt_raw; a.dt_ld = dt_ld; a.w = w; a.b = b; a.A_log = A_log; a.dt_bias = dt_bias; a.window = window; a.slots = slots; a.cu = cu;
  a.fresh = fresh; a.out = out; a.gates = reinterpret_cast<float2*>(gates); a.T = T; a.B = B; a.H = H; a.C = C; a.K = K;
  return fp32 ? ssm_prepare_t<float>(a, st) : ssm_prepare_t<__nv_bfloat16>(a, st);
}

// The recurrence token by token.  q, k [T, Hk, Dk], v [T, H, Dv] in the activation dtype (row strides in elements, heads packed), gates
// [T, H, 2] or null (then decay [H]), skip [H] or null, state [S, H, Dv, Dk] fp32, raw [T, H, Dv] fp32.  below > 0: only the sequences with fewer
// new tokens than that.
extern "C" int ne_decay_scan(const void* q, long long q_ld, const void* k, long long k_ld, const void* v, long long v_ld, const float* gates, const float* decay,
                             const float* skip, float* state, const int* slots, const int* cu, const int* fresh, float* raw, int T, int B, int H, int Hk, int Dk,
                             int Dv, int act, int max_q, int below, int fp32, cudaStream_t st) {
  if (T <= 0 || B <= 0) return 0;
  if (Hk < 1 || H % Hk || Dk < 1 || Dk > 512 || Dv < 1 || B > 65535 || (!gates && !decay)) return 1001;
  ScanArgs a;
  a.q = q; a.k = k; a.v = v; a.q_ld = q_ld; a.k_ld = k_ld; a.v_ld = v_ld; a.gates = reinterpret_cast<const float2*>(gates); a.decay = decay; a.skip = skip;
  a.state = state; a.slots = slots; a.cu = cu; a.fresh = fresh; a.raw = raw; a.T = T; a.B = B; a.H = H; a.Hk = Hk; a.Dk = Dk; a.Dv = Dv; a.act = act; a.below = below;
  if (below > 0 && max_q >= below) max_q = below - 1;
  return fp32 ? scan_t<float>(a, max_q, st) : scan_t<__nv_bfloat16>(a, max_q, st);
}

extern "C" int ne_gated_norm(const float* raw, const void* gate, long long g_ld, const void* w, void* out, long long o_ld, int T, int W, int parts, int before,
                             float eps, float scale, int fp32, cudaStream_t st) {
  if (T <= 0) return 0;
  if (parts < 1 || W % parts || parts > 65535 || W / parts > 48 * 1024) return 1001;
  return fp32 ? gated_norm_t<float>(raw, gate, g_ld, w, out, o_ld, T, W, parts, before, eps, scale, st)
              : gated_norm_t<__nv_bfloat16>(raw, gate, g_ld, w, out, o_ld, T, W, parts, before, eps, scale, st);
}
