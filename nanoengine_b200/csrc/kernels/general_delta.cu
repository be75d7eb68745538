// Generalised delta rule with a decay and a removal rate per key channel, everything between the projections in 32-bit: any head sizes
// (Dk <= 512), bf16 or fp32 activations, any mix of prompt portions and single tokens in one call.  Per head, with u = k / |k|:
//   S <- S diag(w) - (S u) (a u)^T + v k^T,   o = S r      (rows of S: value channels; both terms read the old state)
//   w = exp(-exp(-1/2) sigmoid(decay + w0)),  a = sigmoid(a + a_bias);  then o / rms(o) * norm_w * sigmoid(g)
// Rows of a head's [Dv, Dk] state are independent of each other, so a CTA owns some rows of one (sequence, head) in registers: 8 lanes share
// a row (each CPL of its columns), a warp holds 4 R rows.  A token costs two dot products with the old state, p = S.u and q = S.(r w), and one
// update, all in packed pairs of fp32; o = q + (|k| v) (r.u) - p (r.(a u)), so nothing waits for the new state.  The 2 R sums of a row group are
// reduced over its lanes by halving (every exchange leaves each lane half of the sums) and the p handed back.
//   single tokens: one kernel.  A CTA or a pair of them holds a whole head; its state is fetched while the kernel in front still runs; gates and unit keys are
//   made in it, and norm and gate are applied before the row leaves.
//   otherwise: general_delta_prepare (one warp per (token, head)) writes u | w | a u | r w, general_delta_scan runs the recurrence with the
//   next tokens' vectors on their way (bulk copies), general_delta_norm finishes.
// The same arithmetic in the same order runs whatever the portions are, so a sequence cut differently gives the same state.
#include "ptx.cuh"

namespace ne {

__device__ __forceinline__ float ldg_(const float* p) { return *p; }
__device__ __forceinline__ float ldg_(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stg_(float* p, float v) { *p = v; }
__device__ __forceinline__ void stg_(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void ldv4(const float* p, float* o) {
  const float4 v = *reinterpret_cast<const float4*>(p);
  o[0] = v.x; o[1] = v.y; o[2] = v.z; o[3] = v.w;
}
__device__ __forceinline__ void ldv4(const __nv_bfloat16* p, float* o) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 x = unpack_bf16x2(u.x), y = unpack_bf16x2(u.y);
  o[0] = x.x; o[1] = x.y; o[2] = y.x; o[3] = y.y;
}
__device__ __forceinline__ float sigmoid_(float x) { return 1.f / (1.f + expf(-x)); }

// pairs of fp32
typedef unsigned long long f2;
__device__ __forceinline__ f2 pack2(float a, float b) { f2 r; asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b)); return r; }
__device__ __forceinline__ float2 unpack2(f2 v) { float2 r; asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v)); return r; }
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) { f2 r; asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c)); return r; }
__device__ __forceinline__ f2 mul2(f2 a, f2 b) { f2 r; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b)); return r; }

struct GdArgs {
  const void* proj; long long proj_ld;       // [T, r | k | a | v | g]
  const float* decay; long long decay_ld;    // [T, >= H Dk]
  const float* w0; const float* a_bias;      // [H Dk]
  const void* norm_w; float eps;             // [H Dv]
  float* state;                              // [S, H, Dv, Dk]
  const int* slots; const int* cu; const int* fresh;
  float* vec; float* val; float* scal;       // [T, H, 4, DkP]: u, w, a u, r w (zeros past Dk); [T, H, DvP]: |k| v, then o; [T, H, 4]: r.u, r.(a u)
  void* out;                                 // [T, H, Dv]
  int T, B, H, Dk, Dv, DkP, DvP;
};

// Whole warp: the vectors of one (token, head), `ld` floats apart, zeros from Dk to `pad`.  Returns |k|; r.u and r.(a u) in ru, rau.
template <typename T, int V>
__device__ __forceinline__ float head_vectors(const GdArgs& a, long long t, int h, float* dst, int ld, int pad, float& ru, float& rau) {
  constexpr float kRate = 0.60653065971263342f;      // exp(-1/2)
  const int lane = threadIdx.x & 31, Dk = a.Dk, hk = a.H * Dk;
  const T* row = reinterpret_cast<const T*>(a.proj) + t * a.proj_ld + h * Dk;
  const float* dec = a.decay + t * a.decay_ld + h * Dk;
  const float *w0 = a.w0 + h * Dk, *ab = a.a_bias + h * Dk;
  float kk = 0.f;
  for (int c = lane * V; c < Dk; c += 32 * V) {
    float k[V];
    if constexpr (V == 4) ldv4(row + hk + c, k); else k[0] = ldg_(row + hk + c);
#pragma unroll
    for (int e = 0; e < V; e++) kk += k[e] * k[e];
  }
  kk = warp_sum(kk) + 1e-6f;
  const float inv = rsqrtf(kk);
  ru = rau = 0.f;
  for (int c = lane * V; c < pad; c += 32 * V) {
    float r[V], k[V], z[V], s[V], o[4][V];
    if (c < Dk) {
      if constexpr (V == 4) {
        ldv4(row + c, r); ldv4(row + hk + c, k); ldv4(row + 2 * hk + c, s); ldv4(dec + c, z);
        float b[4], d[4];
        ldv4(w0 + c, d); ldv4(ab + c, b);
#pragma unroll
        for (int e = 0; e < 4; e++) { z[e] += d[e]; s[e] += b[e]; }
      } else { r[0] = ldg_(row + c); k[0] = ldg_(row + hk + c); s[0] = ldg_(row + 2 * hk + c) + ab[c]; z[0] = dec[c] + w0[c]; }
#pragma unroll
      for (int e = 0; e < V; e++) {
        const float w = expf(-kRate * sigmoid_(z[e])), u = k[e] * inv, au = sigmoid_(s[e]) * u;
        o[0][e] = u; o[1][e] = w; o[2][e] = au; o[3][e] = r[e] * w;
        ru = fmaf(r[e], u, ru); rau = fmaf(r[e], au, rau);
      }
    } else {
#pragma unroll
      for (int e = 0; e < V; e++) o[0][e] = o[1][e] = o[2][e] = o[3][e] = 0.f;
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
      if constexpr (V == 4) *reinterpret_cast<float4*>(dst + i * ld + c) = make_float4(o[i][0], o[i][1], o[i][2], o[i][3]);
      else dst[i * ld + c] = o[i][0];
    }
  }
  ru = warp_sum(ru); rau = warp_sum(rau);
  return kk * inv;
}

template <typename T, int V>
__global__ void __launch_bounds__(256) general_delta_prepare_kernel(const GdArgs a) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const long long i = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (i >= (long long)a.T * a.H) return;
  const int lane = threadIdx.x & 31, h = (int)(i % a.H);
  const long long t = i / a.H;
  float ru, rau;
  const float kn = head_vectors<T, V>(a, t, h, a.vec + i * 4 * a.DkP, a.DkP, a.DkP, ru, rau);
  const T* v = reinterpret_cast<const T*>(a.proj) + t * a.proj_ld + 3 * a.H * a.Dk + h * a.Dv;
  float* vo = a.val + i * a.DvP;
  if (V == 4 && a.Dv % 4 == 0) {
    for (int c = lane * 4; c < a.Dv; c += 128) {
      float x[4];
      ldv4(v + c, x);
      *reinterpret_cast<float4*>(vo + c) = make_float4(kn * x[0], kn * x[1], kn * x[2], kn * x[3]);
    }
  } else {
    for (int c = lane; c < a.Dv; c += 32) vo[c] = kn * ldg_(v + c);
  }
  if (lane == 0) { a.scal[i * 4] = ru; a.scal[i * 4 + 1] = rau; }
}

// One token for the rows of a row group.  S: packed columns j * 32 + cg * 4 + {0, 1}, {2, 3}; vec: u | w | a u | r w, `ld` floats apart; kv: |k| v of
// the thread's rows, kv_o that of the row whose output this lane returns (see out_row).  kHold: u stays in
// registers for the update.
template <int CPL, int R, bool kHold>
__device__ __forceinline__ float delta_token(f2 (&S)[R][CPL / 2], const float* vec, int ld, int cg, const float (&kv)[R], float kv_o, float ru, float rau) {
  f2 p2[R], q2[R];
#pragma unroll
  for (int r = 0; r < R; r++) p2[r] = q2[r] = 0ull;
  ulonglong2 uh[kHold ? CPL / 4 : 1];
#pragma unroll
  for (int j = 0; j < CPL / 4; j++) {
    const ulonglong2 u = *reinterpret_cast<const ulonglong2*>(vec + j * 32 + cg * 4);
    if (kHold) uh[j] = u;
    const ulonglong2 q = *reinterpret_cast<const ulonglong2*>(vec + 3 * ld + j * 32 + cg * 4);
#pragma unroll
    for (int r = 0; r < R; r++) {
      p2[r] = fma2(S[r][2 * j], u.x, p2[r]); q2[r] = fma2(S[r][2 * j], q.x, q2[r]);
      p2[r] = fma2(S[r][2 * j + 1], u.y, p2[r]); q2[r] = fma2(S[r][2 * j + 1], q.y, q2[r]);
    }
  }
  float x[2 * R];
#pragma unroll
  for (int r = 0; r < R; r++) {
    const float2 a = unpack2(p2[r]), b = unpack2(q2[r]);
    x[r] = a.x + a.y; x[R + r] = b.x + b.y;
  }
  // lanes 0-3 of the group keep p, 4-7 keep q; then rows are halved, and what is left is summed over the lanes that share it
#pragma unroll
  for (int n = R, o = 4; o > 0; o >>= 1, n >>= 1) {
    if (n >= 1) {
      const bool up = (cg & o) != 0;
#pragma unroll
      for (int i = 0; i < n; i++) {
        const float keep = up ? x[n + i] : x[i], send = up ? x[i] : x[n + i];
        x[i] = keep + __shfl_xor_sync(0xffffffffu, send, o);
      }
    } else {
      x[0] += __shfl_xor_sync(0xffffffffu, x[0], o);
    }
  }
  const float p_o = __shfl_xor_sync(0xffffffffu, x[0], 4);      // for the upper lanes: p of the row whose q they hold
  float p[R];
#pragma unroll
  for (int r = 0; r < R; r++) p[r] = __shfl_sync(0xffffffffu, x[0], (threadIdx.x & 24) + r * (4 / R));
  const float out = fmaf(kv_o, ru, fmaf(-p_o, rau, x[0]));
  f2 kv2[R], np2[R];
#pragma unroll
  for (int r = 0; r < R; r++) { kv2[r] = pack2(kv[r], kv[r]); np2[r] = pack2(-p[r], -p[r]); }
#pragma unroll
  for (int j = 0; j < CPL / 4; j++) {
    const ulonglong2 u = kHold ? uh[kHold ? j : 0] : *reinterpret_cast<const ulonglong2*>(vec + j * 32 + cg * 4);
    const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(vec + ld + j * 32 + cg * 4),
                     au = *reinterpret_cast<const ulonglong2*>(vec + 2 * ld + j * 32 + cg * 4);
#pragma unroll
    for (int r = 0; r < R; r++) {
      S[r][2 * j] = fma2(w.x, S[r][2 * j], fma2(u.x, kv2[r], mul2(au.x, np2[r])));
      S[r][2 * j + 1] = fma2(w.y, S[r][2 * j + 1], fma2(u.y, kv2[r], mul2(au.y, np2[r])));
    }
  }
  return out;
}
// the row (of the thread's R) whose output a lane of the group gets from delta_token, -1: none
template <int R> __device__ __forceinline__ int out_row(int cg) { return cg < 4 || (cg & (4 / R - 1)) ? -1 : (cg & 3) / (4 / R); }

template <int CPL, int R>
__device__ __forceinline__ void load_state(f2 (&S)[R][CPL / 2], const float* Sg, int row0, int rg, int cg, int Dv, int Dk, bool zero) {
  if (Dk == CPL * 8 && row0 + 4 * R <= Dv) {          // whole rows: nothing between one load and the next
    if (zero) {
#pragma unroll
      for (int r = 0; r < R; r++)
#pragma unroll
        for (int j = 0; j < CPL / 2; j++) S[r][j] = 0ull;
      return;
    }
    const float* src = Sg + (long long)(row0 + rg) * Dk + cg * 4;
#pragma unroll
    for (int r = 0; r < R; r++)
#pragma unroll
      for (int j = 0; j < CPL / 4; j++) {
        const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(src + r * 4 * CPL * 8 + j * 32);
        S[r][2 * j] = v.x; S[r][2 * j + 1] = v.y;
      }
    return;
  }
  const bool vec = (Dk & 3) == 0;
#pragma unroll
  for (int r = 0; r < R; r++) {
    const int row = row0 + r * 4 + rg;
#pragma unroll
    for (int j = 0; j < CPL / 4; j++) {
      const int c = j * 32 + cg * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!zero && row < Dv) {
        const float* src = Sg + (long long)row * Dk + c;
        if (vec) { if (c < Dk) v = *reinterpret_cast<const float4*>(src); }
        else { if (c < Dk) v.x = src[0]; if (c + 1 < Dk) v.y = src[1]; if (c + 2 < Dk) v.z = src[2]; if (c + 3 < Dk) v.w = src[3]; }
      }
      S[r][2 * j] = pack2(v.x, v.y); S[r][2 * j + 1] = pack2(v.z, v.w);
    }
  }
}
template <int CPL, int R>
__device__ __forceinline__ void store_state(const f2 (&S)[R][CPL / 2], float* Sg, int row0, int rg, int cg, int Dv, int Dk) {
  if (Dk == CPL * 8 && row0 + 4 * R <= Dv) {
    float* dst = Sg + (long long)(row0 + rg) * Dk + cg * 4;
#pragma unroll
    for (int r = 0; r < R; r++)
#pragma unroll
      for (int j = 0; j < CPL / 4; j++) *reinterpret_cast<ulonglong2*>(dst + r * 4 * CPL * 8 + j * 32) = make_ulonglong2(S[r][2 * j], S[r][2 * j + 1]);
    return;
  }
  const bool vec = (Dk & 3) == 0;
#pragma unroll
  for (int r = 0; r < R; r++) {
    const int row = row0 + r * 4 + rg;
    if (row >= Dv) continue;
#pragma unroll
    for (int j = 0; j < CPL / 4; j++) {
      const int c = j * 32 + cg * 4;
      float* dst = Sg + (long long)row * Dk + c;
      const float2 x = unpack2(S[r][2 * j]), y = unpack2(S[r][2 * j + 1]);
      if (vec) { if (c < Dk) *reinterpret_cast<float4*>(dst) = make_float4(x.x, x.y, y.x, y.y); }
      else { if (c < Dk) dst[0] = x.x; if (c + 1 < Dk) dst[1] = x.y; if (c + 2 < Dk) dst[2] = y.x; if (c + 3 < Dk) dst[3] = y.y; }
    }
  }
}

// up to four elements from column c of n; vec: one access
template <typename T>
__device__ __forceinline__ void ld_up4(const T* p, int c, int n, bool vec, float* o) {
  if (vec) { if (c < n) ldv4(p + c, o); else o[0] = o[1] = o[2] = o[3] = 0.f; return; }
#pragma unroll
  for (int e = 0; e < 4; e++) o[e] = c + e < n ? ldg_(p + c + e) : 0.f;
}

__device__ __forceinline__ void st_cluster(uint32_t addr, float v) { asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(addr), "f"(v) : "memory"); }

// arrive / wait of the cluster's barrier
__device__ __forceinline__ void cluster_arrive_() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait_() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }

// Single tokens (a sequence may bring a few): grid (H CL, B), a cluster of CL CTAs holds a head in warps of 16 rows (small CTAs: more of them
// are at different stages of fetching, computing and storing on an SM); warp 0 makes the token's vectors while the state is on its way.
template <int CPL, int CL, typename T, bool VEC>
__global__ void __cluster_dims__(CL, 1, 1) __launch_bounds__(256 / CL, 2 * CL) general_delta_step_kernel(const GdArgs a) {
  constexpr int DKP = CPL * 8, R = 4;
  constexpr float kRate = 0.60653065971263342f;      // exp(-1/2)
  __shared__ float4 s_vec4[DKP];             // u | w | a u | r w
  __shared__ float4 s_kv4[32], s_out4[32];   // v; norm weight * sigmoid(g)
  __shared__ float s_scal[3], s_red[2][8];   // r.u, r.(a u), |k|; sums of squares of every warp of the cluster
  float *s_vec = reinterpret_cast<float*>(s_vec4), *s_kv = reinterpret_cast<float*>(s_kv4), *s_out = reinterpret_cast<float*>(s_out4);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, cg = lane & 7, rg = lane >> 3, nw = blockDim.x >> 5;
  const int h = blockIdx.x / CL, part = blockIdx.x % CL, row0 = part * nw * 16 + warp * 16, seq = blockIdx.y, Dk = a.Dk, Dv = a.Dv, hk = a.H * Dk, c = lane * 4;
  // The step's tables and the state are older than the kernel in front (every kernel triggers behind its own wait): fetched while it runs.
  const int start = a.cu[seq], n = a.cu[seq + 1] - start, slot = a.slots[seq];
  if (n <= 0 || !NE_INDEX_OK(slot, BK_STATE_SLOTS, 48, __LINE__)) { pdl_wait(); return; }
  float* Sg = a.state + (((long long)slot * a.H + h) * Dv) * Dk;
  const bool fresh = a.fresh[seq] != 0;
  f2 S[R][CPL / 2];
  if (warp != 0) load_state<CPL, R>(S, Sg, row0, rg, cg, Dv, Dk, fresh);
  pdl_wait(); pdl_trigger();
  const int orow = out_row<R>(cg), lrow = row0 + max(orow, 0) * 4 + rg;
  for (int i = 0; i < n; i++) {
    const long long t = start + i;
    if (warp == 0) {                         // the vectors' loads in front of the state's
      const T* p = reinterpret_cast<const T*>(a.proj) + t * a.proj_ld + h * Dk;
      float r[4], k[4], s[4], z[4], w0[4], ab[4];
      ld_up4(p + hk, c, Dk, VEC, k); ld_up4(a.decay + t * a.decay_ld + h * Dk, c, Dk, VEC, z); ld_up4(p + 2 * hk, c, Dk, VEC, s); ld_up4(p, c, Dk, VEC, r);
      ld_up4(a.w0 + h * Dk, c, Dk, VEC, w0); ld_up4(a.a_bias + h * Dk, c, Dk, VEC, ab);
      if (i == 0) load_state<CPL, R>(S, Sg, row0, rg, cg, Dv, Dk, fresh);
      const float kk = warp_sum(k[0] * k[0] + k[1] * k[1] + k[2] * k[2] + k[3] * k[3]) + 1e-6f;
      const float inv = rsqrtf(kk);
      float ru = 0.f, rau = 0.f, o[4][4];
#pragma unroll
      for (int e = 0; e < 4; e++) {
        const float w = expf(-kRate * sigmoid_(z[e] + w0[e])), u = k[e] * inv, au = sigmoid_(s[e] + ab[e]) * u;
        o[0][e] = u; o[1][e] = w; o[2][e] = au; o[3][e] = r[e] * w;
        ru = fmaf(r[e], u, ru); rau = fmaf(r[e], au, rau);
      }
      if (c < DKP)
#pragma unroll
        for (int x = 0; x < 4; x++) *reinterpret_cast<float4*>(s_vec + x * DKP + c) = make_float4(o[x][0], o[x][1], o[x][2], o[x][3]);
      ru = warp_sum(ru); rau = warp_sum(rau);
      if (lane == 0) { s_scal[0] = ru; s_scal[1] = rau; s_scal[2] = kk * inv; }
    }
    if (warp == nw / 2) {                    // and another warp those of its rows
      const T* pv = reinterpret_cast<const T*>(a.proj) + t * a.proj_ld + 3 * hk + h * Dv;
      float v[4], g[4], nw4[4];
      ld_up4(pv, c, Dv, VEC, v); ld_up4(pv + a.H * Dv, c, Dv, VEC, g); ld_up4(reinterpret_cast<const T*>(a.norm_w) + h * Dv, c, Dv, VEC, nw4);
      s_kv4[lane] = make_float4(v[0], v[1], v[2], v[3]);
      s_out4[lane] = make_float4(nw4[0] * sigmoid_(g[0]), nw4[1] * sigmoid_(g[1]), nw4[2] * sigmoid_(g[2]), nw4[3] * sigmoid_(g[3]));
    }
    __syncthreads();
    const float kn = s_scal[2];
    float kv[R];
#pragma unroll
    for (int r = 0; r < R; r++) kv[r] = kn * s_kv[row0 + r * 4 + rg];
    const float o = delta_token<CPL, R, false>(S, s_vec, DKP, cg, kv, kn * s_kv[lrow], s_scal[0], s_scal[1]);
    const bool mine = orow >= 0 && lrow < Dv;
    const float ss = warp_sum(mine ? o * o : 0.f);
    if (CL > 1) { if (lane < CL) st_cluster(mapa_shared(smem_u32(&s_red[i & 1][part * nw + warp]), lane), ss); }
    else if (lane == 0) s_red[i & 1][warp] = ss;
    if (CL > 1) cluster_arrive_();
    if (i + 1 == n) store_state<CPL, R>(S, Sg, row0, rg, cg, Dv, Dk);
    if (CL > 1) cluster_wait_(); else __syncthreads();
    float tot = 0.f;
    for (int w = 0; w < CL * nw; w++) tot += s_red[i & 1][w];
    if (mine) stg_(reinterpret_cast<T*>(a.out) + (t * a.H + h) * Dv + lrow, o * rsqrtf(tot / (float)Dv + a.eps) * s_out[lrow]);
    if (i + 1 < n) __syncthreads();          // the vectors are read by now (and the sums of the token before the next)
  }
}

// untiled bulk copy: addresses and size in multiples of 16 bytes
__device__ __forceinline__ void bulk_load(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}
constexpr int kKernelGd = 15;

// grid = (H * splits, B), 4 warps of 4 R rows; `splits` CTAs share a head's Dv rows.  CH tokens are staged at a time, three buffers; every
// warp issues the bulk copies of a quarter of them, and the warps drift apart by up to a chunk (full and empty barriers, no CTA-wide one).
template <int CPL, int R, int CH>
__global__ void __launch_bounds__(128, CPL * R >= 64 ? 3 : CPL * R >= 32 ? 4 : 6) general_delta_scan_kernel(const GdArgs a) {
  constexpr int DKP = CPL * 8, rows = 16 * R, kBuf = CH * (4 * DKP + rows + 4);
  extern __shared__ __align__(128) float sm[];                    // per buffer: vectors [CH][4][DKP] | |k| v [CH][rows] | r.u, r.(a u) [CH][4]
  constexpr int NB = 3;
  __shared__ uint64_t bars[2 * NB];                                // full | empty
  __shared__ int abort_word;
  volatile int* abort_flag = &abort_word;
  const int splits = gridDim.x / a.H, h = blockIdx.x / splits, row0 = (blockIdx.x % splits) * rows;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, cg = lane & 7, rg = lane >> 3;
  const int Dk = a.Dk, Dv = a.Dv, seq = blockIdx.y;
  const int start = a.cu[seq], n = a.cu[seq + 1] - start, slot = a.slots[seq];
  if (n <= 0 || !NE_INDEX_OK(slot, BK_STATE_SLOTS, 49, __LINE__)) return;
  if (threadIdx.x == 0) {
    for (int b = 0; b < NB; b++) { mbar_init(smem_u32(bars + b), 4); mbar_init(smem_u32(bars + NB + b), 4); }
    abort_word = 0;
    mbar_fence_init();
  }
  __syncthreads();
  const int vrows = min(rows, a.DvP - row0);                       // a multiple of 4; rows past Dv read whatever their scratch holds and are not kept
  static_assert(CH % 4 == 0 && CH <= 32, "a warp's share of a chunk is whole tokens, one copy per lane");
  auto stage = [&](int buf, int i0) {
    const int first = warp * (CH / 4), m = max(0, min(CH / 4, n - i0 - first));       // this warp's tokens of the chunk
    float* base = sm + buf * kBuf;
    const uint32_t bar = smem_u32(bars + buf);
    if (lane == 0) { if (m) mbar_expect_tx(bar, m * (4 * DKP + vrows + 4) * 4); else mbar_arrive(bar); }
    __syncwarp();
    if (lane < 3 * m) {
      const int tok = first + lane / 3, which = lane % 3;
      const long long th = (long long)(start + i0 + tok) * a.H + h;
      if (which == 0) bulk_load(smem_u32(base + tok * 4 * DKP), a.vec + th * 4 * DKP, 16 * DKP, bar);
      else if (which == 1) bulk_load(smem_u32(base + CH * 4 * DKP + tok * rows), a.val + th * a.DvP + row0, vrows * 4, bar);
      else bulk_load(smem_u32(base + CH * (4 * DKP + rows) + tok * 4), a.scal + th * 4, 16, bar);
    }
  };
  for (int c = 0; c < NB - 1 && c * CH < n; c++) stage(c, c * CH);
  float* Sg = a.state + (((long long)slot * a.H + h) * Dv) * Dk;
  f2 S[R][CPL / 2];
  const int wrow = warp * 4 * R;
  load_state<CPL, R>(S, Sg, row0 + wrow, rg, cg, Dv, Dk, a.fresh[seq] != 0);
  const int orow = out_row<R>(cg), lrow = wrow + max(orow, 0) * 4 + rg;
  const bool keep = orow >= 0 && row0 + lrow < Dv;
  bool ok = true;
  for (int i0 = 0, it = 0; i0 < n; i0 += CH, it++) {
    const int m = min(CH, n - i0), buf = it % NB;
    if (i0 + (NB - 1) * CH < n) {                                // chunk it + 2 goes where chunk it - 1 was
      const int nb = (it + NB - 1) % NB;
      if (it > 0 && !mbar_wait(smem_u32(bars + NB + nb), ((it - 1) / NB) & 1, abort_flag, kKernelGd, 410 + nb)) { ok = false; break; }
      stage(nb, i0 + (NB - 1) * CH);
    }
    if (!mbar_wait(smem_u32(bars + buf), (it / NB) & 1, abort_flag, kKernelGd, 400 + buf)) { ok = false; break; }
    const float* vec = sm + buf * kBuf;
    const float *sv = vec + CH * 4 * DKP, *sg = sv + CH * rows;
    float* ov = a.val + ((long long)(start + i0) * a.H + h) * a.DvP + row0 + lrow;       // |k| v of these places has been read
#pragma unroll 2
    for (int i = 0; i < m; i++) {
      float kv[R];
#pragma unroll
      for (int r = 0; r < R; r++) kv[r] = sv[i * rows + wrow + r * 4 + rg];
      const float2 gt = *reinterpret_cast<const float2*>(sg + i * 4);
      const float o = delta_token<CPL, R, (CPL <= 16)>(S, vec + i * 4 * DKP, DKP, cg, kv, sv[i * rows + lrow], gt.x, gt.y);
      if (keep) ov[(long long)i * a.H * a.DvP] = o;
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(smem_u32(bars + NB + buf));
  }
  // a wait gave up (reported): copies in flight land before the CTA goes, and the warp's rows stay as they were
  if (!ok) for (int i = 0; i < 2000; i++) __nanosleep(1000);
  if (ok) store_state<CPL, R>(S, Sg, row0 + wrow, rg, cg, Dv, Dk);
}

// One warp per (token, head): out = o / rms(o) * norm_w * sigmoid(g).  V = 4: sizes, strides and addresses allow groups of four.
template <typename T, int V>
__global__ void __launch_bounds__(256) general_delta_norm_kernel(const GdArgs a) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const long long i = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (i >= (long long)a.T * a.H) return;
  const int lane = threadIdx.x & 31, h = (int)(i % a.H), Dv = a.Dv;
  const float* o = a.val + i * a.DvP;
  const T* g = reinterpret_cast<const T*>(a.proj) + (i / a.H) * a.proj_ld + a.H * (3 * a.Dk + Dv) + h * Dv;
  const T* w = reinterpret_cast<const T*>(a.norm_w) + h * Dv;
  T* out = reinterpret_cast<T*>(a.out) + i * Dv;
  float ss = 0.f;
  for (int d = lane * V; d < Dv; d += 32 * V) {
    float x[V];
    if constexpr (V == 4) ldv4(o + d, x); else x[0] = o[d];
#pragma unroll
    for (int e = 0; e < V; e++) ss += x[e] * x[e];
  }
  const float r = rsqrtf(warp_sum(ss) / (float)Dv + a.eps);
  for (int d = lane * V; d < Dv; d += 32 * V) {
    if constexpr (V == 4) {
      float x[4], gg[4], ww[4];
      ldv4(o + d, x); ldv4(g + d, gg); ldv4(w + d, ww);
      T y[4];
#pragma unroll
      for (int e = 0; e < 4; e++) stg_(y + e, x[e] * r * ww[e] * sigmoid_(gg[e]));
      if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(out + d) = *reinterpret_cast<uint2*>(y);
      else *reinterpret_cast<uint4*>(out + d) = *reinterpret_cast<uint4*>(y);
    } else {
      stg_(out + d, o[d] * r * ldg_(w + d) * sigmoid_(ldg_(g + d)));
    }
  }
}

template <int CPL, int R>
static int gd_scan(const GdArgs& a, cudaStream_t st) {
  constexpr int CH = CPL <= 32 ? 8 : 4, rows = 16 * R;
  const size_t smem = sizeof(float) * 3 * CH * (4 * CPL * 8 + rows + 4);
  auto k = general_delta_scan_kernel<CPL, R, CH>;
  cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return (int)e;
  // an ordinary launch: a dependent one would pack its few long CTAs onto the SMs that drain first
  k<<<dim3((unsigned)(a.H * ((a.Dv + rows - 1) / rows)), (unsigned)a.B), dim3(128), smem, st>>>(a);
  return (int)cudaGetLastError();
}

// columns a row is held in: 8 lanes times the columns of the kernel that takes the size
static int gd_padded(int Dk) { return Dk <= 32 ? 32 : Dk <= 64 ? 64 : Dk <= 96 ? 96 : Dk <= 128 ? 128 : Dk <= 192 ? 192 : Dk <= 256 ? 256 : 512; }
static bool gd_whole(int Dk, int Dv, int max_q) { return max_q <= 2 && Dk <= 128 && Dv <= 128; }

template <typename T>
static int general_delta_t(const GdArgs& a, int max_q, cudaStream_t st) {
  const bool fours = a.Dk % 4 == 0 && a.Dv % 4 == 0 && a.proj_ld % 4 == 0 && a.decay_ld % 4 == 0 &&
                     ((uintptr_t)a.proj | (uintptr_t)a.decay | (uintptr_t)a.w0 | (uintptr_t)a.a_bias | (uintptr_t)a.norm_w | (uintptr_t)a.out) % 16 == 0;
  if (gd_whole(a.Dk, a.Dv, max_q)) {
    const int cl = a.Dv > 64 ? 2 : 1;
    const dim3 grid((unsigned)(a.H * cl), (unsigned)a.B), block((unsigned)(((a.Dv + cl - 1) / cl + 15) / 16 * 32));
#define NE_STEP(CPL_, CL_) (int)launch_pdl(fours ? general_delta_step_kernel<CPL_, CL_, T, true> : general_delta_step_kernel<CPL_, CL_, T, false>, grid, block, 0, st, a)
    if (cl == 2) return a.Dk <= 32 ? NE_STEP(4, 2) : a.Dk <= 64 ? NE_STEP(8, 2) : a.Dk <= 96 ? NE_STEP(12, 2) : NE_STEP(16, 2);
    return a.Dk <= 32 ? NE_STEP(4, 1) : a.Dk <= 64 ? NE_STEP(8, 1) : a.Dk <= 96 ? NE_STEP(12, 1) : NE_STEP(16, 1);
#undef NE_STEP
  }
  const dim3 wgrid((unsigned)(((long long)a.T * a.H + 7) / 8));
  cudaError_t e = launch_pdl(fours ? general_delta_prepare_kernel<T, 4> : general_delta_prepare_kernel<T, 1>, wgrid, dim3(256), 0, st, a);
  if (e != cudaSuccess) return (int)e;
  // the vectors of a token are read from shared memory by every warp, whatever its rows: four rows per thread, unless that leaves SMs idle
  const bool wide = (long long)a.H * a.Dv * a.B > 148ll * 64;
#define NE_SCAN(CPL_) (wide ? gd_scan<CPL_, 4>(a, st) : gd_scan<CPL_, 2>(a, st))
  int rc;
  if (a.Dk <= 32) rc = NE_SCAN(4);
  else if (a.Dk <= 64) rc = NE_SCAN(8);
  else if (a.Dk <= 96) rc = NE_SCAN(12);
  else if (a.Dk <= 128) rc = NE_SCAN(16);
  else if (a.Dk <= 192) rc = gd_scan<24, 2>(a, st);
  else if (a.Dk <= 256) rc = gd_scan<32, 2>(a, st);
  else rc = gd_scan<64, 1>(a, st);
#undef NE_SCAN
  if (rc) return rc;
  return (int)launch_pdl(fours ? general_delta_norm_kernel<T, 4> : general_delta_norm_kernel<T, 1>, wgrid, dim3(256), 0, st, a);
}

}  // namespace ne

using namespace ne;

// fp32 elements of scratch a call needs (none for single-token steps whose heads fit a CTA)
extern "C" long long ne_general_delta_scratch(int T, int H, int Dk, int Dv, int max_q) {
  if (gd_whole(Dk, Dv, max_q)) return 0;
  return (long long)T * H * (4 * gd_padded(Dk) + (Dv + 3) / 4 * 4 + 4);
}

extern "C" int ne_general_delta(const void* proj, long long proj_ld, const float* decay, long long decay_ld, const float* w0, const float* a_bias, const void* norm_w,
                                float eps, float* state, const int* slots, const int* cu, const int* fresh, float* scratch, void* out, int T, int B, int H, int Dk,
                                int Dv, int max_q, int fp32, int* launches, cudaStream_t st) {
  if (T <= 0 || B <= 0) return 0;
  if (H < 1 || Dk < 1 || Dk > 512 || Dv < 1 || B > 65535 || max_q < 1) return 1001;
  const bool whole = gd_whole(Dk, Dv, max_q);
  if (!whole && (!scratch || ((uintptr_t)scratch & 15))) return 1002;
  GdArgs a;
  a.proj = proj; a.proj_ld = proj_ld; a.decay = decay; a.decay_ld = decay_ld; a.w0 = w0; a.a_bias = a_bias; a.norm_w = norm_w; a.eps = eps; a.state = state;
  a.slots = slots; a.cu = cu; a.fresh = fresh; a.out = out; a.T = T; a.B = B; a.H = H; a.Dk = Dk; a.Dv = Dv; a.DkP = gd_padded(Dk); a.DvP = (Dv + 3) / 4 * 4;
  const long long th = (long long)T * H;
  a.vec = scratch; a.val = whole ? nullptr : a.vec + th * 4 * a.DkP; a.scal = whole ? nullptr : a.val + th * a.DvP;
  *launches = whole ? 1 : 3;
  return fp32 ? general_delta_t<float>(a, max_q, st) : general_delta_t<__nv_bfloat16>(a, max_q, st);
}
