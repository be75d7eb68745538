// Row operators around a 32-bit residual stream, for bf16 and fp32 activations and any row width:
//   * residual_norm: x += rmsnorm(y, w_post); out = rmsnorm(x, w_next)   (norm after a sublayer, residual add, norm before the next)
//     or, as the start of the stream, x = table[id]; out = rmsnorm(x, w_next)
//   * postnorm: x <- rmsnorm(alpha x + y, w); out = x, or rmsnorm(x, w_last) in front of the head; or, as the start, x = scale * table[id]
//   * gated activation of [gate | up] rows
//   * latent_prepare: rotary part of every query head in place, and the latent cache row [rmsnorm(kv[:R]) | rope(kv[R:])]
//   * gather of cache rows
//   * stream_mix: constant hyper-connections - the streams of a token mixed with a sublayer's output, the next sublayer's normed input
//   * depth_mix: the sum behind a sublayer, behind a layer the weighted sum of all layers' results so far, and the next norm (one number as weight)
//   * poly_norm: weighted sum of the normed first three powers of a row
//   * kv_rows: new key and value rows of any width into paged caches;  cap_rows: cap * tanh(x / cap) in place
#include "ptx.cuh"

namespace ne {

template <typename T> struct Vec4;
template <> struct Vec4<float> {
  static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
  static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Vec4<__nv_bfloat16> {
  static __device__ __forceinline__ float4 load(const __nv_bfloat16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
    return make_float4(a.x, a.y, b.x, b.y);
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
  }
};
__device__ __forceinline__ float ldx(const float* p) { return *p; }
__device__ __forceinline__ float ldx(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void stx(float* p, float v) { *p = v; }
__device__ __forceinline__ void stx(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// sum over the CTA; `red` holds two rows of partial sums used in turn, so one barrier per call is enough
__device__ __forceinline__ float cta_sum(float v, float (*red)[32], int turn) {
  v = warp_sum(v);
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (l == 0) red[turn][w] = v;
  __syncthreads();
  return warp_sum(l < nw ? red[turn][l] : 0.f);
}

// One CTA per row.  V = 4: W, the row strides and the base addresses allow 4-element accesses; V = 1: anything.
template <typename T, int V>
__global__ void __launch_bounds__(512) residual_norm_kernel(const T* __restrict__ y, long long y_ld, float* __restrict__ x, const T* __restrict__ w_post,
                                                           const T* __restrict__ w_next, T* __restrict__ out, int W, float eps, float w_off,
                                                           const long long* __restrict__ ids, const T* __restrict__ table, int vocab) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  extern __shared__ float srow[];            // W floats
  __shared__ float red[2][32];
  const long long row = blockIdx.x;
  float* xr = x + row * W;
  float ss = 0.f;
  if (ids) {
    const long long id = ids[row];
    const bool ok = id >= 0 && id < vocab;
    if (!ok && threadIdx.x == 0) report(ST_BAD_INDEX, 40, (int)row, (int)id);
    for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
      if constexpr (V == 4) {
        const float4 t = ok ? Vec4<T>::load(table + id * W + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        *reinterpret_cast<float4*>(srow + i) = t;
        *reinterpret_cast<float4*>(xr + i) = t;
        ss += t.x * t.x + t.y * t.y + t.z * t.z + t.w * t.w;
      } else {
        const float t = ok ? ldx(table + id * W + i) : 0.f;
        srow[i] = t; xr[i] = t; ss += t * t;
      }
    }
  } else {
    const T* yr = y + row * y_ld;
    float sy = 0.f;
    for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
      if constexpr (V == 4) {
        const float4 t = Vec4<T>::load(yr + i);
        *reinterpret_cast<float4*>(srow + i) = t;
        sy += t.x * t.x + t.y * t.y + t.z * t.z + t.w * t.w;
      } else {
        const float t = ldx(yr + i);
        srow[i] = t; sy += t * t;
      }
    }
    const float r = rsqrtf(cta_sum(sy, red, 0) / (float)W + eps);
    for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {      // a thread rereads only what it stored itself
      if constexpr (V == 4) {
        const float4 t = *reinterpret_cast<const float4*>(srow + i), w = Vec4<T>::load(w_post + i);
        float4 v = *reinterpret_cast<const float4*>(xr + i);
        v.x += t.x * r * (w.x + w_off); v.y += t.y * r * (w.y + w_off); v.z += t.z * r * (w.z + w_off); v.w += t.w * r * (w.w + w_off);
        *reinterpret_cast<float4*>(srow + i) = v;
        *reinterpret_cast<float4*>(xr + i) = v;
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      } else {
        const float v = xr[i] + srow[i] * r * (ldx(w_post + i) + w_off);
        srow[i] = v; xr[i] = v; ss += v * v;
      }
    }
  }
  const float r2 = rsqrtf(cta_sum(ss, red, 1) / (float)W + eps);
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    if constexpr (V == 4) {
      const float4 v = *reinterpret_cast<const float4*>(srow + i), w = Vec4<T>::load(w_next + i);
      Vec4<T>::store(out + row * W + i, make_float4(v.x * r2 * (w.x + w_off), v.y * r2 * (w.y + w_off), v.z * r2 * (w.z + w_off), v.w * r2 * (w.w + w_off)));
    } else {
      stx(out + row * W + i, srow[i] * r2 * (ldx(w_next + i) + w_off));
    }
  }
}

// One CTA per row, the row in shared memory between the passes.  ids given: x = alpha table[id], out = x.
struct PostnormArgs {
  const void* y; long long y_ld; float* x; const void* w; const void* w_last; void* out; const long long* ids; const void* table; int W, vocab; float alpha, eps;
};
template <typename T, int V>
__global__ void __launch_bounds__(512) postnorm_kernel(const PostnormArgs a) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  extern __shared__ float srow[];            // W floats
  __shared__ float red[2][32];
  const long long row = blockIdx.x;
  const int W = a.W;
  float* xr = a.x + row * W;
  T* out = reinterpret_cast<T*>(a.out) + row * W;
  if (a.ids) {
    const long long id = a.ids[row];
    const bool ok = id >= 0 && id < a.vocab;
    if (!ok && threadIdx.x == 0) report(ST_BAD_INDEX, 47, (int)row, (int)id);
    const T* tr = reinterpret_cast<const T*>(a.table) + (ok ? id : 0) * W;
    for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
      if constexpr (V == 4) {
        float4 t = Vec4<T>::load(tr + i);
        t.x *= a.alpha; t.y *= a.alpha; t.z *= a.alpha; t.w *= a.alpha;
        *reinterpret_cast<float4*>(xr + i) = t;
        Vec4<T>::store(out + i, t);
      } else {
        const float t = ldx(tr + i) * a.alpha;
        xr[i] = t; stx(out + i, t);
      }
    }
    return;
  }
  const T* yr = reinterpret_cast<const T*>(a.y) + row * a.y_ld;
  const T* w = reinterpret_cast<const T*>(a.w);
  const T* wl = reinterpret_cast<const T*>(a.w_last);
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    if constexpr (V == 4) {
      const float4 t = Vec4<T>::load(yr + i);
      float4 v = *reinterpret_cast<const float4*>(xr + i);
      v.x = fmaf(a.alpha, v.x, t.x); v.y = fmaf(a.alpha, v.y, t.y); v.z = fmaf(a.alpha, v.z, t.z); v.w = fmaf(a.alpha, v.w, t.w);
      *reinterpret_cast<float4*>(srow + i) = v;
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    } else {
      const float v = fmaf(a.alpha, xr[i], ldx(yr + i));
      srow[i] = v; ss += v * v;
    }
  }
  const float r = rsqrtf(cta_sum(ss, red, 0) / (float)W + a.eps);
  float s2 = 0.f;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {        // a thread rereads only what it stored itself
    if constexpr (V == 4) {
      float4 v = *reinterpret_cast<const float4*>(srow + i);
      const float4 g = Vec4<T>::load(w + i);
      v.x *= r * g.x; v.y *= r * g.y; v.z *= r * g.z; v.w *= r * g.w;
      *reinterpret_cast<float4*>(xr + i) = v;
      if (wl) { *reinterpret_cast<float4*>(srow + i) = v; s2 += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
      else Vec4<T>::store(out + i, v);
    } else {
      const float v = srow[i] * r * ldx(w + i);
      xr[i] = v;
      if (wl) { srow[i] = v; s2 += v * v; } else stx(out + i, v);
    }
  }
  if (!wl) return;
  const float r2 = rsqrtf(cta_sum(s2, red, 1) / (float)W + a.eps);
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    if constexpr (V == 4) {
      const float4 v = *reinterpret_cast<const float4*>(srow + i), g = Vec4<T>::load(wl + i);
      Vec4<T>::store(out + i, make_float4(v.x * r2 * g.x, v.y * r2 * g.y, v.z * r2 * g.z, v.w * r2 * g.w));
    } else {
      stx(out + i, srow[i] * r2 * ldx(wl + i));
    }
  }
}

template <typename T>
static int postnorm_t(const PostnormArgs& a, int rows, cudaStream_t st) {
  const size_t smem = (size_t)a.W * sizeof(float);
  const uintptr_t al = (uintptr_t)a.y | (uintptr_t)a.x | (uintptr_t)a.w | (uintptr_t)a.w_last | (uintptr_t)a.out | (uintptr_t)a.table;
  const bool vec = a.W % 4 == 0 && a.y_ld % 4 == 0 && al % 16 == 0;
  const int per = vec ? 4 : 1;
  int threads = ((a.W + per - 1) / per + 31) / 32 * 32;
  threads = threads > 512 ? 512 : threads;
  auto k = vec ? postnorm_kernel<T, 4> : postnorm_kernel<T, 1>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)launch_pdl(k, dim3((unsigned)rows), dim3((unsigned)threads), smem, st, a);
}

// Gated activation (see elementwise.cu for the modes): x [T, >= 2I] rows with stride ld -> y [T, I]
__device__ __forceinline__ float glu_exact(float g, float u, int act, float p0, float p1) {
  if (act == 3) return 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
  if (act == 4) { g = fminf(g, p0); return g / (1.f + expf(-p1 * g)) * (fminf(fmaxf(u, -p0), p0) + 1.f); }
  if (act == 1) { u = fminf(fmaxf(u, -p0), p0); g = fminf(g, p0); }
  if (act == 2) {
    if (p1 > 0.f) u = p1 * tanhf(u / p1);
    return p0 * tanhf(g / p0) / (1.f + expf(-g)) * u;
  }
  return g / (1.f + expf(-g)) * u;
}
template <typename T, int V>
__global__ void __launch_bounds__(256) glu_rows_kernel(const T* __restrict__ x, long long ld, T* __restrict__ y, long long n, int I, int act, float p0, float p1) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (i >= n) return;
  const long long t = i / I;
  const int c = (int)(i - t * I);
  const T* g = x + t * ld + c;
  if constexpr (V == 4) {
    const float4 a = Vec4<T>::load(g), b = Vec4<T>::load(g + I);
    Vec4<T>::store(y + i, make_float4(glu_exact(a.x, b.x, act, p0, p1), glu_exact(a.y, b.y, act, p0, p1), glu_exact(a.z, b.z, act, p0, p1),
                                      glu_exact(a.w, b.w, act, p0, p1)));
  } else {
    stx(y + i, glu_exact(ldx(g), ldx(g + I), act, p0, p1));
  }
}

__device__ __forceinline__ float2 ldx2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 ldx2(const __nv_bfloat16* p) { return unpack_bf16x2(*reinterpret_cast<const uint32_t*>(p)); }
__device__ __forceinline__ void stx2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void stx2(__nv_bfloat16* p, float a, float b) { *reinterpret_cast<uint32_t*>(p) = pack_bf16x2(a, b); }

// One warp per (token, unit): unit 0 .. H-1 rotates the rotary tail of that query head (q -> dst), unit H (when kv is given) writes the
// token's cache row.  kv_kind: 0 bf16 rows, 1 e4m3 rows (clamped cast of the bf16 value), 2 fp32 rows.
// kPairs: R, the strides and the addresses allow two elements per access.
template <typename T, bool kPairs>
__global__ void __launch_bounds__(256) latent_prepare_kernel(const T* q, long long q_ld, int q_hs, T* dst, long long d_ld, int d_hs, int H, const T* __restrict__ kv,
                                                            long long kv_ld, const T* __restrict__ w, float eps, const long long* __restrict__ positions,
                                                            const float* __restrict__ rope_cache, void* __restrict__ cache,
                                                            const long long* __restrict__ slots, int T_, int R, int rope, int kv_kind) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const int units = H + (kv ? 1 : 0), lane = threadIdx.x & 31, half = rope / 2;
  const long long wid = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (wid >= (long long)T_ * units) return;
  const int t = (int)(wid / units), u = (int)(wid % units);
  const float* cs = rope_cache + positions[t] * rope;
  if (u < H) {
    const T* p = q + (long long)t * q_ld + (long long)u * q_hs;        // may be the destination itself
    T* o = dst + (long long)t * d_ld + (long long)u * d_hs;
    for (int i = lane; i < half; i += 32) {
      const float c = cs[i], s = cs[half + i];
      if constexpr (kPairs) {
        const float2 v = ldx2(p + 2 * i);
        stx2(o + 2 * i, v.x * c - v.y * s, v.y * c + v.x * s);
      } else {
        const float a = ldx(p + 2 * i), b = ldx(p + 2 * i + 1);
        stx(o + 2 * i, a * c - b * s);
        stx(o + 2 * i + 1, b * c + a * s);
      }
    }
    return;
  }
  const long long slot = slots[t];
  if (slot < 0 || !NE_INDEX_OK(slot, BK_CACHE_ROWS, 41, __LINE__)) return;
  const T* row = kv + (long long)t * kv_ld;
  float ss = 0.f;
  if constexpr (kPairs) { for (int c = lane * 2; c < R; c += 64) { const float2 f = ldx2(row + c); ss += f.x * f.x + f.y * f.y; } }
  else { for (int c = lane; c < R; c += 32) { const float f = ldx(row + c); ss += f * f; } }
  const float r = rsqrtf(warp_sum(ss) / (float)R + eps);
  auto put = [&](int c, float v) {
    const long long o = slot * (R + rope) + c;
    if (kv_kind == 2) reinterpret_cast<float*>(cache)[o] = v;
    else if (kv_kind == 1) reinterpret_cast<uint8_t*>(cache)[o] = to_e4m3(__bfloat162float(__float2bfloat16(v)));
    else reinterpret_cast<__nv_bfloat16*>(cache)[o] = __float2bfloat16(v);
  };
  if (kPairs && kv_kind != 1) {
    T* dst = reinterpret_cast<T*>(cache) + slot * (R + rope);
    for (int c = lane * 2; c < R; c += 64) {
      const float2 f = ldx2(row + c), g = ldx2(w + c);
      stx2(dst + c, f.x * r * g.x, f.y * r * g.y);
    }
    for (int i = lane; i < half; i += 32) {
      const float2 v = ldx2(row + R + 2 * i);
      const float c = cs[i], s = cs[half + i];
      stx2(dst + R + 2 * i, v.x * c - v.y * s, v.y * c + v.x * s);
    }
    return;
  }
  for (int c = lane; c < R; c += 32) put(c, ldx(row + c) * r * ldx(w + c));
  for (int i = lane; i < half; i += 32) {
    const float a = ldx(row + R + 2 * i), b = ldx(row + R + 2 * i + 1), c = cs[i], s = cs[half + i];
    put(R + 2 * i, a * c - b * s);
    put(R + 2 * i + 1, b * c + a * s);
  }
}

// rows[t] = cache[slots[t]] (slot -1: row 0); 16-byte pieces
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4* __restrict__ cache, const long long* __restrict__ slots, uint4* __restrict__ rows,
                                                           int T, int pieces) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (long long)T * pieces) return;
  const int t = (int)(i / pieces), c = (int)(i % pieces);
  long long slot = slots[t];
  if (slot < 0 || !NE_INDEX_OK(slot, BK_CACHE_ROWS, 42, __LINE__)) slot = 0;
  rows[i] = cache[slot * pieces + c];
}

// ---- constant hyper-connections -----------------------------------------------------------------------------------------
// x [rows, S, W] fp32 streams.  y given: x_t <- sum_s mix[s, t] x_s + w_out[t] y (all streams from the old ones, written back unless
// `last`).  ids given: every stream starts as table[id] + pos[position] instead.  Then u = sum_s w_in[s] x_s and out = rmsnorm(u) * w_next.
// One CTA per row; S = 0: any number of streams up to kMaxStreams (then V = 1).
constexpr int kMaxStreams = 16;
struct StreamArgs {
  const void* y; long long y_ld; float* x; const float* w_out; const float* mix; const float* w_in; const void* w_next; void* out;
  const long long* ids; const long long* positions; const void* table; const void* pos;
  int streams, W, vocab, n_pos, last; float eps;
};
template <typename T, int V, int S>
__global__ void __launch_bounds__(512) stream_mix_kernel(const StreamArgs a) {
  constexpr int SM = S ? S : kMaxStreams;
  extern __shared__ float srow[];            // W floats: u
  __shared__ float red[2][32];
  __shared__ float s_in[SM], s_out[SM], s_mix[SM * SM];
  const int ns = S ? S : a.streams, W = a.W;
  // the coefficients are weights: they may be read before the kernel in front has finished
  for (int i = threadIdx.x; i < ns; i += blockDim.x) { s_in[i] = a.w_in[i]; if (a.y) s_out[i] = a.w_out[i]; }
  if (a.y) for (int i = threadIdx.x; i < ns * ns; i += blockDim.x) s_mix[i] = a.mix[i];
  pdl_wait(); pdl_trigger();
  __syncthreads();
  const long long row = blockIdx.x;
  float* xr = a.x + row * ns * W;
  float ss = 0.f;
  if (a.ids) {
    const long long id = a.ids[row], p = a.positions[row];
    const bool ok = id >= 0 && id < a.vocab && (!a.pos || (p >= 0 && p < a.n_pos));
    if (!ok && threadIdx.x == 0) report(ST_BAD_INDEX, 45, (int)id, (int)p);
    const T* tr = reinterpret_cast<const T*>(a.table) + (ok ? id : 0) * W;
    const T* pr = a.pos ? reinterpret_cast<const T*>(a.pos) + (ok ? p : 0) * W : nullptr;
    float wsum = 0.f;
    for (int s = 0; s < ns; s++) wsum += s_in[s];
    for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
      if constexpr (V == 4) {
        float4 t = Vec4<T>::load(tr + i);
        if (pr) { const float4 q = Vec4<T>::load(pr + i); t.x += q.x; t.y += q.y; t.z += q.z; t.w += q.w; }
        for (int s = 0; s < ns; s++) *reinterpret_cast<float4*>(xr + (long long)s * W + i) = t;
        t.x *= wsum; t.y *= wsum; t.z *= wsum; t.w *= wsum;
        *reinterpret_cast<float4*>(srow + i) = t;
        ss += t.x * t.x + t.y * t.y + t.z * t.z + t.w * t.w;
      } else {
        float t = ldx(tr + i);
        if (pr) t += ldx(pr + i);
        for (int s = 0; s < ns; s++) xr[(long long)s * W + i] = t;
        t *= wsum;
        srow[i] = t; ss += t * t;
      }
    }
  } else {
    const T* yr = reinterpret_cast<const T*>(a.y) + row * a.y_ld;
    for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
      float xs[SM][V], yv[V], u[V];
#pragma unroll
      for (int s = 0; s < SM; s++) {
        if (!S && s >= ns) break;
        if constexpr (V == 4) {
          const float4 t = *reinterpret_cast<const float4*>(xr + (long long)s * W + i);
          xs[s][0] = t.x; xs[s][1] = t.y; xs[s][2] = t.z; xs[s][3] = t.w;
        } else xs[s][0] = xr[(long long)s * W + i];
      }
      if constexpr (V == 4) { const float4 t = Vec4<T>::load(yr + i); yv[0] = t.x; yv[1] = t.y; yv[2] = t.z; yv[3] = t.w; }
      else yv[0] = ldx(yr + i);
#pragma unroll
      for (int e = 0; e < V; e++) u[e] = 0.f;
#pragma unroll (S ? SM : 1)
      for (int t = 0; t < SM; t++) {
        if (!S && t >= ns) break;
        float n[V];
#pragma unroll
        for (int e = 0; e < V; e++) n[e] = s_out[t] * yv[e];
#pragma unroll
        for (int s = 0; s < SM; s++) {
          if (!S && s >= ns) break;
          const float m = s_mix[s * ns + t];
#pragma unroll
          for (int e = 0; e < V; e++) n[e] = fmaf(m, xs[s][e], n[e]);
        }
        const float wi = s_in[t];
#pragma unroll
        for (int e = 0; e < V; e++) u[e] = fmaf(wi, n[e], u[e]);
        if (!a.last) {
          if constexpr (V == 4) *reinterpret_cast<float4*>(xr + (long long)t * W + i) = make_float4(n[0], n[1], n[2], n[3]);
          else xr[(long long)t * W + i] = n[0];
        }
      }
#pragma unroll
      for (int e = 0; e < V; e++) { srow[i + e] = u[e]; ss += u[e] * u[e]; }
    }
  }
  const float r = rsqrtf(cta_sum(ss, red, 0) / (float)W + a.eps);
  const T* wn = reinterpret_cast<const T*>(a.w_next);
  T* out = reinterpret_cast<T*>(a.out) + row * W;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {        // a thread rereads only what it stored itself
    if constexpr (V == 4) {
      const float4 v = *reinterpret_cast<const float4*>(srow + i), w = Vec4<T>::load(wn + i);
      Vec4<T>::store(out + i, make_float4(v.x * r * w.x, v.y * r * w.y, v.z * r * w.z, v.w * r * w.w));
    } else {
      stx(out + i, srow[i] * r * ldx(wn + i));
    }
  }
}

template <typename T>
static int stream_mix_t(const StreamArgs& a, int rows, cudaStream_t st) {
  const size_t smem = (size_t)a.W * sizeof(float);
  const uintptr_t al = (uintptr_t)a.y | (uintptr_t)a.x | (uintptr_t)a.w_next | (uintptr_t)a.out | (uintptr_t)a.table | (uintptr_t)a.pos;
  const bool vec = a.W % 4 == 0 && a.y_ld % 4 == 0 && al % 16 == 0 && a.streams <= 4;
  const int per = vec ? 4 : 1;
  int threads = ((a.W + per - 1) / per + 31) / 32 * 32;
  threads = threads > 512 ? 512 : threads;
  void (*k)(const StreamArgs) = stream_mix_kernel<T, 1, 0>;
  if (vec) k = a.streams == 1 ? stream_mix_kernel<T, 4, 1> : a.streams == 2 ? stream_mix_kernel<T, 4, 2> : a.streams == 3 ? stream_mix_kernel<T, 4, 3> : stream_mix_kernel<T, 4, 4>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)launch_pdl(k, dim3((unsigned)rows), dim3((unsigned)threads), smem, st, a);
}

// ---- averages over the depth ------------------------------------------------------------------------------------------------
// v = x + y (ids given: v = table[id], at = 0).  With a bank of [.., rows, W] fp32: bank[at] = v and, behind a layer (w given), v = sum_{j <= at} w[j] bank[j].
// x = v, out = rmsnorm(v) * g.  `last`: neither x nor the bank is written.  One CTA per row.
struct DepthArgs {
  const void* y; long long y_ld; float* x; float* bank; long long bank_ld; const float* w; const float* g; void* out; const long long* ids; const void* table;
  int at, W, vocab, last; float eps;
};
template <typename T, int V, bool kMix>
__global__ void __launch_bounds__(512, kMix ? 2 : 3) depth_mix_kernel(const DepthArgs a) {
  extern __shared__ float srow[];            // W floats, then at + 1 weights
  __shared__ float red[2][32];
  const int W = a.W;
  float* sw = srow + (W + 3) / 4 * 4;
  // the coefficients are weights: they may be read before the kernel in front has finished
  if (kMix) for (int j = threadIdx.x; j <= a.at; j += blockDim.x) sw[j] = a.w[j];
  const float g = *a.g;
  pdl_wait(); pdl_trigger();
  if (kMix) __syncthreads();
  const long long row = blockIdx.x;
  float* xr = a.x + row * W;
  float* br = a.bank ? a.bank + row * W : nullptr;
  const T* yr = nullptr;
  bool ok = true;
  if (a.ids) {
    const long long id = a.ids[row];
    ok = id >= 0 && id < a.vocab;
    if (!ok && threadIdx.x == 0) report(ST_BAD_INDEX, 49, (int)row, (int)id);
    yr = reinterpret_cast<const T*>(a.table) + (ok ? id : 0) * W;
  } else {
    yr = reinterpret_cast<const T*>(a.y) + row * a.y_ld;
  }
  float ss = 0.f;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {
    float v[V];
    if constexpr (V == 4) { const float4 t = Vec4<T>::load(yr + i); v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w; }
    else v[0] = ldx(yr + i);
    if (a.ids) {
      if (!ok) for (int e = 0; e < V; e++) v[e] = 0.f;
    } else if constexpr (V == 4) {
      const float4 t = *reinterpret_cast<const float4*>(xr + i);
      v[0] += t.x; v[1] += t.y; v[2] += t.z; v[3] += t.w;
    } else v[0] += xr[i];
    if (br && !a.last) {
      if constexpr (V == 4) *reinterpret_cast<float4*>(br + a.at * a.bank_ld + i) = make_float4(v[0], v[1], v[2], v[3]);
      else br[a.at * a.bank_ld + i] = v[0];
    }
    if constexpr (kMix) {
      const float wn = sw[a.at];
#pragma unroll
      for (int e = 0; e < V; e++) v[e] *= wn;
#pragma unroll 4
      for (int j = 0; j < a.at; j++) {
        const float wj = sw[j];
        if constexpr (V == 4) {
          const float4 t = __ldcs(reinterpret_cast<const float4*>(br + j * a.bank_ld + i));
          v[0] = fmaf(wj, t.x, v[0]); v[1] = fmaf(wj, t.y, v[1]); v[2] = fmaf(wj, t.z, v[2]); v[3] = fmaf(wj, t.w, v[3]);
        } else v[0] = fmaf(wj, br[j * a.bank_ld + i], v[0]);
      }
    }
    if constexpr (V == 4) {
      const float4 t = make_float4(v[0], v[1], v[2], v[3]);
      if (!a.last) *reinterpret_cast<float4*>(xr + i) = t;
      *reinterpret_cast<float4*>(srow + i) = t;
    } else { if (!a.last) xr[i] = v[0]; srow[i] = v[0]; }
#pragma unroll
    for (int e = 0; e < V; e++) ss += v[e] * v[e];
  }
  const float r = rsqrtf(cta_sum(ss, red, 0) / (float)W + a.eps) * g;
  T* out = reinterpret_cast<T*>(a.out) + row * W;
  for (int i = threadIdx.x * V; i < W; i += blockDim.x * V) {        // a thread rereads only what it stored itself
    if constexpr (V == 4) {
      const float4 v = *reinterpret_cast<const float4*>(srow + i);
      Vec4<T>::store(out + i, make_float4(v.x * r, v.y * r, v.z * r, v.w * r));
    } else stx(out + i, srow[i] * r);
  }
}

template <typename T>
static int depth_mix_t(const DepthArgs& a, int rows, cudaStream_t st) {
  const size_t smem = ((size_t)(a.W + 3) / 4 * 4 + (a.w ? a.at + 1 : 0)) * sizeof(float);
  const uintptr_t al = (uintptr_t)a.y | (uintptr_t)a.x | (uintptr_t)a.out | (uintptr_t)a.table | (uintptr_t)a.bank;
  const bool vec = a.W % 4 == 0 && a.y_ld % 4 == 0 && al % 16 == 0;
  const int per = vec ? 4 : 1;
  int threads = ((a.W + per - 1) / per + 31) / 32 * 32;
  threads = threads > 512 ? 512 : threads;
  auto k = a.w ? (vec ? depth_mix_kernel<T, 4, true> : depth_mix_kernel<T, 1, true>) : vec ? depth_mix_kernel<T, 4, false> : depth_mix_kernel<T, 1, false>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)launch_pdl(k, dim3((unsigned)rows), dim3((unsigned)threads), smem, st, a);
}

// ---- normed powers ------------------------------------------------------------------------------------------------------------
// out = a z / rms(z) + b z^2 / rms(z^2) + c z^3 / rms(z^3) + e over rows of F; coef = (a, b, c, e).  One CTA per row, the row in shared memory.
template <typename T, int V>
__global__ void __launch_bounds__(512) poly_norm_kernel(const T* __restrict__ z, long long ld, T* __restrict__ out, int F, const float* __restrict__ coef, float eps) {
  extern __shared__ float srow[];            // F floats
  __shared__ float red[3][32];
  const float ca = coef[0], cb = coef[1], cc = coef[2], ce = coef[3];      // weights: they may be read before the kernel in front has finished
  pdl_wait(); pdl_trigger();
  const long long row = blockIdx.x;
  const T* zr = z + row * ld;
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  auto add = [&](float v) { const float p = v * v; s2 += p; s4 = fmaf(p, p, s4); s6 = fmaf(p * p, p, s6); };
  for (int i = threadIdx.x * V; i < F; i += blockDim.x * V) {
    if constexpr (V == 4) {
      const float4 t = Vec4<T>::load(zr + i);
      *reinterpret_cast<float4*>(srow + i) = t;
      add(t.x); add(t.y); add(t.z); add(t.w);
    } else { const float t = ldx(zr + i); srow[i] = t; add(t); }
  }
  const int w = threadIdx.x >> 5, l = threadIdx.x & 31, nw = blockDim.x >> 5;
  s2 = warp_sum(s2); s4 = warp_sum(s4); s6 = warp_sum(s6);
  if (l == 0) { red[0][w] = s2; red[1][w] = s4; red[2][w] = s6; }
  __syncthreads();
  const float n = (float)F;
  const float r1 = ca * rsqrtf(warp_sum(l < nw ? red[0][l] : 0.f) / n + eps), r2 = cb * rsqrtf(warp_sum(l < nw ? red[1][l] : 0.f) / n + eps),
              r3 = cc * rsqrtf(warp_sum(l < nw ? red[2][l] : 0.f) / n + eps);
  auto f = [&](float v) { return fmaf(v, fmaf(v, fmaf(v, r3, r2), r1), ce); };
  T* o = out + row * F;
  for (int i = threadIdx.x * V; i < F; i += blockDim.x * V) {        // a thread rereads only what it stored itself
    if constexpr (V == 4) {
      const float4 t = *reinterpret_cast<const float4*>(srow + i);
      Vec4<T>::store(o + i, make_float4(f(t.x), f(t.y), f(t.z), f(t.w)));
    } else stx(o + i, f(srow[i]));
  }
}

template <typename T>
static int poly_norm_t(const void* z, long long ld, void* out, int rows, int F, const float* coef, float eps, cudaStream_t st) {
  const size_t smem = (size_t)F * sizeof(float);
  const bool vec = F % 4 == 0 && ld % 4 == 0 && ((uintptr_t)z | (uintptr_t)out) % 16 == 0;
  const int per = vec ? 4 : 1;
  int threads = ((F + per - 1) / per + 31) / 32 * 32;
  threads = threads > 512 ? 512 : threads;
  auto k = vec ? poly_norm_kernel<T, 4> : poly_norm_kernel<T, 1>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)launch_pdl(k, dim3((unsigned)rows), dim3((unsigned)threads), smem, st, (const T*)z, ld, (T*)out, F, coef, eps);
}

// Gated activation of the valid rows of an expert-major layout: rows [row_start[g], row_start[g] + counts[g]) of x [rows, 2I] -> y [rows, I].
// blockIdx.x: a row; rows of no group are left as they are.
template <typename T, int V>
__global__ void __launch_bounds__(128) glu_groups_kernel(const T* __restrict__ x, T* __restrict__ y, const int* __restrict__ counts, const int* __restrict__ row_start,
                                                         int groups, int I, int act, float p0, float p1) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const int row = blockIdx.x;
  if (row >= row_start[groups]) return;
  int lo = 0, hi = groups - 1;              // the last group that starts at or before the row
  while (lo < hi) { const int mid = (lo + hi + 1) >> 1; if (row_start[mid] <= row) lo = mid; else hi = mid - 1; }
  if (row >= row_start[lo] + counts[lo]) return;
  const T* g = x + (long long)row * 2 * I;
  T* o = y + (long long)row * I;
  for (int c = threadIdx.x * V; c < I; c += 128 * V) {
    if constexpr (V == 4) {
      const float4 a = Vec4<T>::load(g + c), b = Vec4<T>::load(g + I + c);
      Vec4<T>::store(o + c, make_float4(glu_exact(a.x, b.x, act, p0, p1), glu_exact(a.y, b.y, act, p0, p1), glu_exact(a.z, b.z, act, p0, p1),
                                        glu_exact(a.w, b.w, act, p0, p1)));
    } else stx(o + c, glu_exact(ldx(g + c), ldx(g + I + c), act, p0, p1));
  }
}

template <typename T>
static int glu_groups_t(const void* x, void* y, const int* counts, const int* row_start, int groups, int rows, int I, int act, float p0, float p1, cudaStream_t st) {
  const bool vec = I % 4 == 0 && ((uintptr_t)x | (uintptr_t)y) % 16 == 0;
  return (int)launch_pdl(vec ? glu_groups_kernel<T, 4> : glu_groups_kernel<T, 1>, dim3((unsigned)rows), dim3(128), 0, st, (const T*)x, (T*)y, counts, row_start, groups, I,
                         act, p0, p1);
}

// ---- key / value rows into paged caches -------------------------------------------------------------------------------------
// Row t of k (kw elements, row stride k_ld) goes to cache row slots[t], the same for v.  U: the access unit (uint4 where everything is
// 16-byte aligned, else one element); widths and strides in units.
template <typename U>
__global__ void __launch_bounds__(256) kv_rows_kernel(const U* __restrict__ k, long long k_ld, const U* __restrict__ v, long long v_ld, U* __restrict__ kc, U* __restrict__ vc,
                                                     const long long* __restrict__ slots, int T, int kw, int vw) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  const int w = kw + vw;
  if (i >= (long long)T * w) return;
  const int t = (int)(i / w), c = (int)(i - (long long)t * w);
  const long long slot = slots[t];
  if (slot < 0 || !NE_INDEX_OK(slot, BK_CACHE_ROWS, 46, __LINE__)) return;
  if (c < kw) kc[slot * kw + c] = k[(long long)t * k_ld + c];
  else vc[slot * vw + c - kw] = v[(long long)t * v_ld + c - kw];
}

__global__ void __launch_bounds__(256) cap_rows_kernel(float* __restrict__ x, long long n, float cap) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) x[i] = cap * tanhf(x[i] / cap);
}

template <typename T>
static int residual_norm_t(const void* y, long long y_ld, float* x, const void* w_post, const void* w_next, void* out, int T_, int W, float eps,
                           float w_off, const long long* ids, const void* table, int vocab, cudaStream_t st) {
  const size_t smem = (size_t)W * sizeof(float);
  const uintptr_t al = (uintptr_t)y | (uintptr_t)x | (uintptr_t)w_post | (uintptr_t)w_next | (uintptr_t)out | (uintptr_t)table;
  const bool vec = W % 4 == 0 && y_ld % 4 == 0 && al % 16 == 0;
  const int per = vec ? 4 : 1;
  int threads = ((W + per - 1) / per + 31) / 32 * 32;
  threads = threads > 512 ? 512 : threads;
  auto k = vec ? residual_norm_kernel<T, 4> : residual_norm_kernel<T, 1>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)launch_pdl(k, dim3((unsigned)T_), dim3((unsigned)threads), smem, st, (const T*)y, y_ld, x, (const T*)w_post, (const T*)w_next, (T*)out, W, eps,
                         w_off, ids, (const T*)table, vocab);
}

template <typename T>
static int glu_rows_t(const void* x, long long ld, void* y, int T_, int I, int act, float p0, float p1, cudaStream_t st) {
  const bool vec = I % 4 == 0 && ld % 4 == 0 && ((uintptr_t)x | (uintptr_t)y) % 16 == 0;
  const long long n = (long long)T_ * I, items = vec ? n / 4 : n;
  return (int)launch_pdl(vec ? glu_rows_kernel<T, 4> : glu_rows_kernel<T, 1>, dim3((unsigned)((items + 255) / 256)), dim3(256), 0, st, (const T*)x, ld, (T*)y, n,
                         I, act, p0, p1);
}

}  // namespace ne

using namespace ne;

// y [T, W] (row stride y_ld), x [T, W] fp32 updated in place, out [T, W].  With `ids` (and table [vocab, W]) y is not read: x = table[ids].
extern "C" int ne_residual_norm(const void* y, long long y_ld, float* x, const void* w_post, const void* w_next, void* out, int T, int W, float eps,
                                float w_off, const long long* ids, const void* table, int vocab, int fp32, cudaStream_t st) {
  if (T <= 0) return 0;
  if (W <= 0 || W > 48 * 1024 || (!ids && (!y || !w_post)) || (ids && !table)) return 1001;
  return fp32 ? residual_norm_t<float>(y, y_ld, x, w_post, w_next, out, T, W, eps, w_off, ids, table, vocab, st)
              : residual_norm_t<__nv_bfloat16>(y, y_ld, x, w_post, w_next, out, T, W, eps, w_off, ids, table, vocab, st);
}

// y [T, W] (row stride y_ld), x [T, W] fp32 updated in place, out [T, W]; w_last null: out is x itself.  With `ids` (and table [vocab, W]) y and
// the norms are not read: x = out = alpha * table[ids].
extern "C" int ne_postnorm(const void* y, long long y_ld, float* x, float alpha, const void* w, const void* w_last, void* out, int T, int W, float eps,
                           const long long* ids, const void* table, int vocab, int fp32, cudaStream_t st) {
  if (T <= 0) return 0;
  if (W <= 0 || W > 48 * 1024 || (!ids && (!y || !w)) || (ids && !table)) return 1001;
  PostnormArgs a;
  a.y = ids ? nullptr : y; a.y_ld = ids ? 0 : y_ld; a.x = x; a.w = ids ? nullptr : w; a.w_last = ids ? nullptr : w_last; a.out = out; a.ids = ids;
  a.table = ids ? table : nullptr; a.W = W; a.vocab = vocab; a.alpha = alpha; a.eps = eps;
  return fp32 ? postnorm_t<float>(a, T, st) : postnorm_t<__nv_bfloat16>(a, T, st);
}

extern "C" int ne_glu_rows(const void* x, long long ld, void* y, int T, int I, int act, float p0, float p1, int fp32, cudaStream_t st) {
  if (T <= 0 || I <= 0) return 0;
  if (act < 0 || act > 4 || ld < 2 * I) return 1001;
  return fp32 ? glu_rows_t<float>(x, ld, y, T, I, act, p0, p1, st) : glu_rows_t<__nv_bfloat16>(x, ld, y, T, I, act, p0, p1, st);
}

// q [T, H, rope], the rotary tails (row stride q_ld, head stride q_hs, elements), dst the same or another view; kv [T, R + rope] (row
// stride kv_ld) or null
extern "C" int ne_latent_prepare(const void* q, long long q_ld, int q_hs, void* dst, long long d_ld, int d_hs, int H, const void* kv, long long kv_ld, const void* w, float eps,
                                 const long long* positions, const float* rope_cache, void* cache, const long long* slots, int T, int R, int rope,
                                 int kv_kind, int fp32, cudaStream_t st) {
  if (T <= 0) return 0;
  if (rope < 0 || rope % 2 || R <= 0 || kv_kind < 0 || kv_kind > 2 || (fp32 != 0) != (kv_kind == 2)) return 1001;
  const long long warps = (long long)T * (H + (kv ? 1 : 0));
  const dim3 grid((unsigned)((warps + 7) / 8));
  const bool pairs = R % 2 == 0 && q_ld % 2 == 0 && q_hs % 2 == 0 && d_ld % 2 == 0 && d_hs % 2 == 0 && kv_ld % 2 == 0 &&
                     ((uintptr_t)q | (uintptr_t)dst | (uintptr_t)kv | (uintptr_t)w | (uintptr_t)cache) % (fp32 ? 8 : 4) == 0;
  if (fp32)
    return (int)launch_pdl(pairs ? latent_prepare_kernel<float, true> : latent_prepare_kernel<float, false>, grid, dim3(256), 0, st, (const float*)q, q_ld, q_hs,
                           (float*)dst, d_ld, d_hs, H, (const float*)kv, kv_ld, (const float*)w, eps, positions, rope_cache, cache, slots, T, R, rope, kv_kind);
  return (int)launch_pdl(pairs ? latent_prepare_kernel<__nv_bfloat16, true> : latent_prepare_kernel<__nv_bfloat16, false>, grid, dim3(256), 0, st,
                         (const __nv_bfloat16*)q, q_ld, q_hs, (__nv_bfloat16*)dst, d_ld, d_hs, H, (const __nv_bfloat16*)kv, kv_ld, (const __nv_bfloat16*)w, eps,
                         positions, rope_cache, cache, slots, T, R, rope, kv_kind);
}

extern "C" int ne_latent_gather(const void* cache, const long long* slots, void* rows, int T, int row_bytes, cudaStream_t st) {
  if (T <= 0) return 0;
  if (row_bytes % 16) return 1001;
  const int pieces = row_bytes / 16;
  return (int)launch_pdl(latent_gather_kernel, dim3((unsigned)(((long long)T * pieces + 255) / 256)), dim3(256), 0, st, (const uint4*)cache, slots, (uint4*)rows, T,
                         pieces);
}

// See StreamArgs.  w_out [S], mix [S, S] (from, to), w_in [S] fp32; y / table / pos / w_next / out in the activation dtype.
extern "C" int ne_stream_mix(const void* y, long long y_ld, float* x, const float* w_out, const float* mix, const float* w_in, const void* w_next, void* out,
                             const long long* ids, const long long* positions, const void* table, int vocab, const void* pos, int n_pos, int T, int S, int W,
                             float eps, int last, int fp32, cudaStream_t st) {
  if (T <= 0) return 0;
  if (S < 1 || S > kMaxStreams || W < 1 || W > 48 * 1024 || (!ids && (!y || !w_out || !mix)) || (ids && (!table || !positions)) || !w_in) return 1001;
  StreamArgs a;
  a.y = ids ? nullptr : y; a.y_ld = ids ? 0 : y_ld; a.x = x; a.w_out = w_out; a.mix = mix; a.w_in = w_in; a.w_next = w_next; a.out = out; a.ids = ids;
  a.positions = positions; a.table = ids ? table : nullptr; a.pos = ids ? pos : nullptr; a.streams = S; a.W = W; a.vocab = vocab; a.n_pos = n_pos; a.last = last; a.eps = eps;
  return fp32 ? stream_mix_t<float>(a, T, st) : stream_mix_t<__nv_bfloat16>(a, T, st);
}

// k [T, kw], v [T, vw] (row strides k_ld, v_ld, elements of `es` bytes) -> rows slots[t] of caches [rows, kw] and [rows, vw]
extern "C" int ne_kv_rows(const void* k, long long k_ld, const void* v, long long v_ld, void* kc, void* vc, const long long* slots, int T, int kw, int vw, int es,
                          cudaStream_t st) {
  if (T <= 0) return 0;
  if ((es != 2 && es != 4) || kw < 1 || vw < 1) return 1001;
  const int per = 16 / es;
  const bool vec = kw % per == 0 && vw % per == 0 && k_ld % per == 0 && v_ld % per == 0 && ((uintptr_t)k | (uintptr_t)v | (uintptr_t)kc | (uintptr_t)vc) % 16 == 0;
  const long long n = (long long)T * (kw + vw) / (vec ? per : 1);
  const dim3 grid((unsigned)((n + 255) / 256));
  if (vec)
    return (int)launch_pdl(kv_rows_kernel<uint4>, grid, dim3(256), 0, st, (const uint4*)k, k_ld / per, (const uint4*)v, v_ld / per, (uint4*)kc, (uint4*)vc, slots, T,
                           kw / per, vw / per);
  if (es == 2)
    return (int)launch_pdl(kv_rows_kernel<uint16_t>, grid, dim3(256), 0, st, (const uint16_t*)k, k_ld, (const uint16_t*)v, v_ld, (uint16_t*)kc, (uint16_t*)vc, slots, T,
                           kw, vw);
  return (int)launch_pdl(kv_rows_kernel<uint32_t>, grid, dim3(256), 0, st, (const uint32_t*)k, k_ld, (const uint32_t*)v, v_ld, (uint32_t*)kc, (uint32_t*)vc, slots, T, kw,
                         vw);
}

// x [n] fp32 <- cap * tanh(x / cap)
extern "C" int ne_cap_rows(float* x, long long n, float cap, cudaStream_t st) {
  if (n <= 0) return 0;
  if (!(cap > 0.f)) return 1001;
  return (int)launch_pdl(cap_rows_kernel, dim3((unsigned)((n + 255) / 256)), dim3(256), 0, st, x, n, cap);
}

// See DepthArgs.  y [T, W] (row stride y_ld), x [T, W], bank [layers, T, W] or null, w [at + 1] or null (then at is the bank row to fill), g [1] fp32, out [T, W]
extern "C" int ne_depth_mix(const void* y, long long y_ld, float* x, float* bank, int at, const float* w, const float* g, void* out, const long long* ids,
                            const void* table, int vocab, int T, int W, float eps, int last, int fp32, cudaStream_t st) {
  if (T <= 0) return 0;
  if (W <= 0 || W > 48 * 1024 || at < 0 || at > 1024 || !g || (w && !bank) || (!ids && !y) || (ids && (!table || w || last))) return 1001;
  DepthArgs a;
  a.y = ids ? nullptr : y; a.y_ld = ids ? 0 : y_ld; a.x = x; a.bank = bank; a.bank_ld = (long long)T * W; a.w = w; a.g = g; a.out = out; a.ids = ids;
  a.table = ids ? table : nullptr; a.at = at; a.W = W; a.vocab = vocab; a.last = last; a.eps = eps;
  return fp32 ? depth_mix_t<float>(a, T, st) : depth_mix_t<__nv_bfloat16>(a, T, st);
}

// z [T, F] (row stride ld) -> out [T, F]; coef fp32 [4]
extern "C" int ne_poly_norm(const void* z, long long ld, void* out, int T, int F, const float* coef, float eps, int fp32, cudaStream_t st) {
  if (T <= 0) return 0;
  if (F <= 0 || F > 48 * 1024 || ld < F) return 1001;
  return fp32 ? poly_norm_t<float>(z, ld, out, T, F, coef, eps, st) : poly_norm_t<__nv_bfloat16>(z, ld, out, T, F, coef, eps, st);
}

// x [rows, 2I] -> y [rows, I] for the rows of `groups` experts (counts [groups], row_start [groups + 1])
extern "C" int ne_glu_groups(const void* x, void* y, const int* counts, const int* row_start, int groups, int rows, int I, int act, float p0, float p1, int fp32,
                             cudaStream_t st) {
  if (rows <= 0 || I <= 0) return 0;
  if (act < 0 || act > 4 || groups < 1) return 1001;
  return fp32 ? glu_groups_t<float>(x, y, counts, row_start, groups, rows, I, act, p0, p1, st)
              : glu_groups_t<__nv_bfloat16>(x, y, counts, row_start, groups, rows, I, act, p0, p1, st);
}
