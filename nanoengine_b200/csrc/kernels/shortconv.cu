// Short causal convolution over time behind a merged projection: y_t = sum_j w[j] u_{t - taps + 1 + j} on each of C channels, the results of the
// query columns into a buffer, those of the key and value columns straight into their paged caches.  The last taps - 1 inputs of a sequence are
// its state.  bf16 or fp32 rows, fp32 sums.
//
// One CTA = kTile tokens of one sequence x 128 threads of V channels; a thread holds its tokens and the inputs in front of them in registers.  The
// CTA of a sequence's first tokens also writes the sequence's next window: nobody else reads the old one (kTile >= taps - 1 unless every sequence
// brings a single token).
#include "ptx.cuh"
#include "seq_tile.cuh"

namespace ne {

constexpr int kKernelShortConv = 48;
constexpr int kMaxTaps = 16;

struct ShortConvArgs {
  const void* u; long long ld; const void* w; void* q; void* kc; void* vc; const long long* rows; void* window;
  const int* slots; const int* cu; const int* fresh;
  int num_seqs, C, qw, kw, vw, taps;
};

// V values of type T as they lie in memory, in 32-bit words
template <typename T, int V> struct Pack;
template <> struct Pack<__nv_bfloat16, 8> {
  static constexpr int kWords = 4;
  uint32_t w[4];
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { const uint4 r = *reinterpret_cast<const uint4*>(p); w[0] = r.x; w[1] = r.y; w[2] = r.z; w[3] = r.w; }
  __device__ __forceinline__ void store(__nv_bfloat16* p) const { *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]); }
};
template <> struct Pack<float, 4> {
  static constexpr int kWords = 4;
  uint32_t w[4];
  __device__ __forceinline__ void load(const float* p) { const uint4 r = *reinterpret_cast<const uint4*>(p); w[0] = r.x; w[1] = r.y; w[2] = r.z; w[3] = r.w; }
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<uint4*>(p) = make_uint4(w[0], w[1], w[2], w[3]); }
};
template <> struct Pack<__nv_bfloat16, 1> {
  static constexpr int kWords = 1;
  uint32_t w[1];
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { w[0] = *reinterpret_cast<const uint16_t*>(p); }
  __device__ __forceinline__ void store(__nv_bfloat16* p) const { *reinterpret_cast<uint16_t*>(p) = (uint16_t)w[0]; }
};
template <> struct Pack<float, 1> {
  static constexpr int kWords = 1;
  uint32_t w[1];
  __device__ __forceinline__ void load(const float* p) { w[0] = *reinterpret_cast<const uint32_t*>(p); }
  __device__ __forceinline__ void store(float* p) const { *reinterpret_cast<uint32_t*>(p) = w[0]; }
};
// the values of one word: a pair of bf16 (the upper one unused in a pack of one), or a float
__device__ __forceinline__ float2 word_get(uint32_t w, const __nv_bfloat16*) { return unpack_bf16x2(w); }
__device__ __forceinline__ float2 word_get(uint32_t w, const float*) { return make_float2(__uint_as_float(w), 0.f); }
__device__ __forceinline__ uint32_t word_put(float2 f, const __nv_bfloat16*) { return pack_bf16x2(f.x, f.y); }
__device__ __forceinline__ uint32_t word_put(float2 f, const float*) { return __float_as_uint(f.x); }

// kTaps = 0: any number up to kMaxTaps, with the inputs read again for every tap
template <typename T, int V, int kTaps, int kTile>
__global__ void __launch_bounds__(128, kTile == 8 ? 5 : 6) shortconv_kernel(const ShortConvArgs a) {
  const int c = (int)(blockIdx.y * 128 + threadIdx.x) * V, taps = kTaps ? kTaps : a.taps;
  constexpr int kW = Pack<T, V>::kWords;
  const T* kind = nullptr;           // picks the word functions
  const bool live = c < a.C;
  const T* w = reinterpret_cast<const T*>(a.w) + c;
  Pack<T, V> wv[kTaps ? kTaps : 1];
  if (kTaps && live)                  // weights may be read before the kernel in front has finished
#pragma unroll
    for (int j = 0; j < kTaps; j++) wv[j].load(w + (long long)j * a.C);
  pdl_wait(); pdl_trigger();
  int seq, tok0;
  find_seq_tile(a.cu, a.num_seqs, kTile, blockIdx.x, seq, tok0);
  if (seq < 0 || !live) return;
  const int q_beg = a.cu[seq], q_len = a.cu[seq + 1] - q_beg, r0 = tok0 - q_beg, n = min(kTile, q_len - r0), back = taps - 1;
  const T* u = reinterpret_cast<const T*>(a.u) + (long long)q_beg * a.ld + c;
  int slot = taps > 1 ? a.slots[seq] : 0;
  const bool fresh = taps <= 1 || a.fresh[seq] != 0;
  if (!NE_INDEX_OK(slot, BK_STATE_SLOTS, kKernelShortConv, __LINE__)) slot = 0;
  T* win = reinterpret_cast<T*>(a.window) + (long long)slot * back * a.C + c;
  // input s of the sequence, counted from the first token of this step
  auto input = [&](int s, Pack<T, V>& p) {
    if (s >= 0) p.load(u + (long long)s * a.ld);
    else if (fresh) {
#pragma unroll
      for (int e = 0; e < kW; e++) p.w[e] = 0;
    }
    else p.load(win + (long long)(back + s) * a.C);
  };
  auto put = [&](int t, const Pack<T, V>& o) {
    const long long tok = tok0 + t;
    if (c < a.qw) { o.store(reinterpret_cast<T*>(a.q) + tok * a.qw + c); return; }
    const long long row = a.rows[tok];
    if (row < 0 || !NE_INDEX_OK(row, BK_CACHE_ROWS, kKernelShortConv, __LINE__)) return;
    if (c < a.qw + a.kw) o.store(reinterpret_cast<T*>(a.kc) + row * a.kw + c - a.qw);
    else o.store(reinterpret_cast<T*>(a.vc) + row * a.vw + c - a.qw - a.kw);
  };
  if constexpr (kTaps > 0) {
    Pack<T, V> in[kTile + kTaps - 1];
#pragma unroll
    for (int j = 0; j < kTile + kTaps - 1; j++)
      if (j < kTaps - 1) input(r0 - (kTaps - 1) + j, in[j]);
      else if (j < n + kTaps - 1) in[j].load(u + (long long)(r0 - (kTaps - 1) + j) * a.ld);
      else {
#pragma unroll
        for (int e = 0; e < kW; e++) in[j].w[e] = 0;
      }
    // word by word, the results in place of the oldest input of each
#pragma unroll
    for (int e = 0; e < kW; e++) {
      float2 f[kTaps + 1], wf[kTaps];
#pragma unroll
      for (int j = 0; j < kTaps; j++) { wf[j] = word_get(wv[j].w[e], kind); f[j] = word_get(in[j].w[e], kind); }
#pragma unroll
      for (int t = 0; t < kTile; t++) {
        float2 y = make_float2(0.f, 0.f);
#pragma unroll
        for (int j = 0; j < kTaps; j++) { y.x = fmaf(wf[j].x, f[j].x, y.x); y.y = fmaf(wf[j].y, f[j].y, y.y); }
        in[t].w[e] = word_put(y, kind);
#pragma unroll
        for (int j = 0; j + 1 < kTaps; j++) f[j] = f[j + 1];
        if (t + 1 < kTile) f[kTaps - 1] = word_get(in[t + kTaps].w[e], kind);
      }
    }
#pragma unroll
    for (int t = 0; t < kTile; t++)
      if (t < n) put(t, in[t]);
  } else {
    for (int t = 0; t < n; t++) {
      float2 y[kW];
#pragma unroll
      for (int e = 0; e < kW; e++) y[e] = make_float2(0.f, 0.f);
      for (int j = 0; j < taps; j++) {
        Pack<T, V> p, q;
        input(r0 + t - back + j, p);
        q.load(w + (long long)j * a.C);
#pragma unroll
        for (int e = 0; e < kW; e++) {
          const float2 f = word_get(p.w[e], kind), g = word_get(q.w[e], kind);
          y[e].x = fmaf(g.x, f.x, y[e].x); y[e].y = fmaf(g.y, f.y, y[e].y);
        }
      }
      Pack<T, V> o;
#pragma unroll
      for (int e = 0; e < kW; e++) o.w[e] = word_put(y[e], kind);
      put(t, o);
    }
  }
  if (r0 == 0)                       // the next window; a short portion keeps the end of the old one, which lies behind the row being written
    for (int i = 0; i < back; i++) {
      Pack<T, V> p;
      input(q_len - back + i, p);
      p.store(win + (long long)i * a.C);
    }
}

template <typename T, int V>
static int shortconv_t(const ShortConvArgs& a, int T_, int max_q, cudaStream_t st) {
  const unsigned cy = (unsigned)((a.C + 128 * V - 1) / (128 * V));
  const bool one = max_q == 1;
  const int tile = one ? 1 : (a.taps >= 2 && a.taps <= 4 ? 8 : 16);
  const long long all = (long long)T_ / tile + a.num_seqs;
  const dim3 grid((unsigned)(all < T_ ? all : T_), cy);
  void (*k)(const ShortConvArgs);
  switch (a.taps) {
    case 2: k = one ? shortconv_kernel<T, V, 2, 1> : shortconv_kernel<T, V, 2, 8>; break;
    case 3: k = one ? shortconv_kernel<T, V, 3, 1> : shortconv_kernel<T, V, 3, 8>; break;
    case 4: k = one ? shortconv_kernel<T, V, 4, 1> : shortconv_kernel<T, V, 4, 8>; break;
    default: k = one ? shortconv_kernel<T, V, 0, 1> : shortconv_kernel<T, V, 0, 16>; break;
  }
  return (int)launch_pdl(k, grid, dim3(128), 0, st, a);
}

}  // namespace ne

using namespace ne;

// u [T, >= C] (row stride ld), w [taps, C], C = qw + kw + vw; q [T, qw]; kc / vc: caches of rows kw and vw wide, row numbers `rows` [T] (-1: not
// stored), unused when kw = vw = 0.  window [slots, taps - 1, C] with slots / fresh [num_seqs] (unused for one tap).  max_q: longest run of new
// tokens of a sequence.
extern "C" int ne_shortconv(const void* u, long long ld, const void* w, int taps, void* q, int qw, void* kc, int kw, void* vc, int vw, const long long* rows,
                            void* window, const int* slots, const int* cu, const int* fresh, int T, int num_seqs, int max_q, int fp32, cudaStream_t st) {
  if (T <= 0) return 0;
  const int C = qw + kw + vw;
  if (taps < 1 || taps > kMaxTaps || qw < 1 || kw < 0 || vw < 0 || ld < C || max_q < 1 || num_seqs < 1) return 1001;
  if ((kw && (!kc || !rows)) || (vw && (!vc || !rows)) || (taps > 1 && (!window || !slots || !fresh))) return 1002;
  ShortConvArgs a;
  a.u = u; a.ld = ld; a.w = w; a.q = q; a.kc = kc; a.vc = vc; a.rows = rows; a.window = window; a.slots = slots; a.cu = cu; a.fresh = fresh;
  a.num_seqs = num_seqs; a.C = C; a.qw = qw; a.kw = kw; a.vw = vw; a.taps = taps;
  const int per = fp32 ? 4 : 8;
  const uintptr_t al = (uintptr_t)u | (uintptr_t)w | (uintptr_t)q | (uintptr_t)kc | (uintptr_t)vc | (uintptr_t)window;
  const bool vec = qw % per == 0 && kw % per == 0 && vw % per == 0 && ld % per == 0 && al % 16 == 0;
  if (fp32) return vec ? shortconv_t<float, 4>(a, T, max_q, st) : shortconv_t<float, 1>(a, T, max_q, st);
  return vec ? shortconv_t<__nv_bfloat16, 8>(a, T, max_q, st) : shortconv_t<__nv_bfloat16, 1>(a, T, max_q, st);
}
