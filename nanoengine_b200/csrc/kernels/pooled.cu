// Front end of attention over a window of tokens and pooled blocks of older ones, bf16 and fp32, any sizes:
//   * pooled_prepare: RMS norm of q and of k over all heads at once, rotation of the first `dims` columns of every query and key head and of whole
//     values (column i with column i + half), q back in place, key and value rows into the paged caches.  One CTA per token, its row in shared memory.
//   * block means: a block of P tokens is pooled when its last token arrives - mean of the P rows as the caches hold them, in the order of
//     positions.  Calls of single tokens do it in the same kernel, calls with portions in a second one, when all rows are stored.
// Pooled rows are kept in groups of eight neighbours in the page of the first token of the group's first block.
#include "ptx.cuh"
#include "pooled.cuh"

namespace ne {

__device__ __forceinline__ float pl_ld(const float* p) { return *p; }
__device__ __forceinline__ float pl_ld(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void pl_st(float* p, float v) { *p = v; }
__device__ __forceinline__ void pl_st(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ float4 pl_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 pl_ld4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void pl_st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void pl_st4(__nv_bfloat16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w)); }

__device__ __forceinline__ void cp_async8(uint32_t dst, const void* src) { asm volatile("cp.async.ca.shared.global [%0], [%1], 8;" ::"r"(dst), "l"(src) : "memory"); }

struct PoolArgs {
  void* qkv; long long ld;                   // [T, H D | G D | G Dv]
  const void* q_norm; const void* k_norm; float eps;
  const long long* positions; const float* k_table; const float* v_table; int n_pos;     // [n_pos, dims], [n_pos, Dv]: cos | sin
  void* k_cache; void* v_cache; void* k_pool; void* v_pool; const long long* slots;
  const int* block_tables; int bt_stride; const int* cu; int B;
  int T, H, G, D, Dv, dims, pool, block_size, pool_rows;
};

constexpr int kOffs = 64;                    // rows whose places are looked up at a time

// Where the pooled row goes that token t completes: row of the pooled caches, -1 when it completes none.  bt: the sequence's block table.
__device__ __forceinline__ long long block_place(const PoolArgs& a, int t, long long p, const int*& bt) {
  if (p < 0 || (p + 1) % a.pool || a.slots[t] < 0) return -1;
  int lo = 0, hi = a.B - 1;                   // last sequence whose first token is <= t
  if (t < a.B && a.cu[t] == t && a.cu[t + 1] == t + 1) lo = hi = t;      // single tokens
  while (lo < hi) { const int mid = (lo + hi + 1) >> 1; if (a.cu[mid] <= t) lo = mid; else hi = mid - 1; }
  bt = a.block_tables + (long long)lo * a.bt_stride;
  int page, row;
  pooled_place((int)(p / a.pool), a.pool, a.block_size, page, row);
  if (page >= a.bt_stride || p / a.block_size >= a.bt_stride) { if (threadIdx.x == 0) report(ST_BAD_INDEX, 50, t, page); return -1; }
  const int dst = bt[page];
  return NE_INDEX_OK(dst, BK_CACHE_PAGES, 50, __LINE__) ? (long long)dst * a.pool_rows + row : -1;
}

// Mean of rows p - pool + 1 .. p into pooled row `dst`, summed in the order of positions.  Whole CTA; the rows are stored by now.
template <typename T, int V>
__device__ __forceinline__ void pool_block(const PoolArgs& a, long long p, long long dst, const int* bt, long long* offs) {
  const int kw = a.G * a.D, vw = a.G * a.Dv, bs = a.block_size;
  const float inv = 1.f / (float)a.pool;
  for (int c0 = 0; c0 < kw + vw; c0 += blockDim.x * V) {
    const int c = c0 + threadIdx.x * V;                                   // V divides kw: a group never straddles
    const bool key = c < kw, on = c < kw + vw;
    const int w = key ? kw : vw, cc = key ? c : c - kw;
    const T* src = reinterpret_cast<const T*>(key ? a.k_cache : a.v_cache) + cc;
    float s[V];
#pragma unroll
    for (int e = 0; e < V; e++) s[e] = 0.f;
    for (int j0 = 0; j0 < a.pool; j0 += kOffs) {
      const int m = min(kOffs, a.pool - j0);
      if (a.pool > kOffs || c0 == 0) {
        __syncthreads();
        if ((int)threadIdx.x < m) {
          const int q = (int)p - a.pool + 1 + j0 + threadIdx.x, pg = bt[q / bs];
          offs[threadIdx.x] = NE_INDEX_OK(pg, BK_CACHE_PAGES, 51, __LINE__) ? (long long)pg * bs + q % bs : 0;
        }
        __syncthreads();
      }
      if (!on) continue;
      int j = 0;
      for (; j + 8 <= m; j += 8) {
        if constexpr (V == 4) {
          float4 v[8];
#pragma unroll
          for (int e = 0; e < 8; e++) v[e] = pl_ld4(src + offs[j + e] * w);
#pragma unroll
          for (int e = 0; e < 8; e++) { s[0] += v[e].x; s[1] += v[e].y; s[2] += v[e].z; s[3] += v[e].w; }
        } else {
          float v[8];
#pragma unroll
          for (int e = 0; e < 8; e++) v[e] = pl_ld(src + offs[j + e] * w);
#pragma unroll
          for (int e = 0; e < 8; e++) s[0] += v[e];
        }
      }
      for (; j < m; j++) {
        if constexpr (V == 4) { const float4 v = pl_ld4(src + offs[j] * w); s[0] += v.x; s[1] += v.y; s[2] += v.z; s[3] += v.w; }
        else s[0] += pl_ld(src + offs[j] * w);
      }
    }
    if (!on) continue;
    T* out = reinterpret_cast<T*>(key ? a.k_pool : a.v_pool) + dst * w + cc;
    if constexpr (V == 4) pl_st4(out, make_float4(s[0] * inv, s[1] * inv, s[2] * inv, s[3] * inv));
    else pl_st(out, s[0] * inv);
  }
}

template <typename T, int V>
__global__ void __launch_bounds__(512) pooled_prepare_kernel(const PoolArgs a, const int pool_here) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  extern __shared__ __align__(16) float sm[];       // key table | value table | the row
  __shared__ float red[2][16];
  __shared__ long long offs[kOffs];
  const int t = blockIdx.x, nq = a.H * a.D, nk = a.G * a.D, nv = a.G * a.Dv, W = nq + nk + nv, D = a.D, Dv = a.Dv, dims = a.dims;
  float *s_kt = sm, *s_vt = sm + (dims + 3) / 4 * 4;
  T* x0 = reinterpret_cast<T*>(s_vt + (Dv + 3) / 4 * 4);
  T* row = reinterpret_cast<T*>(a.qkv) + (long long)t * a.ld;
  long long p = a.positions[t];
  const long long slot = a.slots[t];
  // the row is on its way while the position, and the tables' rows that it names, are looked up
  constexpr int PE = V == 4 ? 16 / (int)sizeof(T) : 1;
  const int step = V == 4 ? (W % PE == 0 && a.ld % PE == 0 ? PE : 4) : 1;
  for (int i = threadIdx.x * step; i < W; i += blockDim.x * step) {
    if constexpr (V == 4) {
      if (step == PE) cp_async16(smem_u32(x0 + i), row + i, 16);
      else cp_async8(smem_u32(x0 + i), row + i);
    } else x0[i] = row[i];
  }
  if (p < 0 || p >= a.n_pos) { if (threadIdx.x == 0) report(ST_BAD_INDEX, 52, t, (int)p); p = 0; }
  if constexpr (V == 4) {
    for (int i = threadIdx.x * 4; i < dims; i += blockDim.x * 4) cp_async16(smem_u32(s_kt + i), a.k_table + p * dims + i, 16);
    for (int i = threadIdx.x * 4; i < Dv; i += blockDim.x * 4) cp_async16(smem_u32(s_vt + i), a.v_table + p * Dv + i, 16);
  } else {
    for (int i = threadIdx.x; i < dims; i += blockDim.x) s_kt[i] = a.k_table[p * dims + i];
    for (int i = threadIdx.x; i < Dv; i += blockDim.x) s_vt[i] = a.v_table[p * Dv + i];
  }
  const int* bt = nullptr;
  const long long place = pool_here ? block_place(a, t, p, bt) : -1;
  if constexpr (V == 4) { cp_async_commit(); cp_async_wait<0>(); }
  float qq = 0.f, kk = 0.f;
  for (int i = threadIdx.x * step; i < W; i += blockDim.x * step) {       // what the thread copied itself
    if constexpr (V == 4) {
#pragma unroll
      for (int e = 0; e < PE; e += 4) {
        if (e >= step) break;
        const float4 v = pl_ld4(x0 + i + e);
        const float s = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        if (i + e < nq) qq += s; else if (i + e < nq + nk) kk += s;       // 4 divides nq and nk
      }
    } else {
      const float v = pl_ld(x0 + i);
      if (i < nq) qq += v * v; else if (i < nq + nk) kk += v * v;
    }
  }
  qq = warp_sum(qq); kk = warp_sum(kk);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) { red[0][warp] = qq; red[1][warp] = kk; }
  __syncthreads();
  const float rq = rsqrtf(warp_sum(lane < nw ? red[0][lane] : 0.f) / (float)nq + a.eps), rk = rsqrtf(warp_sum(lane < nw ? red[1][lane] : 0.f) / (float)nk + a.eps);
  const bool store = slot >= 0 && NE_INDEX_OK(slot, BK_CACHE_ROWS, 53, __LINE__);
  // one warp per head; V divides the head sizes and the halves of the rotations
  for (int u = warp; u < a.H + 2 * a.G; u += nw) {
    const int part = u < a.H ? 0 : u < a.H + a.G ? 1 : 2;
    if (part && !store) break;
    const int j0 = part == 0 ? u * D : part == 1 ? (u - a.H) * D : (u - a.H - a.G) * Dv, i0 = part == 0 ? j0 : part == 1 ? nq + j0 : nq + nk + j0;
    const int width = part == 2 ? Dv : D, turned = part == 2 ? Dv : dims, half = turned >> 1;
    const float* tab = part == 2 ? s_vt : s_kt;
    const T* w = reinterpret_cast<const T*>(part == 0 ? a.q_norm : a.k_norm) + j0;
    const float r = part == 0 ? rq : rk;
    T* dst = part == 0 ? row + j0 : part == 1 ? reinterpret_cast<T*>(a.k_cache) + slot * nk + j0 : reinterpret_cast<T*>(a.v_cache) + slot * nv + j0;
    // items of V columns: the pairs of a rotation (columns d and d + half), then the columns that pass
    const int pairs = half / V, items = pairs + (width - turned) / V;
    for (int item = lane; item < items; item += 32) {
      const int d = item < pairs ? item * V : turned + (item - pairs) * V;
      if constexpr (V == 4) {
        float4 x = pl_ld4(x0 + i0 + d);
        if (part < 2) { const float4 g = pl_ld4(w + d); x.x *= r * g.x; x.y *= r * g.y; x.z *= r * g.z; x.w *= r * g.w; }
        if (item < pairs) {
          float4 y = pl_ld4(x0 + i0 + d + half);
          if (part < 2) { const float4 g = pl_ld4(w + d + half); y.x *= r * g.x; y.y *= r * g.y; y.z *= r * g.z; y.w *= r * g.w; }
          const float4 c = *reinterpret_cast<const float4*>(tab + d), s = *reinterpret_cast<const float4*>(tab + half + d);
          pl_st4(dst + d + half, make_float4(y.x * c.x + x.x * s.x, y.y * c.y + x.y * s.y, y.z * c.z + x.z * s.z, y.w * c.w + x.w * s.w));
          x = make_float4(x.x * c.x - y.x * s.x, x.y * c.y - y.y * s.y, x.z * c.z - y.z * s.z, x.w * c.w - y.w * s.w);
        }
        pl_st4(dst + d, x);
      } else {
        float x = pl_ld(x0 + i0 + d);
        if (part < 2) x *= r * pl_ld(w + d);
        if (item < pairs) {
          float y = pl_ld(x0 + i0 + d + half);
          if (part < 2) y *= r * pl_ld(w + d + half);
          const float c = tab[d], s = tab[half + d];
          pl_st(dst + d + half, y * c + x * s);
          x = x * c - y * s;
        }
        pl_st(dst + d, x);
      }
    }
  }
  if (place < 0) return;
  __syncthreads();                                   // this token's rows are stored
  pool_block<T, V>(a, p, place, bt, offs);
}

// One CTA per block completed in this call: CTA i takes the i-th, counted over the sequences.
template <typename T, int V>
__global__ void __launch_bounds__(256) pooled_means_kernel(const PoolArgs a) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  __shared__ long long offs[kOffs];
  __shared__ int s_tok;
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    int rem = blockIdx.x, tok = -1;
    for (int s0 = 0; s0 < a.B && tok < 0; s0 += 32) {
      const int s = s0 + lane;
      int t0 = 0, n = 0, done = 0;
      long long p0 = 0;
      if (s < a.B) {
        t0 = a.cu[s];
        n = a.cu[s + 1] - t0;
        if (n > 0) { p0 = a.positions[t0]; done = (int)((p0 + n) / a.pool - p0 / a.pool); }
      }
      int incl = done;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) { const int v = __shfl_up_sync(0xffffffffu, incl, o); if (lane >= o) incl += v; }
      const unsigned hit = __ballot_sync(0xffffffffu, rem < incl);
      if (hit) {
        const int l = __ffs(hit) - 1;
        // the token at the end of the block
        const long long mine = t0 + (p0 / a.pool + 1 + rem - (incl - done)) * a.pool - 1 - p0;
        tok = __shfl_sync(0xffffffffu, (int)mine, l);
      } else {
        rem -= __shfl_sync(0xffffffffu, incl, 31);
      }
    }
    if (lane == 0) s_tok = tok;
  }
  __syncthreads();
  const int t = s_tok;
  if (t < 0 || t >= a.T) return;
  const long long p = a.positions[t];
  const int* bt = nullptr;
  const long long place = block_place(a, t, p, bt);
  if (place >= 0) pool_block<T, V>(a, p, place, bt, offs);
}

template <typename T>
static int pooled_t(const PoolArgs& a, int max_q, cudaStream_t st) {
  const int W = a.H * a.D + a.G * (a.D + a.Dv);
  const uintptr_t al = (uintptr_t)a.qkv | (uintptr_t)a.q_norm | (uintptr_t)a.k_norm | (uintptr_t)a.k_cache | (uintptr_t)a.v_cache | (uintptr_t)a.k_pool | (uintptr_t)a.v_pool;
  const bool vec = (uintptr_t)a.k_table % 16 == 0 && (uintptr_t)a.v_table % 16 == 0 && a.D % 4 == 0 && a.Dv % 8 == 0 && a.dims % 8 == 0 && a.ld % 4 == 0 && al % 16 == 0;
  const int per = vec ? 4 : 1;
  int threads = ((W + per - 1) / per + 31) / 32 * 32;
  const int most = max_q == 1 ? 512 : 256;           // few CTAs: wide ones
  threads = threads > most ? most : threads < 64 ? 64 : threads;
  const size_t smem = sizeof(float) * ((a.dims + 3) / 4 * 4 + (a.Dv + 3) / 4 * 4) + sizeof(T) * (size_t)W;
  auto k = vec ? pooled_prepare_kernel<T, 4> : pooled_prepare_kernel<T, 1>;
  if (smem > 40 * 1024) {
    if (smem > 227 * 1024) return 1001;
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  cudaError_t e = launch_pdl(k, dim3((unsigned)a.T), dim3((unsigned)threads), smem, st, a, max_q == 1 ? 1 : 0);
  if (e != cudaSuccess || max_q == 1) return (int)e;
  const long long blocks = (long long)a.T / a.pool + a.B, most_blocks = blocks < a.T ? blocks : a.T;
  int mt = (a.G * (a.D + a.Dv) / per + 31) / 32 * 32;
  mt = mt > 256 ? 256 : mt < 64 ? 64 : mt;           // at least kOffs threads
  return (int)launch_pdl(vec ? pooled_means_kernel<T, 4> : pooled_means_kernel<T, 1>, dim3((unsigned)most_blocks), dim3((unsigned)mt), 0, st, a);
}

}  // namespace ne

using namespace ne;

// See PoolArgs.  Caches [pages, block_size, G, D / Dv], pooled rows [pages, pool_rows, G, D / Dv], all in the activation dtype (fp32 = 1: float).
// max_q: most tokens a sequence brings; 1 pools in the same kernel (a call then has no two tokens of one sequence).
extern "C" int ne_pooled_prepare(void* qkv, long long ld, const void* q_norm, const void* k_norm, float eps, const long long* positions, const float* k_table,
                                 const float* v_table, int n_pos, void* k_cache, void* v_cache, void* k_pool, void* v_pool, const long long* slots,
                                 const int* block_tables, int bt_stride, const int* cu, int B, int T, int H, int G, int D, int Dv, int dims, int pool, int block_size,
                                 int pool_rows, int max_q, int fp32, cudaStream_t st) {
  if (T <= 0 || B <= 0) return 0;
  if (H < 1 || G < 1 || D < 1 || Dv < 2 || Dv % 2 || dims < 0 || dims % 2 || dims > D || pool < 1 || block_size < 1 || n_pos < 1 ||
      pool_rows < (block_size + 8 * pool - 1) / (8 * pool) * 8 || ld < (long long)H * D + (long long)G * (D + Dv)) return 1001;
  PoolArgs a;
  a.qkv = qkv; a.ld = ld; a.q_norm = q_norm; a.k_norm = k_norm; a.eps = eps; a.positions = positions; a.k_table = k_table; a.v_table = v_table; a.n_pos = n_pos;
  a.k_cache = k_cache; a.v_cache = v_cache; a.k_pool = k_pool; a.v_pool = v_pool; a.slots = slots; a.block_tables = block_tables; a.bt_stride = bt_stride; a.cu = cu;
  a.B = B; a.T = T; a.H = H; a.G = G; a.D = D; a.Dv = Dv; a.dims = dims; a.pool = pool; a.block_size = block_size; a.pool_rows = pool_rows;
  return fp32 ? pooled_t<float>(a, max_q, st) : pooled_t<__nv_bfloat16>(a, max_q, st);
}
