// Plain tiled matrix product on CUDA cores: D[b] = A[b] B[b]^T with fp32 accumulation in the order of K.  Serves what the
// tensor-core GEMM does not take: true 32-bit operands (fp32 runs, no TF32) and bf16 operands whose sizes or strides TMA cannot
// address (K or N not a multiple of 8, unaligned rows), also over the expert-major rows of a mixture.  The result of a row does not depend on the other rows of the call.
#include "ptx.cuh"

namespace ne {

__device__ __forceinline__ float ld_f(const float* p) { return *p; }
__device__ __forceinline__ float ld_f(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void st_f(float* p, float v) { *p = v; }
__device__ __forceinline__ void st_f(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

constexpr int kTile = 64, kTileK = 16;

// grid = (ceil(N / 64), ceil(M / 64), batch); 256 threads, 4 x 4 outputs each
template <typename TI, typename TO>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const TI* __restrict__ A, long long lda, long long a_bs, const TI* __restrict__ B, long long ldb,
                                                       long long b_bs, TO* __restrict__ D, long long ldd, long long d_bs, int M, int N, int K,
                                                       const float* __restrict__ bias, int act, int act_from, const int* __restrict__ counts,
                                                       const int* __restrict__ row_start, int groups) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  __shared__ float sA[kTileK][kTile + 4], sB[kTileK][kTile + 4];
  A += blockIdx.z * a_bs; B += blockIdx.z * b_bs; D += blockIdx.z * d_bs;
  const int m0 = blockIdx.y * kTile, n0 = blockIdx.x * kTile;
  if (row_start) {                  // rows of group g start at a multiple of the tile; a tile belongs to the last group that starts at or before it
    if (m0 >= row_start[groups]) return;
    int lo = 0, hi = groups - 1;
    while (lo < hi) { const int mid = (lo + hi + 1) >> 1; if (row_start[mid] <= m0) lo = mid; else hi = mid - 1; }
    M = min(M, row_start[lo] + counts[lo]);
    if (m0 >= M) return;
    B += lo * b_bs;
  }
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += kTileK) {
    for (int i = threadIdx.x; i < kTile * kTileK; i += 256) {
      const int r = i / kTileK, k = i % kTileK;
      sA[k][r] = (m0 + r < M && k0 + k < K) ? ld_f(A + (long long)(m0 + r) * lda + k0 + k) : 0.f;
      sB[k][r] = (n0 + r < N && k0 + k < K) ? ld_f(B + (long long)(n0 + r) * ldb + k0 + k) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kTileK; k++) {
      const float4 a = *reinterpret_cast<const float4*>(&sA[k][ty * 4]), b = *reinterpret_cast<const float4*>(&sB[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; i++)
#pragma unroll
    for (int j = 0; j < 4; j++) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m >= M || n >= N) continue;
      float v = bias ? acc[i][j] + bias[n] : acc[i][j];
      if (act && n >= act_from) { if (act == 1) { v = fmaxf(v, 0.f); v *= v; } else v = tanhf(v); }
      st_f(D + (long long)m * ldd + n, v);
    }
}

template <typename TI, typename TO>
static int simt(const void* A, long long lda, long long a_bs, const void* B, long long ldb, long long b_bs, void* D, long long ldd, long long d_bs,
                int M, int N, int K, int batch, const float* bias, int act, int act_from, cudaStream_t st, const int* counts = nullptr, const int* row_start = nullptr,
                int groups = 0) {
  const dim3 grid((unsigned)((N + kTile - 1) / kTile), (unsigned)((M + kTile - 1) / kTile), (unsigned)batch);
  return (int)launch_pdl(gemm_simt_kernel<TI, TO>, grid, dim3(256), 0, st, (const TI*)A, lda, a_bs, (const TI*)B, ldb, b_bs, (TO*)D, ldd, d_bs, M, N, K, bias, act, act_from,
                         counts, row_start, groups);
}

}  // namespace ne

using namespace ne;

// A [batch, M, K] (row stride lda, batch stride a_bs, elements), B [batch, N, K], D [batch, M, N].  in_fp32 / out_fp32: element types
// of the operands and of the result (bf16 otherwise).  bias (fp32 [N] or null) is added before the result is rounded; then act (0 none,
// 1 square of relu, 2 tanh) on the columns from act_from on.
extern "C" int ne_gemm_simt(const void* A, long long lda, long long a_bs, const void* B, long long ldb, long long b_bs, void* D, long long ldd,
                            long long d_bs, int M, int N, int K, int batch, int in_fp32, int out_fp32, const float* bias, int act, int act_from, cudaStream_t st) {
  if (M <= 0 || N <= 0 || batch <= 0) return 0;
  if (K < 0 || batch > 65535 || (M + kTile - 1) / kTile > 65535) return 1001;
  if (in_fp32) return out_fp32 ? simt<float, float>(A, lda, a_bs, B, ldb, b_bs, D, ldd, d_bs, M, N, K, batch, bias, act, act_from, st) : 1002;
  return out_fp32 ? simt<__nv_bfloat16, float>(A, lda, a_bs, B, ldb, b_bs, D, ldd, d_bs, M, N, K, batch, bias, act, act_from, st)
                  : simt<__nv_bfloat16, __nv_bfloat16>(A, lda, a_bs, B, ldb, b_bs, D, ldd, d_bs, M, N, K, batch, bias, act, act_from, st);
}

// Grouped form: rows [row_start[g], row_start[g] + counts[g]) of A [M, K] times B[g] [N, K]; group starts are multiples of 64, D [M, N] as A.
extern "C" int ne_gemm_simt_groups(const void* A, const void* B, void* D, int M, int N, int K, int groups, const int* counts, const int* row_start, int fp32,
                                   cudaStream_t st) {
  if (M <= 0 || N <= 0) return 0;
  if (K < 0 || groups < 1 || (M + kTile - 1) / kTile > 65535 || !counts || !row_start) return 1001;
  const long long b_bs = (long long)N * K;
  return fp32 ? simt<float, float>(A, K, 0, B, K, b_bs, D, N, 0, M, N, K, 1, nullptr, 0, 0, st, counts, row_start, groups)
              : simt<__nv_bfloat16, __nv_bfloat16>(A, K, 0, B, K, b_bs, D, N, 0, M, N, K, 1, nullptr, 0, 0, st, counts, row_start, groups);
}
