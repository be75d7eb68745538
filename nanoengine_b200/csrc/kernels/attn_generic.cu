// Shape-generic paged attention on CUDA cores: the path for head sizes the tensor-core kernels do not cover
// (small test models), for DSA sparse key lists, and for GQA caches.  One CTA per (query token, group of 4 heads),
// one warp per head; keys are staged through shared memory 32 at a time, each lane scores one key, the
// softmax is online, and each lane owns a slice of the output dimensions.
//
//   MLA:  q [T, H, Dk], cache rows [Dk] (first Dv values double as V), out [T, H, Dv]
//   GQA:  q [T, Hq, D], k/v caches [slots, Hkv, D], out [T, Hq, D]
// Keys of a query: positions [0, limit] of its sequence through the block table (causal), or an explicit list of
// physical slots (sparse, -1 = skip).  Cache dtype bf16, e4m3 (query is then clamped and cast to e4m3 as well) or fp32 (query and
// output fp32 too: runs in true 32-bit).  Options: a window of the last keys, scores capped as cap tanh(s / cap), a distance bias
// -slope[head] (query position - key position) after the cap, the output of a head times sigmoid(gate[token, head]) and a constant.
// With pooled rows (pooled.cuh) a query also sees the blocks wholly in front of its window, in the same softmax; an output may be rotated back by
// its position (pairs of columns d, d + Dv / 2).  Behind a window the first `keep` tokens of the sequence stay visible.
// Differential form (maps = 2): a head has two query vectors, a key / value head two key vectors side by side; two warps take the two maps of a head
// over the same values, and o = a1 - mixing a2 is divided by its root mean square, scaled, and multiplied by sigmoid(egate) element by element.
//
// Replaces in the reference: attention/base.py:451-525 (SDPA reference), flash_mla sparse decode call sites
// (layers/backends/mla/flash_mla.py:22-121) for the sparse case, flashinfer / FA paged GQA wrappers.
#include "ptx.cuh"
#include "pooled.cuh"
#include <cstring>

namespace ne {

constexpr int kKeysPerTile = 32;
constexpr int kHeadsPerCta = 4;

struct AttnArgs {
  const void* q; long long q_tok_stride; int q_head_stride;
  const void* k_cache; const void* v_cache;      // v_cache == nullptr: V is the first Dv values of the K row (MLA)
  long long kv_slot_stride; int kv_head_stride;   // in elements
  int kv_group;                                   // query heads per kv head (1 for MLA where kv_head_stride = 0)
  const int* block_tables; int bt_stride; int block_size;
  const int* cu_seqlens_q; const int* context_lens; int num_seqs;
  const int* sparse; int topk;                    // [T, topk] physical slots or nullptr
  void* out; long long o_tok_stride; int o_head_stride;
  float* lse;                                     // optional [T, H] natural-log LSE
  int T, H, Dk, Dv; float scale; int fp8;
  int window;                                     // > 0: a query sees only the last `window` key positions up to its own (sliding-window layers)
  int noncausal;                                  // 1: every query sees all keys of its sequence (vision encoder)
  int heads_per_cta;                              // 4 or the largest smaller divisor of the group: the heads of a CTA share one kv head
  long long v_slot_stride; int v_head_stride;     // of the separate V rows
  float softcap; const float* slopes;             // 0 / null: none
  const void* gate; long long gate_ld; float out_scale;      // gate null: none
  const void* k_pool; const void* v_pool; int pool, pool_rows;      // pool 0: none
  const float* turn; int n_pos;                              // [n_pos, Dv] cos | sin, or null
  int keep;                                                  // > 0, with a window: the first keys that stay visible
  int maps;                                                  // 1, or 2 for the differential form: H, the strides of q and kv_group then count maps
  const float* mixing; float eps; const void* egate; long long egate_ld;
};

// kind: 0 bf16, 1 e4m3, 2 fp32
__device__ __forceinline__ float load_kv(const void* base, long long idx, int kind) {
  if (kind == 2) return reinterpret_cast<const float*>(base)[idx];
  return kind ? e4m3_to_float(reinterpret_cast<const uint8_t*>(base)[idx]) : __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(base)[idx]);
}

__global__ void __launch_bounds__(128) attn_generic_kernel(const AttnArgs a) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  extern __shared__ float sm[];
  // layout: q [4][Dk] | ktile [32][Dk+1] | vtile [32][Dv+1] (only when V is separate)
  const int Dk = a.Dk, Dv = a.Dv, Dks = Dk * a.maps;          // a staged key row holds the keys of all maps
  float* sq = sm;
  float* sk = sq + kHeadsPerCta * Dk;
  float* sv = a.v_cache ? sk + kKeysPerTile * (Dks + 1) : nullptr;
  const int t = blockIdx.x, h0 = blockIdx.y * a.heads_per_cta;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = h0 + warp;
  const bool head_ok = h < a.H && warp < a.heads_per_cta;

  // which sequence owns token t
  int lo = 0, hi = a.num_seqs;
  while (lo + 1 < hi) { int mid = (lo + hi) >> 1; if (a.cu_seqlens_q[mid] <= t) lo = mid; else hi = mid; }
  const int seq = lo;
  const int q_len = a.cu_seqlens_q[seq + 1] - a.cu_seqlens_q[seq];
  const int ctx = a.context_lens[seq];
  const int limit = a.noncausal ? ctx - 1 : ctx - q_len + (t - a.cu_seqlens_q[seq]);   // last visible key position
  const int n_keys = a.sparse ? a.topk : limit + 1;
  const int first_key = (a.window > 0 && !a.sparse) ? max(0, limit - a.window + 1) : 0;

  for (int i = threadIdx.x; i < kHeadsPerCta * Dk; i += blockDim.x) {
    int hh = h0 + i / Dk, d = i % Dk;
    float v = (hh < a.H && i / Dk < a.heads_per_cta) ? load_kv(a.q, (long long)t * a.q_tok_stride + (long long)hh * a.q_head_stride + d, a.fp8 == 2 ? 2 : 0) : 0.f;
    if (a.fp8 == 1) v = e4m3_to_float(to_e4m3(fminf(fmaxf(v, -448.f), 448.f)));
    sq[i] = v;
  }
  // all 4 heads of a CTA must read the same kv head: heads per CTA divide the group size, or the group size is 1 with stride 0
  const int kvh = (a.kv_group > 0) ? h0 / a.kv_group : 0;
  const int per_lane = (Dv + 31) / 32;
  float acc[20];
#pragma unroll
  for (int j = 0; j < 20; j++) acc[j] = 0.f;
  float m_run = -INFINITY, l_run = 0.f;
  constexpr float kLog2e = 1.4426950408889634f;
  const float c = a.scale * kLog2e, slope = (a.slopes && head_ok) ? a.slopes[h] : 0.f;
  const int* bt = a.block_tables + (long long)seq * a.bt_stride;

  const int n_pool = a.pool ? pooled_visible(limit, a.window, a.pool) : 0, pool_tiles = (n_pool + kKeysPerTile - 1) / kKeysPerTile;
  const int keep_tiles = (min(a.keep, first_key) + kKeysPerTile - 1) / kKeysPerTile;          // of kept keys in front of the window
  const int tile0 = max(first_key / kKeysPerTile, keep_tiles), tiles = pool_tiles + keep_tiles + max(0, (n_keys + kKeysPerTile - 1) / kKeysPerTile - tile0);
  for (int it = 0; it < tiles; it++) {
    const bool pooled = it < pool_tiles;
    const int at = it - pool_tiles;
    const int k0 = (pooled ? it : at < keep_tiles ? at : at - keep_tiles + tile0) * kKeysPerTile, k_end = pooled ? n_pool : n_keys, k_first = pooled ? 0 : first_key;
    const void *kbase = pooled ? a.k_pool : a.k_cache, *vbase = pooled ? a.v_pool : a.v_cache;
    __syncthreads();
    // stage 32 key rows (and value rows) as fp32
    for (int r = warp; r < kKeysPerTile; r += 4) {
      int kidx = k0 + r;
      long long slot = -1;
      if (kidx < k_end) {
        if (pooled) {
          int page, row;
          pooled_place(kidx, a.pool, a.block_size, page, row);
          page = bt[page];
          slot = NE_INDEX_OK(page, BK_CACHE_PAGES, 24, __LINE__) ? (long long)page * a.pool_rows + row : -1;
        } else if (a.sparse) slot = a.sparse[(long long)t * a.topk + kidx];
        else {
          const int page = bt[kidx / a.block_size];
          slot = (a.block_size == 1 || NE_INDEX_OK(page, BK_CACHE_PAGES, 23, __LINE__)) ? (long long)page * a.block_size + kidx % a.block_size : -1;
        }
      }
      for (int d = lane; d < Dks; d += 32)
        sk[r * (Dks + 1) + d] = slot >= 0 ? load_kv(kbase, slot * a.kv_slot_stride + (long long)kvh * a.kv_head_stride + d, a.fp8) : 0.f;
      if (sv) for (int d = lane; d < Dv; d += 32)
        sv[r * (Dv + 1) + d] = slot >= 0 ? load_kv(vbase, slot * a.v_slot_stride + (long long)kvh * a.v_head_stride + d, a.fp8) : 0.f;
      if (lane == 0) sk[r * (Dks + 1) + Dks] = slot >= 0 ? 1.f : 0.f;   // validity marker in the padding column
    }
    __syncthreads();
    if (!head_ok) continue;
    // lane scores key `lane`
    const float* kr = sk + lane * (Dks + 1);
    const float* qr = sq + warp * Dk;
    const float* km = a.maps == 2 ? kr + (h & 1) * Dk : kr;
    float s = 0.f;
    for (int d = 0; d < Dk; d++) s = fmaf(qr[d], km[d], s);
    bool valid = (k0 + lane < k_end) && (k0 + lane >= k_first || k0 + lane < a.keep) && kr[Dks] != 0.f;
    float tl = s * c;
    if (a.softcap > 0.f) tl = a.softcap * tanhf(s * a.scale / a.softcap) * kLog2e;
    if (a.slopes) tl -= slope * (float)(limit - (k0 + lane)) * kLog2e;
    if (!valid) tl = -INFINITY;
    float m_new = fmaxf(m_run, warp_max(tl));
    if (m_new == -INFINITY) continue;
    float alpha = exp2f(m_run - m_new);
    float p = valid ? exp2f(tl - m_new) : 0.f;
    l_run = l_run * alpha + warp_sum(p);
    m_run = m_new;
    const float* vt = sv ? sv : sk;
    const int vstride = sv ? Dv + 1 : Dks + 1;
#pragma unroll
    for (int j = 0; j < 20; j++) acc[j] *= alpha;
    for (int kk = 0; kk < kKeysPerTile; kk++) {
      float pk = __shfl_sync(0xffffffffu, p, kk);
      if (pk == 0.f) continue;
#pragma unroll
      for (int j = 0; j < 20; j++) {
        int d = lane + 32 * j;
        if (j < per_lane && d < Dv) acc[j] = fmaf(pk, vt[kk * vstride + d], acc[j]);
      }
    }
  }
  if (a.turn || a.maps == 2) __syncthreads();  // the tiles' memory is free
  if (a.maps == 2) {
    if (head_ok) {
      const float inv = l_run > 0.f ? 1.f / l_run : 0.f;
#pragma unroll
      for (int j = 0; j < 20; j++) { const int d = lane + 32 * j; if (j < per_lane && d < Dv) sk[warp * Dv + d] = acc[j] * inv; }
    }
    __syncthreads();
    const int hr = h0 / 2 + warp;              // the head whose maps the warps 2 w and 2 w + 1 took
    if (2 * warp >= a.heads_per_cta || h0 + 2 * warp >= a.H) return;
    const float* so = sk + 2 * warp * Dv;
    const float lam = *a.mixing;
    float ss = 0.f;
    for (int d = lane; d < Dv; d += 32) { const float o = so[d] - lam * so[Dv + d]; ss += o * o; }
    const float r = rsqrtf(warp_sum(ss) / (float)Dv + a.eps) * a.out_scale;
    for (int d = lane; d < Dv; d += 32) {
      const float o = (so[d] - lam * so[Dv + d]) * r / (1.f + expf(-load_kv(a.egate, (long long)t * a.egate_ld + (long long)hr * Dv + d, a.fp8 == 2 ? 2 : 0)));
      const long long at = (long long)t * a.o_tok_stride + (long long)hr * a.o_head_stride + d;
      if (a.fp8 == 2) reinterpret_cast<float*>(a.out)[at] = o;
      else reinterpret_cast<__nv_bfloat16*>(a.out)[at] = __float2bfloat16(o);
    }
    return;
  }
  if (!head_ok) return;
  float inv = (l_run > 0.f ? 1.f / l_run : 0.f) * a.out_scale;
  if (a.gate) inv /= 1.f + expf(-load_kv(a.gate, (long long)t * a.gate_ld + h, a.fp8 == 2 ? 2 : 0));
  if (a.turn) {
    float* so = sk + warp * Dv;                // a value of the pair sits in another lane
#pragma unroll
    for (int j = 0; j < 20; j++) { const int d = lane + 32 * j; if (j < per_lane && d < Dv) so[d] = acc[j]; }
    __syncwarp();
    const int half = Dv >> 1;
    const float* tab = a.turn + (long long)min(max(limit, 0), a.n_pos - 1) * Dv;
#pragma unroll
    for (int j = 0; j < 20; j++) {
      const int d = lane + 32 * j;
      if (j < per_lane && d < Dv) {
        const int m = d < half ? d : d - half;
        acc[j] = d < half ? acc[j] * tab[m] + so[d + half] * tab[half + m] : acc[j] * tab[m] - so[m] * tab[half + m];
      }
    }
  }
#pragma unroll
  for (int j = 0; j < 20; j++) {
    int d = lane + 32 * j;
    if (j < per_lane && d < Dv) {
      const long long o = (long long)t * a.o_tok_stride + (long long)h * a.o_head_stride + d;
      if (a.fp8 == 2) reinterpret_cast<float*>(a.out)[o] = acc[j] * inv;
      else reinterpret_cast<__nv_bfloat16*>(a.out)[o] = __float2bfloat16(acc[j] * inv);
    }
  }
  if (a.lse && lane == 0) a.lse[(long long)t * a.H + h] = l_run > 0.f ? (m_run * 0.6931471805599453f + logf(l_run)) : -INFINITY;
}

// out = sum_s softmax_s(lse) * part_s  for split-KV attention.  part [S, rows, D] fp32 (already normalised), lse2 [S, rows] (log2 domain).
__global__ void attn_merge_kernel(const float* __restrict__ part, const float* __restrict__ lse2, __nv_bfloat16* __restrict__ out,
                                  int splits, long long rows, int D, int out_row_stride) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  long long row = blockIdx.x;
  float m = -INFINITY;
  for (int s = 0; s < splits; s++) m = fmaxf(m, lse2[(long long)s * rows + row]);
  float den = 0.f;
  for (int s = 0; s < splits; s++) { float l = lse2[(long long)s * rows + row]; den += (l == -INFINITY) ? 0.f : exp2f(l - m); }
  float inv = den > 0.f ? 1.f / den : 0.f;
  for (int d = threadIdx.x; d < D; d += blockDim.x) {
    float acc = 0.f;
    for (int s = 0; s < splits; s++) {
      float l = lse2[(long long)s * rows + row];
      if (l != -INFINITY) acc += exp2f(l - m) * part[((long long)s * rows + row) * D + d];
    }
    out[row * out_row_stride + d] = __float2bfloat16(acc * inv);
  }
}

// ---- sampling --------------------------------------------------------------------------------------
__device__ __forceinline__ uint32_t hash32(uint32_t x) {
  x ^= x >> 16; x *= 0x7feb352du; x ^= x >> 15; x *= 0x846ca68bu; x ^= x >> 16; return x;
}

// One CTA per row.  temperature < 1e-5: argmax.  Otherwise Gumbel-max: argmax(logit / T + g), g = -log(-log(u)), u from a
// counter-based hash of (seed, row, column).  Optionally the log-probability of the chosen token under softmax(logits).
__global__ void __launch_bounds__(1024) sample_kernel(const float* __restrict__ logits, const float* __restrict__ temps, long long* __restrict__ tok,
                                                     float* __restrict__ logprob, int V, uint64_t seed) {
  pdl_wait(); pdl_trigger();      // dependent launch: nothing above this line touches global memory
  __shared__ float s_val[32]; __shared__ int s_idx[32]; __shared__ float s_m[32]; __shared__ float s_s[32];
  const int row = blockIdx.x;
  const float* lr = logits + (long long)row * V;
  const float temp = temps[row];
  const bool greedy = temp < 1e-5f;
  const float it = greedy ? 1.f : 1.f / temp;
  float best = -INFINITY; int bi = 0x7fffffff; float m = -INFINITY, ssum = 0.f;
  for (int i = threadIdx.x; i < V; i += blockDim.x) {
    float x = lr[i];
    float v = x * it;
    if (!greedy) {
      uint32_t hsh = hash32((uint32_t)i * 0x9e3779b9u ^ hash32((uint32_t)row ^ hash32((uint32_t)seed ^ (uint32_t)(seed >> 32))));
      float u = fmaxf((float)(hsh >> 8) * (1.0f / 16777216.0f), 1e-20f);
      v += -__logf(-__logf(u));
    }
    if (v > best || (v == best && i < bi)) { best = v; bi = i; }
    if (logprob) { float nm = fmaxf(m, x); ssum = ssum * __expf(m - nm) + __expf(x - nm); m = nm; }
  }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    float ob = __shfl_xor_sync(0xffffffffu, best, o); int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
    float om = __shfl_xor_sync(0xffffffffu, m, o), os = __shfl_xor_sync(0xffffffffu, ssum, o);
    float nm = fmaxf(m, om);
    ssum = (nm == -INFINITY) ? 0.f : ssum * __expf(m - nm) + os * __expf(om - nm); m = nm;
  }
  if (lane == 0) { s_val[warp] = best; s_idx[warp] = bi; s_m[warp] = m; s_s[warp] = ssum; }
  __syncthreads();
  if (warp == 0) {
    best = lane < nw ? s_val[lane] : -INFINITY; bi = lane < nw ? s_idx[lane] : 0x7fffffff;
    m = lane < nw ? s_m[lane] : -INFINITY; ssum = lane < nw ? s_s[lane] : 0.f;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      float ob = __shfl_xor_sync(0xffffffffu, best, o); int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
      float om = __shfl_xor_sync(0xffffffffu, m, o), os = __shfl_xor_sync(0xffffffffu, ssum, o);
      float nm = fmaxf(m, om);
      ssum = (nm == -INFINITY) ? 0.f : ssum * __expf(m - nm) + os * __expf(om - nm); m = nm;
    }
    if (lane == 0) {
      tok[row] = bi;
      if (logprob) logprob[row] = lr[bi] - (m + __logf(ssum));
    }
  }
}

}  // namespace ne

using namespace ne;

static int attn_generic_launch(AttnArgs& a, cudaStream_t st) {
  // (the way out of a rotated output, kHeadsPerCta rows of Dv, fits in the tiles of 32 keys and values)
  const size_t smem = sizeof(float) * ((size_t)kHeadsPerCta * a.Dk + (size_t)kKeysPerTile * (a.Dk * a.maps + 1) + (a.v_cache ? (size_t)kKeysPerTile * (a.Dv + 1) : 0));
  static size_t configured = 0;
  if (smem > 48 * 1024 && smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(attn_generic_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  return (int)launch_pdl(attn_generic_kernel, dim3(a.T, (a.H + a.heads_per_cta - 1) / a.heads_per_cta), dim3(128), smem, st, a);
}

// Paged grouped-query attention with the options of AttnArgs: q [T, H, D], k_cache [slots, Hkv, D], v_cache [slots, Hkv, Dv] (fp32 all of
// them when fp32 = 1, else bf16), slopes [H] or null, gate [T, >= H] (row stride gate_ld) or null, out [T, ...] with row stride o_ld and head
// stride Dv.  window 0: all earlier keys.  pool > 0: pooled rows k_pool [pages, pool_rows, Hkv, D], v_pool [.., Dv] in front of the window.
extern "C" int ne_attn_biased(const void* q, long long q_ld, const void* k_cache, const void* v_cache, const int* block_tables, int bt_stride, int block_size,
                              const int* cu_seqlens_q, const int* context_lens, int num_seqs, void* out, long long o_ld, int T, int H, int Hkv, int D, int Dv,
                              float scale, float softcap, const float* slopes, int window, const void* gate, long long gate_ld, float out_scale, int fp32,
                              const void* k_pool, const void* v_pool, int pool, int pool_rows, const float* turn, int n_pos, int keep, cudaStream_t st) {
  if (T <= 0) return 0;
  if (keep > 0 && pool > 0) return 1004;
  if (pool > 0 && (window < 1 || softcap > 0.f || slopes || !k_pool || !v_pool || pool_rows < (block_size + 8 * pool - 1) / (8 * pool) * 8)) return 1004;
  if (turn && (n_pos < 1 || Dv % 2)) return 1005;
  if (Hkv < 1 || H % Hkv || Dv < 1 || Dv > 640 || D < 1 || D > 640) return 1001;
  AttnArgs a;
  memset(&a, 0, sizeof(a));
  a.q = q; a.q_tok_stride = q_ld; a.q_head_stride = D; a.k_cache = k_cache; a.v_cache = v_cache; a.kv_slot_stride = (long long)Hkv * D; a.kv_head_stride = D;
  a.v_slot_stride = (long long)Hkv * Dv; a.v_head_stride = Dv; a.kv_group = H / Hkv; a.block_tables = block_tables; a.bt_stride = bt_stride;
  a.block_size = block_size; a.cu_seqlens_q = cu_seqlens_q; a.context_lens = context_lens; a.num_seqs = num_seqs; a.out = out; a.o_tok_stride = o_ld;
  a.o_head_stride = Dv; a.T = T; a.H = H; a.Dk = D; a.Dv = Dv; a.scale = scale; a.fp8 = fp32 ? 2 : 0; a.window = window; a.softcap = softcap; a.slopes = slopes;
  a.gate = gate; a.gate_ld = gate_ld; a.out_scale = out_scale; a.k_pool = k_pool; a.v_pool = v_pool; a.pool = pool > 0 ? pool : 0; a.pool_rows = pool_rows;
  a.turn = turn; a.n_pos = n_pos; a.keep = window > 0 && keep > 0 ? keep : 0; a.maps = 1;
  for (a.heads_per_cta = kHeadsPerCta; a.kv_group % a.heads_per_cta; a.heads_per_cta--) {}
  return attn_generic_launch(a, st);
}

// Differential form: q [T, H, 2, D] (row stride q_ld), k_cache [slots, Hkv, 2 D], v_cache [slots, Hkv, Dv], mixing fp32 [1], gate [T, H Dv] (row stride
// gate_ld), out [T, H Dv] with row stride o_ld.  window 0: all earlier keys; keep: the first keys stay visible behind the window.
extern "C" int ne_attn_diff(const void* q, long long q_ld, const void* k_cache, const void* v_cache, const int* block_tables, int bt_stride, int block_size,
                            const int* cu_seqlens_q, const int* context_lens, int num_seqs, void* out, long long o_ld, int T, int H, int Hkv, int D, int Dv,
                            float scale, int window, int keep, const float* mixing, float out_scale, float eps, const void* gate, long long gate_ld, int fp32,
                            cudaStream_t st) {
  if (T <= 0) return 0;
  if (Hkv < 1 || H % Hkv || Dv < 1 || Dv > 640 || D < 1 || 2 * D > 640 || !mixing || !gate) return 1001;
  AttnArgs a;
  memset(&a, 0, sizeof(a));
  a.q = q; a.q_tok_stride = q_ld; a.q_head_stride = D; a.k_cache = k_cache; a.v_cache = v_cache; a.kv_slot_stride = (long long)Hkv * 2 * D; a.kv_head_stride = 2 * D;
  a.v_slot_stride = (long long)Hkv * Dv; a.v_head_stride = Dv; a.kv_group = 2 * (H / Hkv); a.block_tables = block_tables; a.bt_stride = bt_stride;
  a.block_size = block_size; a.cu_seqlens_q = cu_seqlens_q; a.context_lens = context_lens; a.num_seqs = num_seqs; a.out = out; a.o_tok_stride = o_ld;
  a.o_head_stride = Dv; a.T = T; a.H = 2 * H; a.Dk = D; a.Dv = Dv; a.scale = scale; a.fp8 = fp32 ? 2 : 0; a.window = window; a.keep = window > 0 && keep > 0 ? keep : 0;
  a.maps = 2; a.mixing = mixing; a.out_scale = out_scale; a.eps = eps; a.egate = gate; a.egate_ld = gate_ld;
  a.heads_per_cta = a.kv_group % 4 ? 2 : 4;
  return attn_generic_launch(a, st);
}

extern "C" int ne_attn_generic(const void* q, long long q_tok_stride, int q_head_stride, const void* k_cache, const void* v_cache,
                               long long kv_slot_stride, int kv_head_stride, int kv_group, const int* block_tables, int bt_stride,
                               int block_size, const int* cu_seqlens_q, const int* context_lens, int num_seqs, const int* sparse, int topk,
                               void* out, long long o_tok_stride, int o_head_stride, float* lse, int T, int H, int Dk, int Dv, float scale,
                               int fp8, int window, int noncausal, cudaStream_t st) {
  if (T <= 0) return 0;
  if (Dv > 640 || (kv_group > 1 && kv_group % kHeadsPerCta != 0)) return 1001;
  AttnArgs a;
  memset(&a, 0, sizeof(a));
  a.q = q; a.q_tok_stride = q_tok_stride; a.q_head_stride = q_head_stride; a.k_cache = k_cache; a.v_cache = v_cache;
  a.kv_slot_stride = kv_slot_stride; a.kv_head_stride = kv_head_stride; a.kv_group = kv_group; a.block_tables = block_tables;
  a.bt_stride = bt_stride; a.block_size = block_size; a.cu_seqlens_q = cu_seqlens_q; a.context_lens = context_lens; a.num_seqs = num_seqs;
  a.sparse = sparse; a.topk = topk; a.out = out; a.o_tok_stride = o_tok_stride; a.o_head_stride = o_head_stride; a.lse = lse;
  a.T = T; a.H = H; a.Dk = Dk; a.Dv = Dv; a.scale = scale; a.fp8 = fp8; a.window = window; a.noncausal = noncausal;
  a.v_slot_stride = kv_slot_stride; a.v_head_stride = kv_head_stride; a.out_scale = 1.f; a.maps = 1;
  // multi-head attention proper (one kv head per query head, separate V): the four query heads of a CTA would need four
  // different key tiles, so a CTA serves one head there
  a.heads_per_cta = (kv_group == 1 && kv_head_stride != 0 && v_cache != nullptr) ? 1 : kHeadsPerCta;
  return attn_generic_launch(a, st);
}

extern "C" int ne_attn_merge(const float* part, const float* lse2, void* out, int splits, long long rows, int D, int out_row_stride, cudaStream_t st) {
  if (rows <= 0) return 0;
  return (int)launch_pdl(attn_merge_kernel, dim3((unsigned)rows), dim3(128), 0, st, part, lse2, (__nv_bfloat16*)out, splits, rows, D, out_row_stride);
}

extern "C" int ne_sample(const float* logits, const float* temps, long long* tok, float* logprob, int rows, int V, unsigned long long seed,
                         cudaStream_t st) {
  if (rows <= 0) return 0;
  return (int)launch_pdl(sample_kernel, dim3(rows), dim3(1024), 0, st, logits, temps, tok, logprob, V, (uint64_t)seed);
}
