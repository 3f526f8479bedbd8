// K10: mixture-of-experts routing, dispatch and combine around the grouped tcgen05 GEMM.
//
//   omni_moe_route     softmax over expert logits, top-k, optional renormalisation
//   omni_moe_router    router product and choice in one launch: fp32 logits with a bias, the top-k largest, softmax
//                      among them, or sigmoid scores divided by their sum, of the best groups of experts (bf16 rows)
//   omni_moe_topk      the same choice from fp32 logits
//   omni_moe_pairs_f32 y[p] = act(W[expert of pair p] x[p / per]) in true fp32 (exact mode)
//   omni_moe_plan      per-expert counts -> segment offsets padded to 128 rows (the GEMM's M
//                      tile), the expert of every M tile, and the row of every (token, k) pair
//   omni_moe_dispatch  copy token rows into the expert-major padded buffer
//   omni_moe_combine   out[t] = sum_k w[t,k] * y[row(t,k)]  (+ optional residual / shared expert)
//
// Padding each expert segment to the 128-row MMA tile keeps every GEMM tile inside one expert,
// so the expert GEMMs are ONE launch of the grouped kernel (gemm_sm100.cu) with a per-tile
// expert index.  The reference reaches vLLM's Triton fused_moe or a Python loop over experts
// (vllm_omni/model_executor/models/qwen3_omni/qwen3_moe.py).
#include "host_util.h"
#include "ptx_sm100.cuh"

namespace omni {

constexpr int MOE_TILE = 128;

// Limits for the checked build (OMNI_IN_BOUNDS in ptx_sm100.cuh; 0 = unknown / unchecked), set by the host
// through omni_moe_set_bounds and passed to the kernels by value: the rows the expert-major buffers hold.
struct MoeBounds {
  long max_rows;
  int* status;
};
static MoeBounds g_moe_bounds = {0, nullptr};
enum { KID_MOE_PLAN = 3, KID_MOE_DISPATCH = 4, KID_MOE_COMBINE = 5 };

// one warp per token; E <= 256 (8 per lane), k <= 16
__global__ void __launch_bounds__(256)
moe_route_kernel(const __nv_bfloat16* __restrict__ logits, int ld, int T, int E, int k, int renorm,
                 int* __restrict__ ids, float* __restrict__ weights) {
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (t >= T) return;
  float v[8];
  float mx = -INFINITY;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int e = lane + i * 32;
    v[i] = e < E ? __bfloat162float(logits[(size_t)t * ld + e]) : -INFINITY;
    mx = fmaxf(mx, v[i]);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) { v[i] = v[i] == -INFINITY ? 0.f : __expf(v[i] - mx); sum += v[i]; }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
  const float inv = 1.0f / sum;
  float picked = 0.f;
  for (int j = 0; j < k; ++j) {
    float best = -1.f;
    int bi = 0x7fffffff;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int e = lane + i * 32;
      if (v[i] > best || (v[i] == best && e < bi)) { best = v[i]; bi = e; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ob = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
    }
    if (lane == 0) { ids[(size_t)t * k + j] = bi; weights[(size_t)t * k + j] = best * inv; }
    picked += best * inv;
    if ((bi & 31) == lane) v[bi >> 5] = -1.f;   // remove the winner
  }
  if (renorm && lane == 0) {
    const float r = 1.0f / fmaxf(picked, 1e-20f);
    for (int j = 0; j < k; ++j) weights[(size_t)t * k + j] *= r;
  }
}

// What turns logits into a choice.  sigmoid = 0: softmax among the k largest.  sigmoid = 1: scores 1 / (1 + e^-z); with
// groups > 0 only the `keep` groups of neighbours with the largest sums of their two best scores take part; weights are
// scale * score / (sum of the chosen scores + 1e-20).
struct RouterRule {
  int sigmoid, groups, keep;
  float scale;
};

// the largest of n <= 256 values, value lane + 32 i in v[i]; ties go to the lower index
__device__ __forceinline__ void warp_best(const float (&v)[8], int n, int lane, float& best, int& bi) {
  best = -INFINITY;
  bi = 0x7fffffff;
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (i * 32 < n) {
      const int e = lane + i * 32;
      if (v[i] > best || (v[i] == best && v[i] != -INFINITY && e < bi)) { best = v[i]; bi = e; }
    }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ob = __shfl_xor_sync(0xffffffffu, best, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (ob > best || (ob == best && oi < bi)) { best = ob; bi = oi; }
  }
}

// Leaves the experts of the kept groups in v (scores), -inf elsewhere.  `sh`: 256 floats of this warp.
__device__ __forceinline__ void keep_groups(float (&v)[8], int E, const RouterRule& rule, int lane, float* sh) {
  const int size = E / rule.groups;
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (lane + i * 32 < E) sh[lane + i * 32] = v[i];
  __syncwarp();
  float sum[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int g = lane + i * 32;
    sum[i] = -INFINITY;
    if (i * 32 < rule.groups && g < rule.groups) {
      float a = sh[g * size], b = size > 1 ? -INFINITY : 0.f;
      for (int j = 1; j < size; ++j) {
        const float x = sh[g * size + j];
        b = fmaxf(b, fminf(a, x));
        a = fmaxf(a, x);
      }
      sum[i] = a + b;
    }
  }
  __syncwarp();
  unsigned live = 0u;
  for (int j = 0; j < rule.keep; ++j) {
    float best;
    int g;
    warp_best(sum, rule.groups, lane, best, g);
    if (g >= rule.groups) break;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int e = lane + i * 32;
      if (e == g) sum[i] = -INFINITY;
      if (i * 32 < E && e >= g * size && e < (g + 1) * size) live |= 1u << i;
    }
  }
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (!(live & (1u << i))) v[i] = -INFINITY;
}

// Choice of one token by one warp from logits v (lane + 32 i holds expert lane + 32 i, -inf past the last), ties to the
// lower index.  E <= 256, k <= 16.  `sh`: 256 floats of this warp (groups only).
__device__ __forceinline__ void choose_experts(float (&v)[8], int E, int k, const RouterRule& rule, int lane, float* sh, int* ids,
                                               float* weights) {
  if (rule.sigmoid) {
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i * 32 < E) v[i] = lane + i * 32 < E ? 1.0f / (1.0f + expf(-v[i])) : -INFINITY;
    if (rule.groups > 0) keep_groups(v, E, rule, lane, sh);
  }
  float top = 0.f, sum = 0.f, mine = 0.f;
  int mine_id = 0;
  for (int j = 0; j < k; ++j) {
    float best;
    int bi;
    warp_best(v, E, lane, best, bi);
    if (bi >= E) bi = j;                       // no finite value left: any index inside the range
    if (j == 0) top = best;
    const float w = rule.sigmoid ? best : expf(best - top);
    sum += w;
    if (lane == j) { mine = w; mine_id = bi; }
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (bi == lane + i * 32) v[i] = -INFINITY;
  }
  if (lane < k) {
    ids[lane] = mine_id;
    weights[lane] = rule.sigmoid ? mine / (sum + 1e-20f) * rule.scale : mine / sum;
  }
}

__global__ void __launch_bounds__(256)
moe_topk_kernel(const float* __restrict__ logits, long ld, int T, int E, int k, RouterRule rule, int* __restrict__ ids,
                float* __restrict__ weights) {
  __shared__ float sh[8][256];
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (t >= T) return;
  float v[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int e = lane + i * 32;
    v[i] = e < E ? logits[t * ld + e] : -INFINITY;
  }
  choose_experts(v, E, k, rule, lane, sh[threadIdx.x >> 5], ids + (long)t * k, weights + (long)t * k);
}

// Router of MT * 16 tokens per block: NW warps share the contraction (each takes every NW-th 32-channel chunk), 64 experts
// at a time; partial sums meet in shared memory in a fixed order.  A warp reads 16 bytes per row and chunk: lane group j
// of a quad owns channels 8 j .. 8 j + 7 of the chunk for both operands, which permutes the contraction alike on both
// sides.
template <int MT, int NW>
__global__ void __launch_bounds__(32 * NW)
moe_router_kernel(const __nv_bfloat16* __restrict__ x, long ldx, const __nv_bfloat16* __restrict__ w, long ldw,
                  const float* __restrict__ bias, int T, int D, int E, int Ep, int k, RouterRule rule,
                  int* __restrict__ ids, float* __restrict__ weights) {
  extern __shared__ float sm[];
  float* part = sm;                            // [NW][MT * 16][64]
  float* logit = sm + NW * MT * 16 * 64;        // [MT * 16][256]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, j = lane & 3;
  const int t0 = blockIdx.x * (MT * 16);
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  for (int e0 = 0; e0 < E; e0 += 64) {
    float acc[MT][8][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[m][n][i] = 0.f;
#pragma unroll(MT == 1 ? 2 : 1)
    for (int c = warp * 32; c < D; c += 32 * NW) {
      const int ch = c + j * 8;
      const bool in = ch < D;                  // D is a multiple of 8
      uint4 a[MT][2];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int t = t0 + m * 16 + h * 8 + g;
          a[m][h] = in && t < T ? *reinterpret_cast<const uint4*>(x + (long)t * ldx + ch) : zero;
        }
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        const int e = e0 + n * 8 + g;
        const uint4 b = in && e < Ep ? *reinterpret_cast<const uint4*>(w + (long)e * ldw + ch) : zero;
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
                       "{%0, %1, %2, %3};"
                       : "+f"(acc[m][n][0]), "+f"(acc[m][n][1]), "+f"(acc[m][n][2]), "+f"(acc[m][n][3])
                       : "r"(a[m][0].x), "r"(a[m][1].x), "r"(a[m][0].y), "r"(a[m][1].y), "r"(b.x), "r"(b.y));
          asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
                       "{%0, %1, %2, %3};"
                       : "+f"(acc[m][n][0]), "+f"(acc[m][n][1]), "+f"(acc[m][n][2]), "+f"(acc[m][n][3])
                       : "r"(a[m][0].z), "r"(a[m][1].z), "r"(a[m][0].w), "r"(a[m][1].w), "r"(b.z), "r"(b.w));
        }
      }
    }
    __syncthreads();                           // the previous group's sums are read
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int h = 0; h < 2; ++h)
          *reinterpret_cast<float2*>(part + ((long)warp * MT * 16 + m * 16 + h * 8 + g) * 64 + n * 8 + j * 2) =
              make_float2(acc[m][n][2 * h], acc[m][n][2 * h + 1]);
    __syncthreads();
    for (int i = threadIdx.x; i < MT * 16 * 64; i += 32 * NW) {
      const int e = e0 + (i & 63);
      if (e < E) {
        float s = bias ? bias[e] : 0.f;
#pragma unroll
        for (int q = 0; q < NW; ++q) s += part[q * MT * 16 * 64 + i];
        logit[(i >> 6) * 256 + e] = s;
      }
    }
  }
  __syncthreads();
  for (int r = warp; r < MT * 16; r += NW) {
    const int t = t0 + r;
    if (t >= T) break;
    float v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = lane + i * 32 < E ? logit[r * 256 + lane + i * 32] : -INFINITY;
    __syncwarp();                              // the row's logits become scratch
    choose_experts(v, E, k, rule, lane, logit + r * 256, ids + (long)t * k, weights + (long)t * k);
  }
}

// Exact mode: one warp per (pair, output); a result is one fixed-order chain plus a fixed-order sum over lanes.
__global__ void __launch_bounds__(256)
moe_pairs_f32_kernel(const float* __restrict__ x, long ldx, int per, const int* __restrict__ ids, const float* __restrict__ w,
                     int E, float* __restrict__ y, long ldy, long pairs, int N, int K, int relu2) {
  const long i = (long)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (i >= pairs * N) return;
  const long p = i / N;
  const int n = (int)(i - p * N);
  const int e = min(max(ids[p], 0), E - 1);
  const float* a = x + (p / per) * ldx;
  const float* b = w + ((long)e * N + n) * K;
  float s = 0.f;
  for (int c = lane; c < K; c += 32) s = fmaf(a[c], b[c], s);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
  if (relu2) {
    s = fmaxf(s, 0.f);
    s *= s;
  }
  if (lane == 0) y[p * ldy + n] = s;
}

// single CTA: histogram, padded prefix sum, tile->expert table, (token,k)->row map.
// counts/cursor live in shared memory (E <= 1024).
__global__ void __launch_bounds__(1024)
moe_plan_kernel(const int* __restrict__ ids, int n_pairs, int E, int e_lo, int e_hi, int max_tiles,
                int* __restrict__ row_of_pair, int* __restrict__ tile_expert, int* __restrict__ offsets,
                int* __restrict__ n_rows_out, MoeBounds bd) {
  __shared__ int cnt[1024];
  __shared__ int off[1025];
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) {
    const int e = ids[i];
    if (!OMNI_IN_BOUNDS(e >= 0 && e < E, bd.status, KID_MOE_PLAN)) continue;
    if (e >= e_lo && e < e_hi) atomicAdd(&cnt[e], 1);
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int acc = 0;
    for (int e = 0; e < E; ++e) {
      off[e] = acc;
      acc += (cnt[e] + MOE_TILE - 1) / MOE_TILE * MOE_TILE;
    }
    off[E] = acc;
    *n_rows_out = acc;
  }
  __syncthreads();
  for (int e = threadIdx.x; e <= E; e += blockDim.x) offsets[e] = off[e];
  for (int tile = threadIdx.x; tile < max_tiles; tile += blockDim.x) {
    // expert owning row tile*128: the last e with off[e] <= row (binary search)
    const int row = tile * MOE_TILE;
    int ex = -1;
    if (row < off[E]) {
      int lo = 0, hi = E - 1;
      while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (off[mid] <= row) lo = mid; else hi = mid - 1;
      }
      ex = lo;
    }
    tile_expert[tile] = ex;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;   // reuse as cursors
  __syncthreads();
  // deterministic placement: pairs are placed in index order per expert by one thread per expert
  // when the batch is small, otherwise by atomics (order inside an expert does not affect results)
  for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) {
    const int e = ids[i];
    row_of_pair[i] = (e >= e_lo && e < e_hi) ? off[e] + atomicAdd(&cnt[e], 1) : -1;
  }
}

// Plan without padding: the rows of expert e are [off[e], off[e] + cnt[e]); expert e owns ceil(cnt[e] / 128)
// M tiles; tile t = (expert, first row, rows <= 128).  Unused tiles get expert -1.
__global__ void __launch_bounds__(1024)
moe_plan_compact_kernel(const int* __restrict__ ids, int n_pairs, int E, int e_lo, int e_hi, int max_tiles,
                        int* __restrict__ row_of_pair, int* __restrict__ tile_expert, int* __restrict__ tile_row0,
                        int* __restrict__ tile_rows, int* __restrict__ n_rows_out, MoeBounds bd) {
  __shared__ int cnt[1024];
  __shared__ int off[1025];
  __shared__ int toff[1025];
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) {
    const int e = ids[i];
    if (!OMNI_IN_BOUNDS(e >= 0 && e < E, bd.status, KID_MOE_PLAN)) continue;
    if (e >= e_lo && e < e_hi) atomicAdd(&cnt[e], 1);
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    int acc = 0, tacc = 0;
    for (int e = 0; e < E; ++e) {
      off[e] = acc;
      toff[e] = tacc;
      acc += cnt[e];
      tacc += (cnt[e] + MOE_TILE - 1) / MOE_TILE;
    }
    off[E] = acc;
    toff[E] = tacc;
    *n_rows_out = acc;
  }
  __syncthreads();
  for (int tile = threadIdx.x; tile < max_tiles; tile += blockDim.x) {
    int ex = -1, r0 = 0, nr = 0;
    if (tile < toff[E]) {
      int lo = 0, hi = E - 1;            // the last e with toff[e] <= tile that owns tiles
      while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (toff[mid] <= tile) lo = mid; else hi = mid - 1;
      }
      ex = lo;
      const int within = tile - toff[ex];
      r0 = off[ex] + within * MOE_TILE;
      nr = min(MOE_TILE, cnt[ex] - within * MOE_TILE);
    }
    tile_expert[tile] = ex;
    tile_row0[tile] = r0;
    tile_rows[tile] = nr;
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) cnt[e] = 0;   // reuse as cursors
  __syncthreads();
  for (int i = threadIdx.x; i < n_pairs; i += blockDim.x) {
    const int e = ids[i];
    row_of_pair[i] = (e >= e_lo && e < e_hi) ? off[e] + atomicAdd(&cnt[e], 1) : -1;
  }
}

// x: [T, D] (pitch ldx) -> xp[row_of_pair[t*k+j], :] ; rows not written stay as they are (the GEMM
// output rows of padding are never read back)
__global__ void __launch_bounds__(256)
moe_dispatch_kernel(const __nv_bfloat16* __restrict__ x, long ldx, const int* __restrict__ row_of_pair, int n_pairs,
                    int k, int D, __nv_bfloat16* __restrict__ xp, MoeBounds bd) {
  const int chunks = D >> 3;
  const long total = (long)n_pairs * chunks;
  for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x) {
    const int p = (int)(i / chunks);
    const int c = (int)(i % chunks) * 8;
    const int r = row_of_pair[p];
    if (r < 0) continue;
    if (!OMNI_IN_BOUNDS(bd.max_rows == 0 || r < bd.max_rows, bd.status, KID_MOE_DISPATCH)) continue;
    *reinterpret_cast<uint4*>(xp + (size_t)r * D + c) = *reinterpret_cast<const uint4*>(x + (size_t)(p / k) * ldx + c);
  }
}

// out[t, :] = (residual[t, :]) + sum_j w[t,j] * y[row(t,j), :]; pairs with row < 0 (experts of
// another rank) contribute nothing.
__global__ void __launch_bounds__(256)
moe_combine_kernel(const __nv_bfloat16* __restrict__ y, const int* __restrict__ row_of_pair,
                   const float* __restrict__ weights, int T, int k, int D, const __nv_bfloat16* __restrict__ residual,
                   long ldr, __nv_bfloat16* __restrict__ out, long ldo, MoeBounds bd) {
  const int chunks = D >> 3;
  const long total = (long)T * chunks;
  for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x) {
    const int t = (int)(i / chunks);
    const int c = (int)(i % chunks) * 8;
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (residual) {
      const uint4 u = *reinterpret_cast<const uint4*>(residual + (size_t)t * ldr + c);
      const float2 a = unpack_bf16(u.x), b = unpack_bf16(u.y), cc = unpack_bf16(u.z), d = unpack_bf16(u.w);
      acc[0] = a.x; acc[1] = a.y; acc[2] = b.x; acc[3] = b.y; acc[4] = cc.x; acc[5] = cc.y; acc[6] = d.x; acc[7] = d.y;
    }
    for (int j = 0; j < k; ++j) {
      const int r = row_of_pair[(size_t)t * k + j];
      if (r < 0) continue;
      if (!OMNI_IN_BOUNDS(bd.max_rows == 0 || r < bd.max_rows, bd.status, KID_MOE_COMBINE)) continue;
      const float w = weights[(size_t)t * k + j];
      const uint4 u = *reinterpret_cast<const uint4*>(y + (size_t)r * D + c);
      const float2 a = unpack_bf16(u.x), b = unpack_bf16(u.y), cc = unpack_bf16(u.z), d = unpack_bf16(u.w);
      acc[0] += w * a.x; acc[1] += w * a.y; acc[2] += w * b.x; acc[3] += w * b.y;
      acc[4] += w * cc.x; acc[5] += w * cc.y; acc[6] += w * d.x; acc[7] += w * d.y;
    }
    uint4 o;
    o.x = pack_bf16(acc[0], acc[1]); o.y = pack_bf16(acc[2], acc[3]);
    o.z = pack_bf16(acc[4], acc[5]); o.w = pack_bf16(acc[6], acc[7]);
    *reinterpret_cast<uint4*>(out + (size_t)t * ldo + c) = o;
  }
}

// Expert-parallel combine: the weighted sum of THIS rank's experts for token t is a partial result;
// it is stored straight into the slot this rank owns on the rank that owns token t's row block
// (peer_out[t / rows_per_owner], local row t % rows_per_owner, pitch D), so the cross-rank sum needs
// no separate all-reduce of a [T, D] tensor: a local reduce kernel finishes it (tp_reduce.cu).
struct MoePeers {
  __nv_bfloat16* out[16];
};
__global__ void __launch_bounds__(256)
moe_combine_scatter_kernel(const __nv_bfloat16* __restrict__ y, const int* __restrict__ row_of_pair,
                           const float* __restrict__ weights, int T, int k, int D, int rows_per_owner, MoePeers peers,
                           MoeBounds bd) {
  const int chunks = D >> 3;
  const long total = (long)T * chunks;
  for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x) {
    const int t = (int)(i / chunks);
    const int c = (int)(i % chunks) * 8;
    float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    for (int j = 0; j < k; ++j) {
      const int r = row_of_pair[(size_t)t * k + j];
      if (r < 0) continue;
      if (!OMNI_IN_BOUNDS(bd.max_rows == 0 || r < bd.max_rows, bd.status, KID_MOE_COMBINE)) continue;
      const float w = weights[(size_t)t * k + j];
      const uint4 u = *reinterpret_cast<const uint4*>(y + (size_t)r * D + c);
      const float2 a = unpack_bf16(u.x), b = unpack_bf16(u.y), cc = unpack_bf16(u.z), d = unpack_bf16(u.w);
      acc[0] += w * a.x; acc[1] += w * a.y; acc[2] += w * b.x; acc[3] += w * b.y;
      acc[4] += w * cc.x; acc[5] += w * cc.y; acc[6] += w * d.x; acc[7] += w * d.y;
    }
    uint4 o;
    o.x = pack_bf16(acc[0], acc[1]); o.y = pack_bf16(acc[2], acc[3]);
    o.z = pack_bf16(acc[4], acc[5]); o.w = pack_bf16(acc[6], acc[7]);
    const int owner = t / rows_per_owner;
    *reinterpret_cast<uint4*>(peers.out[owner] + (size_t)(t - owner * rows_per_owner) * D + c) = o;
  }
}

}  // namespace omni

using namespace omni;
typedef __nv_bfloat16 bf16;

// 1 when this library was compiled with -DOMNI_BOUNDS_CHECK
extern "C" int omni_moe_bounds_check_enabled(void) {
#ifdef OMNI_BOUNDS_CHECK
  return 1;
#else
  return 0;
#endif
}

extern "C" void omni_moe_set_bounds(long max_rows, int* status) {
  g_moe_bounds.max_rows = max_rows;
  g_moe_bounds.status = status;
}

extern "C" int omni_moe_combine_scatter(const void* y, const int* row_of_pair, const float* weights, int T, int k, int D,
                                        int rows_per_owner, void* const* peer_out, void* stream) {
  if (T <= 0) return RC_OK;
  if ((D & 7) || rows_per_owner <= 0 || peer_out == nullptr) return RC_BAD_ARG;
  const int owners = (T + rows_per_owner - 1) / rows_per_owner;
  if (owners > 16) return RC_BAD_ARG;
  MoePeers peers;
  for (int i = 0; i < 16; ++i) peers.out[i] = i < owners ? static_cast<__nv_bfloat16*>(peer_out[i]) : nullptr;
  long blocks = ((long)T * (D >> 3) + 255) / 256;
  if (blocks > 148 * 8) blocks = 148 * 8;
  moe_combine_scatter_kernel<<<(unsigned)blocks, 256, 0, (cudaStream_t)stream>>>(
      (const __nv_bfloat16*)y, row_of_pair, weights, T, k, D, rows_per_owner, peers, g_moe_bounds);
  return (int)cudaGetLastError();
}

extern "C" int omni_moe_route(const void* logits, int ld, int T, int E, int k, int renorm, int* ids, float* weights,
                              void* stream) {
  if (T <= 0) return RC_OK;
  if (E > 256 || k > 16 || k > E) return RC_BAD_ARG;
  moe_route_kernel<<<(T + 7) / 8, 256, 0, (cudaStream_t)stream>>>((const __nv_bfloat16*)logits, ld, T, E, k, renorm, ids, weights);
  return (int)cudaGetLastError();
}

static bool router_rule_ok(const RouterRule& r, int E, int k) {
  if (E > 256 || E < 1 || k > 16 || k > E || k < 1) return false;
  return r.groups == 0 || (r.sigmoid && r.groups > 0 && E % r.groups == 0 && r.keep >= 1 && r.keep <= r.groups && r.keep * (E / r.groups) >= k);
}

extern "C" int omni_moe_topk(const float* logits, long ld, int T, int E, int k, const RouterRule* rule, int* ids, float* weights,
                             void* stream) {
  if (T <= 0) return RC_OK;
  if (!router_rule_ok(*rule, E, k)) return RC_BAD_ARG;
  moe_topk_kernel<<<(T + 7) / 8, 256, 0, (cudaStream_t)stream>>>(logits, ld, T, E, k, *rule, ids, weights);
  return (int)cudaGetLastError();
}

// x [T, D] and w [Ep >= E, D] bf16 (D, pitches multiples of 8), bias [E] fp32 or null.
extern "C" int omni_moe_router(const void* x, long ldx, const void* w, long ldw, const float* bias, int T, int D, int E, int Ep,
                               int k, const RouterRule* rule, int* ids, float* weights, void* stream) {
  if (T <= 0) return RC_OK;
  if (!router_rule_ok(*rule, E, k) || D <= 0 || (D & 7) || (ldx & 7) || (ldw & 7)) return RC_BAD_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  const bf16* xb = (const bf16*)x;
  const bf16* wb = (const bf16*)w;
  static unsigned long long prep[2] = {0, 0};
  if (T > 148 * 16) {
    const int smem = (8 * 32 * 64 + 32 * 256) * 4;
    if (int e = ensure_dynamic_smem((const void*)moe_router_kernel<2, 8>, smem, prep[0])) return e;
    moe_router_kernel<2, 8><<<(T + 31) / 32, 256, smem, st>>>(xb, ldx, wb, ldw, bias, T, D, E, Ep, k, *rule, ids, weights);
  } else {
    const int smem = (16 * 16 * 64 + 16 * 256) * 4;
    if (int e = ensure_dynamic_smem((const void*)moe_router_kernel<1, 16>, smem, prep[1])) return e;
    moe_router_kernel<1, 16><<<(T + 15) / 16, 512, smem, st>>>(xb, ldx, wb, ldw, bias, T, D, E, Ep, k, *rule, ids, weights);
  }
  return (int)cudaGetLastError();
}

// Pair p reads row p / per of x.
extern "C" int omni_moe_pairs_f32(const float* x, long ldx, int per, const int* ids, const float* w, int E, float* y, long ldy,
                                  long pairs, int N, int K, int relu2, void* stream) {
  if (pairs <= 0 || N <= 0) return RC_OK;
  if (per < 1 || E < 1 || K < 1) return RC_BAD_ARG;
  const long blocks = (pairs * N + 7) / 8;
  if (blocks > 0x7fffffffL) return RC_BAD_ARG;
  moe_pairs_f32_kernel<<<(unsigned)blocks, 256, 0, (cudaStream_t)stream>>>(x, ldx, per, ids, w, E, y, ldy, pairs, N, K, relu2);
  return (int)cudaGetLastError();
}

// Experts [e_lo, e_hi) are local (expert parallelism); others get row -1.
// max_tiles: capacity of tile_expert = ceil((n_pairs + E*127) / 128).
extern "C" int omni_moe_plan(const int* ids, int n_pairs, int E, int e_lo, int e_hi, int max_tiles, int* row_of_pair,
                             int* tile_expert, int* offsets, int* n_rows_out, void* stream) {
  if (E > 1024) return RC_BAD_ARG;
  moe_plan_kernel<<<1, 1024, 0, (cudaStream_t)stream>>>(ids, n_pairs, E, e_lo, e_hi, max_tiles, row_of_pair, tile_expert, offsets, n_rows_out,
                                                        g_moe_bounds);
  return (int)cudaGetLastError();
}

extern "C" int omni_moe_plan_compact(const int* ids, int n_pairs, int E, int e_lo, int e_hi, int max_tiles, int* row_of_pair,
                                     int* tile_expert, int* tile_row0, int* tile_rows, int* n_rows_out, void* stream) {
  if (E > 1024) return RC_BAD_ARG;
  moe_plan_compact_kernel<<<1, 1024, 0, (cudaStream_t)stream>>>(ids, n_pairs, E, e_lo, e_hi, max_tiles, row_of_pair, tile_expert,
                                                                tile_row0, tile_rows, n_rows_out, g_moe_bounds);
  return (int)cudaGetLastError();
}

extern "C" int omni_moe_dispatch(const void* x, long ldx, const int* row_of_pair, int n_pairs, int k, int D, void* xp,
                                 void* stream) {
  if (n_pairs <= 0) return RC_OK;
  if (D & 7) return RC_BAD_ARG;
  long blocks = ((long)n_pairs * (D >> 3) + 255) / 256;
  if (blocks > 148 * 8) blocks = 148 * 8;
  moe_dispatch_kernel<<<(unsigned)blocks, 256, 0, (cudaStream_t)stream>>>((const __nv_bfloat16*)x, ldx, row_of_pair, n_pairs, k, D, (__nv_bfloat16*)xp,
                                                                          g_moe_bounds);
  return (int)cudaGetLastError();
}

extern "C" int omni_moe_combine(const void* y, const int* row_of_pair, const float* weights, int T, int k, int D,
                                const void* residual, long ldr, void* out, long ldo, void* stream) {
  if (T <= 0) return RC_OK;
  if (D & 7) return RC_BAD_ARG;
  long blocks = ((long)T * (D >> 3) + 255) / 256;
  if (blocks > 148 * 8) blocks = 148 * 8;
  moe_combine_kernel<<<(unsigned)blocks, 256, 0, (cudaStream_t)stream>>>(
      (const __nv_bfloat16*)y, row_of_pair, weights, T, k, D, (const __nv_bfloat16*)residual, ldr, (__nv_bfloat16*)out, ldo,
      g_moe_bounds);
  return (int)cudaGetLastError();
}
