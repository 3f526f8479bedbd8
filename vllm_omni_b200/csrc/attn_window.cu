// Windowed paged attention (see attn_window.h for what is computed).
//
//   omni_attn_window_rows    one block per (row, head), CUDA cores, bf16 or fp32: the exact mode, and head
//                            sizes the tensor-core kernels are not built for
//   omni_attn_window_decode  sequences with one new token, bf16: the query heads that share a KV head are
//                            the rows of 16 x 8 x 16 tensor-core products, four warps stream disjoint
//                            16-key tiles of the VISIBLE keys only (kept first tokens, then the window)
//                            through a three-deep cp.async ring, shares of the keys can go to several
//                            blocks (split) and are merged by a second kernel
//
// A decode step reads every visible K/V byte once and does little arithmetic on it, so the warp-level
// products (which need no operand staging through tensor memory) suffice; prompts run on the tcgen05
// kernel in attn_window_sm100.cu.
#include "attn_window.h"
#include "host_util.h"
#include "ptx_sm100.cuh"

namespace omni {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float wa_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float wa_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float wa_lg2(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ int wa_page(const WinAttn& p, int seq, int j) {
  const int pg = p.block_tables[(long)seq * p.bt_stride + j / p.block_size];
  return min(max(pg, 0), p.num_blocks - 1);
}

// opening of the output gate at channel c of head h (bf16 logits)
__device__ __forceinline__ float wa_gate(const WinAttn& p, int row, int h, int c) {
  if (!p.gate) return 1.f;
  return 1.0f / (1.0f + __expf(-(float)static_cast<const __nv_bfloat16*>(p.gate)[(long)row * p.g_rs + (long)h * p.g_hs + (long)c * p.g_cs]));
}

// ------------------------------------------------------------------- one block per (row, head)
template <typename T, int NACC>
__global__ void __launch_bounds__(128)
attn_window_rows_kernel(WinAttn p) {
  extern __shared__ float sm[];
  float* sq = sm;                       // [dp]
  float* sacc = sm + p.dp;              // [4][vp]
  float* sfirst = sacc + 4 * p.vp;      // [vp]: the first map's result (two maps only)
  __shared__ float s_m[4], s_l[4], s_ss[4];
  const int row = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = min(max(p.row_seq[row], 0), p.num_seqs - 1);
  const int pos = p.context[seq] + row - p.q_start[seq];
  const int g = h / (p.H / p.G);
  const int R = p.H / p.G, n_maps = p.maps == 2 ? 2 : 1;
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int nf = min(p.keep_first, lo);
  const int n = nf + pos - lo + 1;
  const float r1 = p.r1 ? p.r1[h] : 0.f, r2 = p.r1 ? p.r2[h] : 0.f;
  const T* gate = p.gate ? static_cast<const T*>(p.gate) + (long)row * p.g_rs + (long)h * p.g_hs : nullptr;
  T* o = static_cast<T*>(p.out) + (long)row * p.o_rs + (long)h * p.vp;
  for (int map = 0; map < n_maps; ++map) {
    const int qh = n_maps == 2 ? (2 * g + map) * R + h - g * R : h;
    const T* q = static_cast<const T*>(p.q) + (long)row * p.q_rs + (long)qh * p.dp;
    __syncthreads();                    // the first map's queries and sums are read
    for (int c = threadIdx.x; c < p.dp; c += 128) sq[c] = (float)q[c];
    __syncthreads();
    float m = -INFINITY, l = 0.f, acc[NACC];
#pragma unroll
    for (int i = 0; i < NACC; ++i) acc[i] = 0.f;
    for (int v = warp; v < n; v += 4) {
      const int j = v < nf ? v : lo + v - nf;
      const long slot = (long)wa_page(p, seq, j) * p.block_size + j % p.block_size;
      const T* k = static_cast<const T*>(p.k_cache) + slot * p.k_ts + (long)(g * n_maps + map) * p.dp;
      float d = 0.f;
      for (int c = lane; c < p.dp; c += 32) d = fmaf(sq[c], (float)k[c], d);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) d += __shfl_xor_sync(0xffffffffu, d, o);
      float s = d * p.scale;
      if (p.cap > 0.f) s = p.cap * tanhf(s / p.cap);
      if (p.r1) s -= r1 * logf(1.0f + r2 * (float)(pos - j));
      const float mn = fmaxf(m, s);
      const float a = expf(m - mn), e = expf(s - mn);
      l = l * a + e;
      m = mn;
      const T* vv = static_cast<const T*>(p.v_cache) + slot * p.v_ts + (long)g * p.vp;
#pragma unroll
      for (int i = 0; i < NACC; ++i) {
        const int c = lane + 32 * i;
        if (c < p.vp) acc[i] = fmaf(acc[i], a, e * (float)vv[c]);
      }
    }
    if (lane == 0) { s_m[warp] = m; s_l[warp] = l; }
#pragma unroll
    for (int i = 0; i < NACC; ++i) {
      const int c = lane + 32 * i;
      if (c < p.vp) sacc[warp * p.vp + c] = acc[i];
    }
    __syncthreads();
    float top = fmaxf(fmaxf(s_m[0], s_m[1]), fmaxf(s_m[2], s_m[3]));
    if (p.sink) top = fmaxf(top, p.sink[h]);
    float den = p.sink ? expf(p.sink[h] - top) : 0.f;
    float wgt[4];
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      wgt[w] = s_m[w] == -INFINITY ? 0.f : expf(s_m[w] - top);
      den += s_l[w] * wgt[w];
    }
    const float f = 1.0f / den;
    float ss = 0.f;
    for (int c = threadIdx.x; c < p.vp; c += 128) {
      float t = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) t = fmaf(sacc[w * p.vp + c], wgt[w], t);
      t *= f;
      if (n_maps == 1) {
        if (gate) t *= 1.0f / (1.0f + expf(-(float)gate[(long)c * p.g_cs]));
        o[c] = (T)t;
      } else if (map == 0) {
        sfirst[c] = t;
      } else {
        t = sfirst[c] - p.lam * t;
        sfirst[c] = t;
        ss = fmaf(t, t, ss);
      }
    }
    if (map == 1) {
#pragma unroll
      for (int u = 16; u > 0; u >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, u);
      if (lane == 0) s_ss[warp] = ss;
      __syncthreads();
      const float mul = p.out_mul / sqrtf(((s_ss[0] + s_ss[1]) + (s_ss[2] + s_ss[3])) / (float)p.vdim + p.out_eps);
      for (int c = threadIdx.x; c < p.vp; c += 128) {
        float t = sfirst[c] * mul;
        if (gate) t *= 1.0f / (1.0f + expf(-(float)gate[(long)c * p.g_cs]));
        o[c] = (T)t;
      }
    }
  }
}

// ---------------------------------------------------------------------------------- decode
constexpr int WD_STAGES = 3;
constexpr int WD_KEYS = 16;      // keys per warp tile

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma_16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
               "{%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// KS / VS: 16-channel steps of the key and value heads this instance has registers for (dp <= 16 KS,
// vp <= 16 VS).  UP: more than eight query heads per KV head, so rows 8..15 of the tile are live.  PAIR: two maps; rows
// 0..7 of the tile are the first map of eight heads, rows 8..15 the second; a key row holds both maps, each product
// takes the rows of one map and both add into the same tile of scores, so that values are read once.
template <int KS, int VS, bool UP, bool PAIR>
__global__ void __launch_bounds__(128, KS <= 8 && !PAIR ? 3 : 1)
attn_window_decode_kernel(WinAttn p) {
  constexpr int HB = PAIR ? 8 : 16;                         // heads per block
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float s_m[4][16], s_l[4][16];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int R = p.H / p.G, hgroups = (R + HB - 1) / HB;
  const int g = blockIdx.y / hgroups, h0 = g * R + (blockIdx.y % hgroups) * HB;
  const int nh = min(HB, (g + 1) * R - h0);                // live heads of the tile
  const int split = blockIdx.z;
  const int seq = min(max(p.seq_list[blockIdx.x], 0), p.num_seqs - 1);
  const int row = p.q_start[seq];
  const int pos = p.context[seq];
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int nf = min(p.keep_first, lo);
  const int n_vis = nf + pos - lo + 1;
  const int tiles_all = (n_vis + WD_KEYS - 1) / WD_KEYS;
  const int per = (tiles_all + p.splits - 1) / p.splits;
  const int t0 = min(tiles_all, split * per), t1 = min(tiles_all, t0 + per);

  const int kw = PAIR ? 2 * p.dp : p.dp;                      // channels of a key row
  const int kpitch = kw * 2 + 16, vpitch = p.vp * 2 + 16;     // odd multiples of 16 B: conflict-free ldmatrix
  const int stage_bytes = WD_KEYS * (kpitch + vpitch);
  const uint32_t base = smem_u32(smem) + warp * WD_STAGES * stage_bytes;
  const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(p.k_cache);
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(p.v_cache);

  // copy of one 16-key tile: eight lanes per key row, 16 bytes per lane
  auto fetch = [&](int t, int st) {
    const uint32_t kd = base + st * stage_bytes, vd = kd + WD_KEYS * kpitch;
    const int l8 = lane & 7;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = i * 4 + (lane >> 3);
      const int v = min(t * WD_KEYS + r, n_vis - 1);          // past the end: a valid key, masked below
      const int j = v < nf ? v : lo + v - nf;
      const long slot = (long)wa_page(p, seq, j) * p.block_size + j % p.block_size;
      const __nv_bfloat16* ks = kc + slot * p.k_ts + (long)g * kw;
      const __nv_bfloat16* vs = vc + slot * p.v_ts + (long)g * p.vp;
      for (int c = l8 * 8; c < kw; c += 64) cp_async16(kd + r * kpitch + c * 2, ks + c);
      for (int c = l8 * 8; c < p.vp; c += 64) cp_async16(vd + r * vpitch + c * 2, vs + c);
    }
  };

  // query heads as the A operand: rows lane / 4 (and + 8), channel pairs
  uint32_t qa[KS][4];
  {
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q) + (long)row * p.q_rs;
    const int ra = lane >> 2, rb = ra + 8, c0 = (lane & 3) * 2;
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      const bool in = k * 16 < p.dp;
      const int ha = PAIR ? 2 * g * R + h0 - g * R + ra : h0 + ra, hb = PAIR ? ha + R : h0 + rb;
      const bool in_b = UP && in && (PAIR ? ra : rb) < nh;
      const __nv_bfloat16* qr = q + (long)ha * p.dp + k * 16 + c0;
      const __nv_bfloat16* qs = q + (long)hb * p.dp + k * 16 + c0;
      qa[k][0] = in && ra < nh ? *reinterpret_cast<const uint32_t*>(qr) : 0u;
      qa[k][2] = in && ra < nh ? *reinterpret_cast<const uint32_t*>(qr + 8) : 0u;
      qa[k][1] = in_b ? *reinterpret_cast<const uint32_t*>(qs) : 0u;
      qa[k][3] = in_b ? *reinterpret_cast<const uint32_t*>(qs + 8) : 0u;
    }
  }
  float r1[2] = {0.f, 0.f}, r2[2] = {0.f, 0.f};
  if (p.r1) {
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const int r = (lane >> 2) + 8 * u;
      if (r < nh) { r1[u] = p.r1[h0 + r]; r2[u] = p.r2[h0 + r]; }
    }
  }
  const bool capped = p.cap > 0.f;
  const float C = p.cap * LOG2E;
  const float s_mul = capped ? p.scale * 2.0f * LOG2E / p.cap : p.scale * LOG2E;

  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, acc[2 * VS][4];
#pragma unroll
  for (int i = 0; i < 2 * VS; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;

  int tf = t0 + warp;                                       // next tile to fetch
#pragma unroll
  for (int s = 0; s < WD_STAGES - 1; ++s, tf += 4) {
    if (tf < t1) fetch(tf, s);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  int st = 0, sf = WD_STAGES - 1;
  for (int t = t0 + warp; t < t1; t += 4) {
    if (tf < t1) fetch(tf, sf);
    tf += 4;
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group %0;" ::"n"(WD_STAGES - 1) : "memory");
    __syncwarp();
    const uint32_t kd = base + st * stage_bytes, vd = kd + WD_KEYS * kpitch;
    float s[2][4] = {};
    {
      // matrices: keys 0-7 ch 0-7 | keys 0-7 ch 8-15 | keys 8-15 ch 0-7 | keys 8-15 ch 8-15
      const uint32_t a0 = kd + ((lane & 7) + ((lane >> 4) << 3)) * kpitch + ((lane >> 3) & 1) * 16;
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        if (k * 16 < p.dp) {
          uint32_t b[4];
          ldsm4(a0 + k * 32, b);
          if (PAIR) {
            const uint32_t first[4] = {qa[k][0], 0u, qa[k][2], 0u}, second[4] = {0u, qa[k][1], 0u, qa[k][3]};
            mma_16816(s[0], first, b[0], b[1]);
            mma_16816(s[1], first, b[2], b[3]);
            ldsm4(a0 + p.dp * 2 + k * 32, b);
            mma_16816(s[0], second, b[0], b[1]);
            mma_16816(s[1], second, b[2], b[3]);
          } else {
            mma_16816(s[0], qa[k], b[0], b[1]);
            mma_16816(s[1], qa[k], b[2], b[3]);
          }
        }
      }
    }
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int u = e >> 1;
        if (!UP && u == 1) { s[nt][e] = 0.f; continue; }
        const int v = t * WD_KEYS + nt * 8 + (lane & 3) * 2 + (e & 1);
        const int j = v < nf ? v : lo + v - nf;
        float y = s[nt][e] * s_mul;
        if (capped) y = fmaf(-2.0f * C, wa_rcp(wa_ex2(y) + 1.0f), C);
        if (p.r1) y -= r1[u] * wa_lg2(fmaf(r2[u], (float)(pos - j), 1.0f));
        y = v < n_vis ? y : -INFINITY;
        s[nt][e] = y;
        mx[u] = fmaxf(mx[u], y);
      }
    float alpha[2] = {1.f, 1.f};
#pragma unroll
    for (int u = 0; u < (UP ? 2 : 1); ++u) {
      mx[u] = fmaxf(mx[u], __shfl_xor_sync(0xffffffffu, mx[u], 1));
      mx[u] = fmaxf(mx[u], __shfl_xor_sync(0xffffffffu, mx[u], 2));
      const float mn = fmaxf(m[u], mx[u]);                  // finite: a tile holds at least one visible key
      alpha[u] = wa_ex2(m[u] - mn);
      m[u] = mn;
      l[u] *= alpha[u];
    }
    uint32_t pa[4];
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        float e0 = 0.f, e1 = 0.f;
        if (UP || u == 0) {
          e0 = wa_ex2(s[nt][2 * u] - m[u]);
          e1 = wa_ex2(s[nt][2 * u + 1] - m[u]);
          l[u] += e0 + e1;
        }
        pa[nt * 2 + u] = pack_bf16(e0, e1);
      }
#pragma unroll
    for (int i = 0; i < 2 * VS; ++i) {
      acc[i][0] *= alpha[0]; acc[i][1] *= alpha[0];
      if (UP) { acc[i][2] *= alpha[1]; acc[i][3] *= alpha[1]; }
    }
    {
      // transposed matrices: keys 0-7 ch 0-7 | keys 8-15 ch 0-7 | keys 0-7 ch 8-15 | keys 8-15 ch 8-15
      const uint32_t a0 = vd + ((lane & 7) + (((lane >> 3) & 1) << 3)) * vpitch + (lane >> 4) * 16;
#pragma unroll
      for (int k = 0; k < VS; ++k) {
        if (k * 16 < p.vp) {
          uint32_t b[4];
          ldsm4_t(a0 + k * 32, b);
          mma_16816(acc[2 * k], pa, b[0], b[1]);
          mma_16816(acc[2 * k + 1], pa, b[2], b[3]);
        }
      }
    }
    __syncwarp();                                           // the stage may be refilled
    st = st + 1 == WD_STAGES ? 0 : st + 1;
    sf = sf + 1 == WD_STAGES ? 0 : sf + 1;
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();                                          // every warp is done with its ring
  float* sacc = reinterpret_cast<float*>(smem);             // [4][16][vp]
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    l[u] += __shfl_xor_sync(0xffffffffu, l[u], 1);
    l[u] += __shfl_xor_sync(0xffffffffu, l[u], 2);
    const int r = (lane >> 2) + 8 * u;
    if ((lane & 3) == 0) { s_m[warp][r] = m[u]; s_l[warp][r] = l[u]; }
    if ((PAIR ? r & 7 : r) < nh) {
#pragma unroll
      for (int i = 0; i < 2 * VS; ++i)
        if (i * 8 < p.vp)
          *reinterpret_cast<float2*>(sacc + (warp * 16 + r) * p.vp + i * 8 + (lane & 3) * 2) =
              make_float2(acc[i][2 * u], acc[i][2 * u + 1]);
    }
  }
  __syncthreads();
  // channel c of tile row r over the four warps: weighted sum, reference exponent and denominator
  auto gather = [&](int r, int c, float sk, float& top, float& den) {
    top = fmaxf(fmaxf(fmaxf(s_m[0][r], s_m[1][r]), fmaxf(s_m[2][r], s_m[3][r])), sk);
    float o = 0.f;
    den = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float a = s_m[w][r] == -INFINITY ? 0.f : wa_ex2(s_m[w][r] - top);
      den = fmaf(s_l[w][r], a, den);
      o = fmaf(sacc[(w * 16 + r) * p.vp + c], a, o);
    }
    return o;
  };
  if (p.splits > 1) {
    const int maps = PAIR ? 2 : 1;
    for (int idx = threadIdx.x; idx < maps * nh * p.vp; idx += 128) {
      const int i = idx / p.vp, c = idx - i * p.vp, map = i / nh, h = h0 + i - map * nh;
      float top, den;
      const float o = gather(map * 8 + i - map * nh, c, -INFINITY, top, den);
      const long pi = (((long)blockIdx.x * p.H + h) * maps + map) * p.splits + split;
      p.part_o[pi * p.vp + c] = o;
      if (c == 0) { p.part_ml[2 * pi] = top; p.part_ml[2 * pi + 1] = den; }
    }
  } else if (PAIR) {
    for (int r = warp; r < nh; r += 4) {                     // a warp owns a head: lanes over channels
      float u[VS / 2], ss = 0.f;
#pragma unroll
      for (int i = 0; i < VS / 2; ++i) {
        const int c = lane + 32 * i;
        u[i] = 0.f;
        if (c < p.vp) {
          float top, d1, d2;
          const float o1 = gather(r, c, -INFINITY, top, d1), o2 = gather(8 + r, c, -INFINITY, top, d2);
          u[i] = o1 / d1 - p.lam * (o2 / d2);
        }
        ss = fmaf(u[i], u[i], ss);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float f = p.out_mul / sqrtf(ss / (float)p.vdim + p.out_eps);
#pragma unroll
      for (int i = 0; i < VS / 2; ++i) {
        const int c = lane + 32 * i;
        if (c < p.vp)
          static_cast<__nv_bfloat16*>(p.out)[(long)row * p.o_rs + (long)(h0 + r) * p.vp + c] = __float2bfloat16(u[i] * f * wa_gate(p, row, h0 + r, c));
      }
    }
  } else {
    for (int idx = threadIdx.x; idx < nh * p.vp; idx += 128) {
      const int r = idx / p.vp, c = idx - r * p.vp, h = h0 + r;
      const float sk = p.sink ? p.sink[h] * LOG2E : -INFINITY;
      float top, den;
      const float o = gather(r, c, sk, top, den);
      den += p.sink ? wa_ex2(sk - top) : 0.f;
      static_cast<__nv_bfloat16*>(p.out)[(long)row * p.o_rs + (long)h * p.vp + c] = __float2bfloat16(o / den * wa_gate(p, row, h, c));
    }
  }
}

__global__ void __launch_bounds__(256)
attn_window_merge_kernel(WinAttn p) {
  const int seq = min(max(p.seq_list[blockIdx.x], 0), p.num_seqs - 1), h = blockIdx.y;
  const int row = p.q_start[seq];
  const int maps = p.maps == 2 ? 2 : 1;
  const float sk = p.sink ? p.sink[h] * LOG2E : -INFINITY;
  float f[2] = {0.f, 0.f}, top[2] = {sk, sk};
  const long base = ((long)blockIdx.x * p.H + h) * maps * p.splits;
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    if (m >= maps) break;
    const long b = base + (long)m * p.splits;
    for (int s = 0; s < p.splits; ++s) top[m] = fmaxf(top[m], p.part_ml[2 * (b + s)]);
    float den = p.sink ? wa_ex2(sk - top[m]) : 0.f;
    for (int s = 0; s < p.splits; ++s) {
      const float ms = p.part_ml[2 * (b + s)];
      den += ms == -INFINITY ? 0.f : p.part_ml[2 * (b + s) + 1] * wa_ex2(ms - top[m]);
    }
    f[m] = 1.0f / den;
  }
  const int c = threadIdx.x;                                // one channel per thread
  float o[2] = {0.f, 0.f};
#pragma unroll
  for (int m = 0; m < 2; ++m) {
    if (m >= maps || c >= p.vp) break;
    const long b = base + (long)m * p.splits;
    for (int s = 0; s < p.splits; ++s) {
      const float ms = p.part_ml[2 * (b + s)];
      if (ms != -INFINITY) o[m] = fmaf(p.part_o[(b + s) * p.vp + c], wa_ex2(ms - top[m]), o[m]);
    }
  }
  float r = o[0] * f[0];
  if (maps == 2) {
    __shared__ float sh[32];
    r -= p.lam * (o[1] * f[1]);
    float ss = r * r;
#pragma unroll
    for (int i = 16; i > 0; i >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, i);
    if ((threadIdx.x & 31) == 0) sh[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
    for (int w = 0; w < (int)(blockDim.x >> 5); ++w) ss += sh[w];
    r *= p.out_mul / sqrtf(ss / (float)p.vdim + p.out_eps);
  }
  if (c < p.vp)
    static_cast<__nv_bfloat16*>(p.out)[(long)row * p.o_rs + (long)h * p.vp + c] = __float2bfloat16(r * wa_gate(p, row, h, c));
}

static bool win_args_ok(const WinAttn& p) {
  return p.H > 0 && p.G > 0 && p.H % p.G == 0 && (p.dp & 15) == 0 && (p.vp & 15) == 0 && p.dp > 0 && p.vp > 0 &&
         p.num_seqs > 0 && p.num_blocks > 0 && p.block_size > 0 && p.keep_first >= 0 && p.k_ts > 0 && p.v_ts > 0 && p.dp_u == p.dp &&
         p.key_start == nullptr && (p.r1 == nullptr) == (p.r2 == nullptr) && (p.maps != 2 || (p.vdim > 0 && p.vdim <= p.vp && !p.r1 && !p.sink));
}

template <int KS, int VS, bool UP, bool PAIR>
static int launch_decode_as(const WinAttn& p, cudaStream_t st) {
  const int R = p.H / p.G, hb = PAIR ? 8 : 16, maps = PAIR ? 2 : 1;
  const int smem = 4 * WD_STAGES * WD_KEYS * (p.dp * maps * 2 + 16 + p.vp * 2 + 16);
  int cap = 4 * WD_STAGES * WD_KEYS * (KS * 32 * maps + VS * 32 + 32);
  if (cap > 226 * 1024) cap = 226 * 1024;
  if (smem > cap) return RC_BAD_ARG;
  static unsigned long long prep = 0;
  if (int e = ensure_dynamic_smem((const void*)attn_window_decode_kernel<KS, VS, UP, PAIR>, cap, prep)) return e;
  attn_window_decode_kernel<KS, VS, UP, PAIR><<<dim3(p.n_list, p.G * ((R + hb - 1) / hb), p.splits), 128, smem, st>>>(p);
  return (int)cudaGetLastError();
}

template <int KS, int VS>
static int launch_decode(const WinAttn& p, cudaStream_t st) {
  return p.H / p.G > 8 ? launch_decode_as<KS, VS, true, false>(p, st) : launch_decode_as<KS, VS, false, false>(p, st);
}

}  // namespace omni

using namespace omni;

extern "C" int omni_attn_window_rows(const WinAttn* args, int is_bf16, void* stream) {
  const WinAttn& p = *args;
  if (p.T <= 0) return RC_OK;
  if (!win_args_ok(p) || p.vp > 1024 || p.dp > 4096 || p.row_seq == nullptr) return RC_BAD_ARG;
  dim3 grid(p.T, p.H);
  const int smem = (p.dp + 5 * p.vp) * 4;
  cudaStream_t st = (cudaStream_t)stream;
#define OMNI_ROWS(T)                                                                        \
  do {                                                                                      \
    if (p.vp <= 128) attn_window_rows_kernel<T, 4><<<grid, 128, smem, st>>>(p);             \
    else if (p.vp <= 512) attn_window_rows_kernel<T, 16><<<grid, 128, smem, st>>>(p);       \
    else attn_window_rows_kernel<T, 32><<<grid, 128, smem, st>>>(p);                        \
  } while (0)
  if (is_bf16) OMNI_ROWS(__nv_bfloat16); else OMNI_ROWS(float);
#undef OMNI_ROWS
  return (int)cudaGetLastError();
}

// splits > 1: part_o holds n_list * H * maps * splits * vp floats, part_ml n_list * H * maps * splits * 2.
extern "C" int omni_attn_window_decode(const WinAttn* args, void* stream) {
  const WinAttn& p = *args;
  if (p.n_list <= 0) return RC_OK;
  if (!win_args_ok(p) || p.dp > 256 || p.vp > 256 || p.splits < 1 || p.seq_list == nullptr) return RC_BAD_ARG;
  if ((p.q_rs & 1) || (p.k_ts & 7) || (p.v_ts & 7) || (p.splits > 1 && (p.part_o == nullptr || p.part_ml == nullptr))) return RC_BAD_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  const int mx = p.dp > p.vp ? p.dp : p.vp;
  int rc;
  if (p.maps == 2) {
    if (p.dp > 128) return RC_BAD_ARG;
    rc = p.dp <= 64 && p.vp <= 128 ? launch_decode_as<4, 8, true, true>(p, st) : launch_decode_as<8, 16, true, true>(p, st);
  } else
    rc = mx <= 64 ? launch_decode<4, 4>(p, st) : (mx <= 128 ? launch_decode<8, 8>(p, st) : launch_decode<16, 16>(p, st));
  if (rc) return rc;
  if (p.splits > 1) {
    attn_window_merge_kernel<<<dim3(p.n_list, p.H), p.vp <= 64 ? 64 : (p.vp <= 128 ? 128 : 256), 0, st>>>(p);
    rc = (int)cudaGetLastError();
  }
  return rc;
}
