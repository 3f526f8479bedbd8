// Windowed paged attention of prompt portions on tcgen05 tensor cores (attn_window.h says what is
// computed).
//
// The query heads that share a KV head are packed: row r of a 128-row tile is (token r / R, head r % R) with
// R = heads per KV head, so a K/V tile is fetched once for the whole group and a tile spans only 128 / R
// tokens, which keeps the keys outside a row's window or its future few.  One block owns two such tiles (one
// where two do not fit) of one (sequence, KV head) and visits the key tiles any of its rows sees: the tiles of the kept
// first tokens, then those of the window.  Portions of all sequences of a batch are one launch.
//   warp 0        TMA producer: Q (box {64 channels, R heads, 128 / R tokens}), then K / V pages
//   warp 1        MMA issuer: S_t = Q_t K^T, O_t += P_t V (P read from TMEM)
//   warps 2, 3    distance bias of the key tile: r1 log2(1 + r2 dist) depends on (head, distance) only, so a
//                 tile needs R (127 + 2 * 128 / R) logarithms instead of 2 * 128 * 128; double-buffered table
//                 in shared memory
//   warps 4-11    softmax, one thread per row; scores are bounded, biased and exponentiated in fp32.  The two
//                 exponentials and the reciprocal of a bounded score make the MUFU unit, not the tensor pipe, the
//                 limit; a pair of scores shares one reciprocal.  (Polynomial exponentials on the FMA pipe for 1/8 to
//                 all of them were slower: the issue slots they take are not free.)
// Bounded scores (cap > 0, `bounded` set) never exceed the cap, so max(cap, sink) serves as every row's softmax
// reference: no running maximum, no rescaling, and each chunk of scores goes from tensor memory to weights in one pass.
// The caller sets `bounded` when the smallest weight a row's own key can have, 2^-(2 cap log2 e), is well inside
// fp32's range and the bias never raises a score.
// The keys a block visits are a list of 32-key chunks, those of the kept first tokens followed by those of the
// window; four chunks make a tile, so the kept tokens cost one chunk and the window's ends are cut to 32 keys.
// The one tile that holds chunks of both parts has two bias tables.
// Two maps (differential attention, PAIR): the block's two tiles are the maps of the SAME tokens.  A key tile holds both
// maps' keys, the value tile is shared, and the epilogue combines the two accumulators row by row: warps t = 0 and 1 of a
// quarter share its rows, take every other 16 channels, and exchange denominators and sums of squares in shared memory.
// TMEM columns: S0 [0,128) S1 [128,256) O0 [256,384) O1 [384,512); P_t over the first 64 columns of S_t.
// Every wait is bounded.
#include "attn_window.h"
#include "f32x2.cuh"
#include "host_util.h"
#include "ptx_sm100.cuh"

namespace omni {

constexpr int WP_BM = 128, WP_BN = 128;
constexpr int WP_THREADS = 384;
constexpr int WP_BOX = WP_BM * 64 * 2;          // 64 channels of 128 rows: 16 KiB
constexpr int WP_MAX_STAGES = 4;
constexpr float WP_LOG2E = 1.4426950408889634f;

struct WinPrefill {
  WinAttn a;
  int R, TT;            // heads per KV head, tokens per tile
  int nq;               // query tiles per block (2; 1 where two of the widest heads would not fit)
  int kb, vb;           // 64-channel boxes per key (one map) / value row
  int kbu;              // key boxes of the head's own part; the others hold the part shared by all heads
  int k_stages, v_stages;       // depth of the K and V rings
  int tab_stride;       // floats between the bias rows of two heads
};

__device__ __forceinline__ float wp_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float wp_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float wp_lg2(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// bits [a, b) of a 32-bit word, both clamped to [0, 32]
__device__ __forceinline__ uint32_t bit_range(int a, int b) {
  a = min(max(a, 0), 32);
  b = min(max(b, 0), 32);
  const uint32_t hi = b == 32 ? 0xffffffffu : (1u << b) - 1u;
  const uint32_t lo = a == 32 ? 0xffffffffu : (1u << a) - 1u;
  return hi & ~lo;
}

// sigmoid of a gate logit
__device__ __forceinline__ float wp_open(float z) { return wp_rcp(1.0f + wp_ex2(-WP_LOG2E * z)); }

// 16 channels of a row, times f, channel by channel times the opening of their logits z where `gated`
__device__ __forceinline__ void wp_store16(__nv_bfloat16* dst, const float (&v)[16], float f, bool gated, const uint4 (&z)[2]) {
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    float o[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) o[e] = v[x * 8 + e] * f;
    if (gated) {
      const uint32_t zw[4] = {z[x].x, z[x].y, z[x].z, z[x].w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 g = unpack_bf16(zw[e]);
        o[2 * e] *= wp_open(g.x);
        o[2 * e + 1] *= wp_open(g.y);
      }
    }
    *reinterpret_cast<uint4*>(dst + x * 8) = make_uint4(pack_bf16(o[0], o[1]), pack_bf16(o[2], o[3]), pack_bf16(o[4], o[5]),
                                                        pack_bf16(o[6], o[7]));
  }
}

template <bool CAP, bool BIAS, bool BOUNDED, bool PAIR>
__global__ void __launch_bounds__(WP_THREADS, 1)
attn_window_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                           const __grid_constant__ CUtensorMap tmV, const __grid_constant__ CUtensorMap tmS,
                           const __grid_constant__ WinPrefill w) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t q_full, k_full[WP_MAX_STAGES], k_empty[WP_MAX_STAGES], v_full[WP_MAX_STAGES],
      v_empty[WP_MAX_STAGES];
  __shared__ __align__(8) uint64_t s_full[2], p_full[2][4], o_done[2], tab_full[2], tab_empty[2];
  __shared__ uint32_t tmem_base_s;
  __shared__ int s_abort;

  const WinAttn& p = w.a;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int g = blockIdx.x;                                  // heads vary fastest: the items with the most keys start first
  const int seq = p.items[2 * blockIdx.y], off = p.items[2 * blockIdx.y + 1];
  const int row0 = p.q_start[seq] + off;                     // first batch row of the block
  const int n_seq = p.q_start[seq + 1] - p.q_start[seq];
  const int ctx = p.context[seq];
  const int nt = min((PAIR ? 1 : w.nq) * w.TT, n_seq - off);  // tokens of the block
  const int n_qt = PAIR || nt > w.TT ? 2 : 1;
  const int tile_tokens = PAIR ? 0 : w.TT;                   // tokens from one query tile to the next
  const int p_first = ctx + off, p_last = p_first + nt - 1;
  const int lo_chunk = p.window > 0 ? max(0, p_first - p.window + 1) / 32 : 0;
  const int kept = min(lo_chunk, (p.keep_first + 31) / 32);       // chunks of the kept first tokens
  const int n_kv = (kept + p_last / 32 - lo_chunk + 1 + 3) / 4;    // key tiles
  auto chunk_of = [&](int u) { return u < kept ? u : lo_chunk + u - kept; };

  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const int k_boxes = PAIR ? 2 * w.kb : w.kb;
  const uint32_t q_tile = w.kb * WP_BOX, k_tile = k_boxes * WP_BOX, v_tile = w.vb * WP_BOX;
  const uint32_t sQ = base, sK = base + w.nq * q_tile, sV = sK + w.k_stages * k_tile;
  float* tab = reinterpret_cast<float*>(smem_raw + (sV + w.v_stages * v_tile - smem_u32(smem_raw)));
  const int tab_floats = w.R * w.tab_stride;

  if (threadIdx.x == 0) {
    s_abort = 0;
    mbar_init(smem_u32(&q_full), 1);
    for (int i = 0; i < w.k_stages; ++i) {
      mbar_init(smem_u32(&k_full[i]), 1);
      mbar_init(smem_u32(&k_empty[i]), 1);
    }
    for (int i = 0; i < w.v_stages; ++i) {
      mbar_init(smem_u32(&v_full[i]), 1);
      mbar_init(smem_u32(&v_empty[i]), 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(smem_u32(&s_full[i]), 1);
      for (int c = 0; c < 4; ++c) mbar_init(smem_u32(&p_full[i][c]), 4);
      mbar_init(smem_u32(&o_done[i]), 1);
      mbar_init(smem_u32(&tab_full[i]), 2);                  // the two bias warps
      mbar_init(smem_u32(&tab_empty[i]), 4 * n_qt);          // the softmax warps of the tiles in use
    }
    fence_mbar_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
    if (w.kbu < w.kb) tma_prefetch_desc(&tmS);
  }
  if (warp == 1) {
    tmem_alloc(smem_u32(&tmem_base_s), 512);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = tmem_base_s;
  int* status = p.status;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    // A key tile is 4 * (32 / rows) boxes of `rows` tokens times the 64-channel slices: one lane per copy, so that
    // page lookups and address arithmetic of a tile run side by side, and a tile ahead of the ring.
    if (elect_one()) {
      const uint32_t qb = smem_u32(&q_full);
      mbar_expect_tx(qb, (uint32_t)(n_qt * w.kb * w.R * w.TT * 128));
      for (int t = 0; t < n_qt; ++t)
        for (int x = 0; x < w.kb; ++x)
          tma_load_4d(sQ + t * q_tile + x * WP_BOX, &tmQ, qb, x < w.kbu ? 64 * x : p.dp_u + 64 * (x - w.kbu), 0,
                      row0 + t * tile_tokens, PAIR ? 2 * g + t : g);
    }
    const int* bt = p.block_tables + (long)seq * p.bt_stride;
    const int bs = p.key_start ? 32 : p.block_size, last_page = (ctx + n_seq - 1) / bs;
    const int key0 = p.key_start ? p.key_start[seq] : 0;
    const int rows = min(bs, 32), boxes = 32 / rows;                       // tokens per box, boxes per chunk (1, 2, 4)
    const int n_box = 4 * boxes, box_log2 = boxes == 1 ? 2 : (boxes == 2 ? 3 : 4);
    const uint32_t box_bytes = (uint32_t)rows * 128u;
    const int my_box = lane & (n_box - 1), x_first = lane >> box_log2, x_step = 32 >> box_log2;
    const int in_chunk = (my_box & (boxes - 1)) * rows, my_chunk = my_box / boxes;
    // first cache row of this lane's box of key tile j; boxes past the sequence's last page re-read it: finite
    // data that the mask discards
    auto box_row = [&](int j) {
      const int pos = chunk_of(4 * j + my_chunk) * 32 + in_chunk;
      // back to back: rows past the sequence's last belong to another one or are zero fill, and are masked either way
      if (p.key_start) return key0 + pos;
      const int page = pos / bs;
      const int id = min(max(bt[min(page, last_page)], 0), p.num_blocks - 1);
      return id * bs + min(pos - page * bs, bs - rows);
    };
    int next = box_row(0);
    for (int j = 0; j < n_kv; ++j) {
      const int ks = j % w.k_stages, vs = j % w.v_stages;
      const int r = next;
      if (j + 1 < n_kv) next = box_row(j + 1);
      const uint32_t kbar = smem_u32(&k_full[ks]), vbar = smem_u32(&v_full[vs]);
      mbar_wait(smem_u32(&k_empty[ks]), ((j / w.k_stages) & 1) ^ 1, &s_abort, status, ERR_WAIT_EMPTY);
      if (lane == 0) mbar_expect_tx(kbar, k_tile);
      __syncwarp();
      for (int x = x_first; x < k_boxes; x += x_step) {
        const uint32_t dst = sK + ks * k_tile + x * WP_BOX + my_box * box_bytes;
        if (PAIR) tma_load_3d(dst, &tmK, kbar, 64 * (x < w.kb ? x : x - w.kb), r, 2 * g + (x < w.kb ? 0 : 1));
        else if (x < w.kbu) tma_load_3d(dst, &tmK, kbar, 64 * x, r, g);
        else tma_load_3d(dst, &tmS, kbar, 64 * (x - w.kbu), r, 0);
      }
      mbar_wait(smem_u32(&v_empty[vs]), ((j / w.v_stages) & 1) ^ 1, &s_abort, status, ERR_WAIT_EMPTY);
      if (lane == 0) mbar_expect_tx(vbar, v_tile);
      __syncwarp();
      for (int x = x_first; x < w.vb; x += x_step)
        tma_load_3d(sV + vs * v_tile + x * WP_BOX + my_box * box_bytes, &tmV, vbar, 64 * x, r, g);
    }
  } else if (warp == 1) {
    // -------------------------------------------------------------------- MMA issuer
    if (elect_one()) {
      const uint32_t idesc_qk = umma_idesc(WP_BM, WP_BN, 1, 1, 0, 0);
      const uint32_t idesc_pv = w.vb == 1 ? umma_idesc(WP_BM, 64, 1, 1, 0, 1) : umma_idesc(WP_BM, 128, 1, 1, 0, 1);
      const uint64_t box16 = WP_BOX >> 4, q16 = q_tile >> 4, k16 = k_tile >> 4, v16 = v_tile >> 4;
      const uint64_t dQ = umma_desc_kmajor_sw128(sQ), dK = umma_desc_kmajor_sw128(sK);
      const uint64_t dV = umma_desc_sw128(sV, WP_BOX, 1024);
      const int ks = p.dp >> 4, ksu = p.dp_u >> 4;
      auto issue_s = [&](int t, int st) {
        const uint64_t a0 = dQ + (uint64_t)t * q16, b0 = dK + (uint64_t)st * k16 + (PAIR ? (uint64_t)t * q16 : 0ull);
        auto step = [&](int k0) {
          const int k = k0 < ksu ? k0 : 4 * w.kbu + k0 - ksu;       // the shared part starts a box of its own
          const uint64_t o = (uint64_t)(k >> 2) * box16 + (uint64_t)((k & 3) * 2);   // 16 channels = 32 bytes of a row
          mma_f16_ss(tmem_base + t * 128, a0 + o, b0 + o, idesc_qk, k0 == 0 ? 0u : 1u);
        };
        if (ks == 8 && ksu == 8) {
#pragma unroll
          for (int k = 0; k < 8; ++k) step(k);
        } else if (ks == 4 && ksu == 4) {
#pragma unroll
          for (int k = 0; k < 4; ++k) step(k);
        } else {
          for (int k = 0; k < ks; ++k) step(k);
        }
      };
      mbar_wait(smem_u32(&q_full), 0, &s_abort, status, ERR_WAIT_FULL);
      mbar_wait(smem_u32(&k_full[0]), 0, &s_abort, status, ERR_WAIT_FULL);
      tc_fence_after_sync();
      for (int t = 0; t < n_qt; ++t) {
        issue_s(t, 0);
        tc_commit(smem_u32(&s_full[t]));
      }
      tc_commit(smem_u32(&k_empty[0]));
      for (int j = 0; j < n_kv; ++j) {
        const int st = j % w.v_stages, st1 = (j + 1) % w.k_stages;
        const bool more = j + 1 < n_kv;
        mbar_wait(smem_u32(&v_full[st]), (j / w.v_stages) & 1, &s_abort, status, ERR_WAIT_FULL);
        if (more) mbar_wait(smem_u32(&k_full[st1]), ((j + 1) / w.k_stages) & 1, &s_abort, status, ERR_WAIT_FULL);
        const uint64_t v0 = dV + (uint64_t)st * v16;
        for (int t = 0; t < n_qt; ++t) {
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            // 32 keys of P as the softmax warps hand them over
            mbar_wait(smem_u32(&p_full[t][c]), j & 1, &s_abort, status, ERR_WAIT_SOFTMAX);
            tc_fence_after_sync();
#pragma unroll
            for (int kk = 0; kk < 2; ++kk) {
              const int k = 2 * c + kk;
              mma_f16_ts(tmem_base + 256 + t * 128, tmem_base + t * 128 + k * 8, v0 + (uint64_t)(k * 128), idesc_pv,
                         (k == 0 && j == 0) ? 0u : 1u);
            }
          }
          if (more) {
            issue_s(t, st1);
            tc_commit(smem_u32(&s_full[t]));
          } else {
            tc_commit(smem_u32(&o_done[t]));
          }
        }
        tc_commit(smem_u32(&v_empty[st]));
        if (more) tc_commit(smem_u32(&k_empty[st1]));
      }
    }
  } else if (warp < 4) {
    // ------------------------------------------------------------ bias of the key tiles
    // Entry i of head r is for distance d0 + i, where d0 = p_first - (position of the tile's key 0) - 127.  A tile's
    // keys are consecutive except where the kept part ends: that tile's kept chunks use the third table.
    if (BIAS) {
      const int width = 127 + 2 * w.TT;
      auto fill = [&](float* dst0, int d0) {
        for (int r = 0; r < w.R; ++r) {
          const float r1 = p.r1[g * w.R + r], r2 = p.r2[g * w.R + r];
          float top = CAP ? p.cap * WP_LOG2E : 0.f;
          if (BOUNDED) top = p.sink ? fminf(0.f, top - p.sink[g * w.R + r] * WP_LOG2E) : 0.f;   // less the reference
          float* dst = dst0 + r * w.tab_stride;
          for (int i = threadIdx.x - 64; i < width; i += 64)
            dst[i] = fmaf(-r1, wp_lg2(fmaf(r2, (float)max(d0 + i, 0), 1.0f)), top);
        }
      };
      for (int j = 0; j < n_kv; ++j) {
        const int b = j & 1;
        mbar_wait(smem_u32(&tab_empty[b]), ((j >> 1) & 1) ^ 1, &s_abort, status, ERR_WAIT_EMPTY);
        const bool both = 4 * j < kept && 4 * j + 4 > kept;
        if (4 * j < kept) fill(tab + (both ? 2 : b) * tab_floats, p_first - 128 * j - 127);
        if (4 * j + 4 > kept) fill(tab + b * tab_floats, p_first - 32 * (lo_chunk + 4 * j - kept) - 127);
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(&tab_full[b]));
      }
    }
  } else {
    // -------------------------------------------------------------- softmax + epilogue
    const int t = (warp - 4) >> 2, q = warp & 3;
    const int row = q * 32 + lane;
    const int tok = row / w.R, r = row - tok * w.R;
    const bool tile_used = t < n_qt;
    const bool row_ok = tile_used && tok < w.TT && t * tile_tokens + tok < nt;
    const bool rows_used = __any_sync(0xffffffffu, row_ok);
    const int pos = p_first + t * tile_tokens + tok;
    const uint32_t lane_addr = (uint32_t)(q * 32) << 16;
    const uint32_t tS = tmem_base + lane_addr + t * 128, tO = tmem_base + lane_addr + 256 + t * 128;
    const int h = g * w.R + min(r, w.R - 1);
    const float C = p.cap * WP_LOG2E;
    const float mul = CAP ? p.scale * 2.0f * WP_LOG2E / p.cap : p.scale * WP_LOG2E;
    const float neg2C = -2.0f * C;
    const uint64_t mul_2 = pack2(mul, mul);
    float m = -INFINITY;                         // reference exponent (log2 units)
    uint64_t l2a = 0ull, l2b = 0ull;             // four partial row sums
    if (p.sink) {                                // the sink is a key without a value, seen before all others
      m = p.sink[h] * WP_LOG2E;
      l2a = pack2(1.f, 0.f);
    }
    float b_const = CAP ? C : 0.f;               // what a score without bias is relative to
    if (BOUNDED) {
      const float ref = fmaxf(C, m);
      l2a = p.sink ? pack2(wp_ex2(m - ref), 0.f) : 0ull;
      m = ref;
      b_const = C - ref;
    }
    const long orow = row0 + t * tile_tokens + tok;
    const __nv_bfloat16* gate = p.gate && row_ok ? static_cast<const __nv_bfloat16*>(p.gate) + orow * p.g_rs + (long)h * p.g_hs : nullptr;
    if (gate && p.g_cs) {                        // fetched after the last tile
      for (int c = 0; c < p.vp; c += 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(gate + c));
    }
    const float* my_tab = tab + min(r, w.R - 1) * w.tab_stride + min(t * tile_tokens + tok, 2 * w.TT - 1) + 127;
    for (int j = 0; tile_used && j < n_kv; ++j) {
      mbar_wait(smem_u32(&s_full[t]), j & 1, &s_abort, status, ERR_WAIT_FULL);
      if (!rows_used) {
        if (lane == 0) {
          for (int c = 0; c < 4; ++c) mbar_arrive(smem_u32(&p_full[t][c]));
          if (BIAS) mbar_arrive(smem_u32(&tab_empty[j & 1]));
        }
        continue;
      }
      tc_fence_after_sync();
      if (BIAS) mbar_wait(smem_u32(&tab_full[j & 1]), (j >> 1) & 1, &s_abort, status, ERR_WAIT_FULL);
      const float* tb = my_tab + (j & 1) * tab_floats;
      const float* tb_kept = 4 * j + 4 > kept ? my_tab + 2 * tab_floats : tb;
      uint32_t v0[32], v1[32], v2[32], v3[32];
      tmem_ld_32x32(tS, v0);
      tmem_ld_32x32(tS + 32, v1);
      tmem_ld_32x32(tS + 64, v2);
      tmem_ld_32x32(tS + 96, v3);
      tmem_wait_ld();
      float ma = -INFINITY, mb = -INFINITY, mc = -INFINITY, md = -INFINITY;
      auto score = [&](uint32_t (&v)[32], int c) {
        const int u = 4 * j + c;
        const float* tc = (u < kept ? tb_kept : tb) - c * 32;
#pragma unroll
        for (int e = 0; e < 32; e += 2) {
          uint64_t y2 = mul2(pack2(__uint_as_float(v[e]), __uint_as_float(v[e + 1])), mul_2);
          float y0, y1;
          float b0 = b_const, b1 = b_const;
          if (BIAS) {
            b0 = tc[-e];
            b1 = tc[-e - 1];
          }
          unpack2(y2, y0, y1);
          if (CAP) {
            // cap tanh(s / cap) = C - 2C / (1 + 2^y); the pair shares one reciprocal, and |y| <= 60 keeps the
            // product of the two denominators finite (there the bound is reached to the last bit)
            const uint64_t e2 = pack2(wp_ex2(fminf(y0, 60.f)), wp_ex2(fminf(y1, 60.f)));
            float a0, a1;
            unpack2(add2(e2, pack2(1.f, 1.f)), a0, a1);
            const float k = neg2C * wp_rcp(a0 * a1);
            y0 = fmaf(k, a1, b0);
            y1 = fmaf(k, a0, b1);
          } else if (BIAS) {
            y0 += b0;
            y1 += b1;
          }
          v[e] = __float_as_uint(y0);
          v[e + 1] = __float_as_uint(y1);
        }
        const int kbase = chunk_of(u) * 32;
        const int hi = pos - kbase + 1;                                   // keys e < hi are not in the future
        const int lo = p.window > 0 ? pos - p.window + 1 - kbase : 0;      // keys e >= lo are in the window
        if (__any_sync(0xffffffffu, hi < 32 || lo > 0)) {
          const uint32_t mk = bit_range(lo, hi) | bit_range(0, min(p.keep_first - kbase, hi));
#pragma unroll
          for (int e = 0; e < 32; ++e)
            if (!(mk & (1u << e))) v[e] = 0xff800000u;
        }
        if constexpr (!BOUNDED) {
#pragma unroll
          for (int e = 0; e < 32; e += 8) {
            ma = max3(ma, __uint_as_float(v[e]), __uint_as_float(v[e + 1]));
            mb = max3(mb, __uint_as_float(v[e + 2]), __uint_as_float(v[e + 3]));
            mc = max3(mc, __uint_as_float(v[e + 4]), __uint_as_float(v[e + 5]));
            md = max3(md, __uint_as_float(v[e + 6]), __uint_as_float(v[e + 7]));
          }
        }
      };
      // exponents x (already relative to the reference) -> weights, bf16 pairs over the chunk's first score columns
      auto weights = [&](uint32_t (&v)[32], int c, uint64_t negm2) {
        uint32_t pk[16];
#pragma unroll
        for (int e = 0; e < 32; e += 2) {
          uint64_t x2 = pack2(__uint_as_float(v[e]), __uint_as_float(v[e + 1]));
          if (!BOUNDED) x2 = add2(x2, negm2);
          float e0, e1;
          unpack2(x2, e0, e1);
          e0 = wp_ex2(e0);
          e1 = wp_ex2(e1);
          const uint64_t p2 = pack2(e0, e1);
          if (e & 2) l2b = add2(l2b, p2); else l2a = add2(l2a, p2);
          pk[e >> 1] = pack_bf16(e0, e1);
        }
        tmem_st_32x16(tS + c * 16, pk);
        tmem_wait_st();
        tc_fence_before_sync();
        __syncwarp();
        if (lane == 0) mbar_arrive(smem_u32(&p_full[t][c]));
      };
      auto table_done = [&]() {
        if (BIAS) {
          __syncwarp();
          if (lane == 0) mbar_arrive(smem_u32(&tab_empty[j & 1]));
        }
      };
      if (BOUNDED) {
        score(v0, 0);
        weights(v0, 0, 0ull);
        score(v1, 1);
        weights(v1, 1, 0ull);
        score(v2, 2);
        weights(v2, 2, 0ull);
        score(v3, 3);
        table_done();
        weights(v3, 3, 0ull);
        continue;
      }
      score(v0, 0);
      score(v1, 1);
      score(v2, 2);
      score(v3, 3);
      table_done();
      const float m_new = fmaxf(m, fmaxf(fmaxf(ma, mb), fmaxf(mc, md)));
      if (j == 0) {
        if (m != -INFINITY) l2a = pack2(wp_ex2(m - m_new), 0.f);          // the sink's share so far
        m = m_new;
      } else if (__any_sync(0xffffffffu, m_new > m + 8.0f)) {
        // rare: O follows the new reference; the scores wait in their own TMEM columns meanwhile
        const float alpha = m_new == -INFINITY ? 1.f : wp_ex2(m - m_new);
        l2a = mul2(l2a, pack2(alpha, alpha));
        l2b = mul2(l2b, pack2(alpha, alpha));
        tmem_st_32x32(tS, v0);
        tmem_st_32x32(tS + 32, v1);
        tmem_st_32x32(tS + 64, v2);
        tmem_st_32x32(tS + 96, v3);
        tmem_wait_st();
#pragma unroll 1
        for (int c = 0; c < 2 * w.vb; ++c) {
          uint32_t v[32];
          tmem_ld_32x32(tO + c * 32, v);
          tmem_wait_ld();
#pragma unroll
          for (int e = 0; e < 32; ++e) v[e] = __float_as_uint(__uint_as_float(v[e]) * alpha);
          tmem_st_32x32(tO + c * 32, v);
        }
        tmem_wait_st();
        m = m_new;
        tmem_ld_32x32(tS, v0);
        tmem_ld_32x32(tS + 32, v1);
        tmem_ld_32x32(tS + 64, v2);
        tmem_ld_32x32(tS + 96, v3);
        tmem_wait_ld();
      }
      const float m_use = m == -INFINITY ? 0.f : m;
      const uint64_t negm2 = pack2(-m_use, -m_use);
      weights(v0, 0, negm2);
      weights(v1, 1, negm2);
      weights(v2, 2, negm2);
      weights(v3, 3, negm2);
    }
    if (rows_used) {
      // the gate's logits, on their way while the last products finish
      const bool channels = gate && p.g_cs;
      const float head_gate = gate && p.g_cs == 0 ? wp_open((float)gate[0]) : 1.f;
      uint4 gz[8][2];
      if (channels) {
#pragma unroll
        for (int c = 0; c < 8; ++c)
          if (c * 16 < p.vp) {
            gz[c][0] = *reinterpret_cast<const uint4*>(gate + c * 16);
            gz[c][1] = *reinterpret_cast<const uint4*>(gate + c * 16 + 8);
          }
      }
      mbar_wait(smem_u32(&o_done[t]), 0, &s_abort, status, ERR_WAIT_PV);
      tc_fence_after_sync();
      float s0, s1, s2, s3;
      unpack2(l2a, s0, s1);
      unpack2(l2b, s2, s3);
      float f = 1.0f / ((s0 + s1) + (s2 + s3));
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + orow * p.o_rs + (long)h * p.vp;
      if constexpr (PAIR) {
        mbar_wait(smem_u32(&o_done[t ^ 1]), 0, &s_abort, status, ERR_WAIT_PV);
        tc_fence_after_sync();
        // every product is done: the query tiles' memory takes the exchanged numbers
        float* ex = reinterpret_cast<float*>(smem_raw + (sQ - smem_u32(smem_raw)));
        auto pair_sync = [&]() { asm volatile("bar.sync %0, 64;" ::"r"(1 + q) : "memory"); };
        ex[t * 128 + row] = f;
        pair_sync();
        const float f0 = ex[row], f1 = -p.lam * ex[128 + row];
        const uint32_t o0 = tmem_base + lane_addr + 256, o1 = o0 + 128;
        float ss = 0.f;
        auto combined = [&](int c, float (&u)[16]) {
          uint32_t a[16], b[16];
          tmem_ld_32x16(o0 + c, a);
          tmem_ld_32x16(o1 + c, b);
          tmem_wait_ld();
#pragma unroll
          for (int e = 0; e < 16; ++e) u[e] = fmaf(__uint_as_float(a[e]), f0, __uint_as_float(b[e]) * f1);
        };
#pragma unroll 1
        for (int c = 16 * t; c < p.vp; c += 32) {
          float u[16];
          combined(c, u);
#pragma unroll
          for (int e = 0; e < 16; ++e) ss = fmaf(u[e], u[e], ss);
        }
        ex[256 + t * 128 + row] = ss;
        pair_sync();
        ss = ex[256 + row] + ex[384 + row];
        f = p.out_mul * head_gate / sqrtf(ss / (float)p.vdim + p.out_eps);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int c = 16 * t + 32 * i;
          if (c < p.vp) {
            float u[16];
            combined(c, u);
            if (row_ok) wp_store16(dst + c, u, f, channels, t ? gz[2 * i + 1] : gz[2 * i]);
          }
        }
      } else {
        f *= head_gate;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int c = 16 * i;
          if (c < p.vp) {
            uint32_t v[16];
            tmem_ld_32x16(tO + c, v);
            tmem_wait_ld();
            float u[16];
#pragma unroll
            for (int e = 0; e < 16; ++e) u[e] = __uint_as_float(v[e]);
            if (row_ok) wp_store16(dst + c, u, f, channels, gz[i]);
          }
        }
      }
    }
  }

  tc_fence_before_sync();
  __syncthreads();
  if (s_abort) {
    // a wait ran out: give copies and products in flight time to finish before their memory goes
    const unsigned long long t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) {
    }
  }
  if (warp == 1) tmem_dealloc(tmem_base, 512);
}

// Q as (channel, head of the group, token, KV head and map)
static int make_q_tmap(CUtensorMap* tm, const WinAttn& p, int R, int TT) {
  EncodeTiledFn enc = get_encode_tiled();
  if (!enc) return RC_NO_DRIVER;
  if ((reinterpret_cast<uintptr_t>(p.q) & 15) || (p.q_rs & 7)) return RC_BAD_ARG;
  cuuint64_t gdim[4] = {(cuuint64_t)p.dp, (cuuint64_t)R, (cuuint64_t)p.T, (cuuint64_t)p.G * (p.maps == 2 ? 2 : 1)};
  cuuint64_t gstr[3] = {(cuuint64_t)p.dp * 2, (cuuint64_t)p.q_rs * 2, (cuuint64_t)R * p.dp * 2};
  cuuint32_t box[4] = {64, (cuuint32_t)R, (cuuint32_t)TT, 1};
  cuuint32_t estr[4] = {1, 1, 1, 1};
  CUresult r = enc(tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(p.q), gdim, gstr, box, estr,
                   CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                   CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? RC_OK : RC_TMAP;
}

template <bool CAP, bool BIAS, bool BOUNDED, bool PAIR = false>
static int launch_prefill(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const CUtensorMap& ts, const WinPrefill& w,
                          int smem, cudaStream_t st) {
  static unsigned long long prep = 0;
  if (int e = ensure_dynamic_smem((const void*)attn_window_prefill_kernel<CAP, BIAS, BOUNDED, PAIR>, 227 * 1024 - 512, prep)) return e;
  attn_window_prefill_kernel<CAP, BIAS, BOUNDED, PAIR><<<dim3(w.a.G, w.a.n_items), WP_THREADS, smem, st>>>(tq, tk, tv, ts, w);
  return (int)cudaGetLastError();
}

}  // namespace omni

using namespace omni;

// items: int32 [n_items, 2] (sequence, first row within its portion; blocks of block_tokens rows).
extern "C" int omni_attn_window_prefill(const WinAttn* args, void* stream) {
  WinPrefill w;
  w.a = *args;
  const WinAttn& p = w.a;
  if (p.n_items <= 0) return RC_OK;
  if (p.H <= 0 || p.G <= 0 || p.H % p.G || (p.dp & 15) || (p.vp & 15) || p.dp <= 0 || p.vp <= 0 || p.dp > 256 ||
      p.vp > 128 || p.items == nullptr || p.num_seqs <= 0 || p.num_blocks <= 0 || p.keep_first < 0)
    return RC_BAD_ARG;
  if (p.key_start == nullptr && (p.block_size < 8 || (p.block_size & 7) || 128 % p.block_size)) return RC_BAD_ARG;
  if (p.n_items > 65535 || (p.k_ts & 7) || (p.v_ts & 7) || p.dp_u <= 0 || (p.dp_u & 15) || p.dp_u > p.dp) return RC_BAD_ARG;
  if (p.dp_u < p.dp && (p.k_shared == nullptr || (p.ks_ts & 7))) return RC_BAD_ARG;
  if (p.key_start && (p.key_rows <= 0 || p.key_rows > 0x7fffffffl)) return RC_BAD_ARG;
  if ((p.r1 == nullptr) != (p.r2 == nullptr) || (p.o_rs & 7) || (reinterpret_cast<uintptr_t>(p.out) & 15)) return RC_BAD_ARG;
  w.R = p.H / p.G;
  if (w.R > 128) return RC_BAD_ARG;
  w.TT = 128 / w.R;
  if (p.block_tokens != w.TT && p.block_tokens != 2 * w.TT) return RC_BAD_ARG;
  const bool pair = p.maps == 2;
  if (pair && (p.block_tokens != w.TT || p.dp_u != p.dp || p.key_start || p.r1 || p.sink || p.cap > 0.f || p.vdim <= 0 || p.vdim > p.vp))
    return RC_BAD_ARG;
  if (p.g_cs && ((reinterpret_cast<uintptr_t>(p.gate) & 15) || (p.g_rs & 7) || (p.g_hs & 7) || p.g_cs != 1)) return RC_BAD_ARG;
  w.nq = pair ? 2 : p.block_tokens / w.TT;
  w.kbu = (p.dp_u + 63) / 64;
  w.kb = w.kbu + (p.dp - p.dp_u + 63) / 64;
  w.vb = (p.vp + 63) / 64;
  // rows of the bias table: a warp's 32 rows are 32 / R tokens of R heads; this pitch spreads them over all banks
  const int width = 127 + 2 * w.TT;
  const bool pow2 = (w.R & (w.R - 1)) == 0 && w.R <= 32;
  const int want = pow2 ? (32 / w.R) % 32 : 1;
  w.tab_stride = width;
  while (w.tab_stride % 32 != want) ++w.tab_stride;
  const int tab_bytes = p.r1 ? 3 * w.R * w.tab_stride * 4 : 0;
  const int limit = 227 * 1024 - 1024 - 512;                 // less the alignment slack and the static barriers
  const int q_bytes = w.nq * w.kb * WP_BOX, k_bytes = (pair ? 2 : 1) * w.kb * WP_BOX, v_bytes = w.vb * WP_BOX;
  w.k_stages = w.v_stages = 1;
  int used = q_bytes + tab_bytes + k_bytes + v_bytes;
  if (used > limit) return RC_TOO_LARGE;
  // the value ring grows first: a key slot is free as soon as its scores are issued, a value slot only after the softmax
  for (bool grew = true; grew;) {
    grew = false;
    if (w.v_stages < WP_MAX_STAGES && used + v_bytes <= limit) { ++w.v_stages; used += v_bytes; grew = true; }
    if (w.k_stages < WP_MAX_STAGES && used + k_bytes <= limit) { ++w.k_stages; used += k_bytes; grew = true; }
  }
  const int smem = used + 1024;
  CUtensorMap tq, tk, tv, ts;
  const uint64_t slots = p.key_start ? (uint64_t)p.key_rows : (uint64_t)p.num_blocks * p.block_size;
  const uint32_t box_rows = p.key_start ? 32 : (p.block_size < 32 ? p.block_size : 32);
  int rc = make_q_tmap(&tq, p, w.R, w.TT);
  if (!rc) rc = make_tmap_3d(&tk, p.k_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, p.dp_u, slots, p.G * (pair ? 2 : 1), (uint64_t)p.k_ts * 2,
                             (uint64_t)p.dp_u * 2, 64, box_rows);
  if (!rc) rc = make_tmap_3d(&tv, p.v_cache, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, p.vp, slots, p.G, (uint64_t)p.v_ts * 2,
                             (uint64_t)p.vp * 2, 64, box_rows);
  ts = tk;
  if (!rc && w.kbu < w.kb)
    rc = make_tmap_3d(&ts, p.k_shared, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, p.dp - p.dp_u, slots, 1, (uint64_t)p.ks_ts * 2,
                      (uint64_t)p.ks_ts * 2, 64, box_rows);
  if (rc) return rc;
  cudaStream_t st = (cudaStream_t)stream;
  if (pair) return launch_prefill<false, false, false, true>(tq, tk, tv, ts, w, smem, st);
  if (p.cap > 0.f && p.bounded)
    return p.r1 ? launch_prefill<true, true, true>(tq, tk, tv, ts, w, smem, st) : launch_prefill<true, false, true>(tq, tk, tv, ts, w, smem, st);
  if (p.cap > 0.f)
    return p.r1 ? launch_prefill<true, true, false>(tq, tk, tv, ts, w, smem, st) : launch_prefill<true, false, false>(tq, tk, tv, ts, w, smem, st);
  return p.r1 ? launch_prefill<false, true, false>(tq, tk, tv, ts, w, smem, st) : launch_prefill<false, false, false>(tq, tk, tv, ts, w, smem, st);
}
