// Attention over a cache of latents.  A token leaves one row in the pages, shared by all heads: its latent c (rank_p
// channels, normed) and a rotated key part (rot_p channels).  Head h has keys [W_uk[h] c, rotated part] and values
// W_uv[h] c; queries are [dim_p unrotated | rot_p rotated] channels per head.  All sizes are multiples of 16 with
// zero padding.
//
//   omni_latent_rows     rotates the queries in place, norms and rotates a token's row, writes it to its page, norms a
//                        latent of the queries in place (each part optional)
//   omni_latent_gather   rows of several sequences from their pages to one buffer (prompts expand them to keys and
//                        values with one GEMM and run on attn_window_sm100.cu)
//   omni_head_gemm       one small product per head: queries into the latent space (W_uk^T q) and attention results
//                        out of it (W_uv o, times the output gate); weights are read once per 16 rows
//   omni_gate_channels   out *= sigmoid(gate), channel by channel (where no other kernel's epilogue does it)
//   omni_latent_decode   decoded tokens (and rows of short portions): scores and weighted sums directly on the
//                        latent rows, so a row is read once per 16 or 32 heads.  A block owns one token's heads and a
//                        share of its keys; a producer warp copies 32-key tiles into a ring (bulk copies), two groups of
//                        eight warps take tiles in turn (or, with more than 16 heads, the same tile for 16 heads each);
//                        a group's warps share the score product by (keys, channel quarter) and the weighted sum by
//                        channels.  Every wait is bounded
//
// A decode step reads every latent once per group of heads and does little arithmetic on it, so the warp-level
// products (no operand staging through tensor memory) suffice.
#include "host_util.h"
#include "row_ops.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

// ------------------------------------------------------------------------------- rows and pages
struct LatentRows {
  void* q; long ldq;               // [T, H, dim_p + rot_p] or nullptr: rotated parts are turned in place
  int T, H, dim_p, rot, rot_p;
  const void* z; long ldz;         // [T, rank_p | rot_p] or nullptr: the layer writes no row
  int rank, rank_p;
  const float* turns;              // [T, rot / 2, 2] cos, sin
  const int* slots;                // [T], < 0: not written
  void* pages; long num_slots;     // [num_slots, rank_p + rot_p]
  const float* norm;               // [rank_p]
  float eps;
  int* status;
  void* qc; long ldqc;             // [T, q_rank_p] or nullptr: latent of the queries, normed in place
  int q_rank, q_rank_p;
  const float* q_norm;             // [q_rank_p]
};

// four rotated pairs: channels 8 i .. 8 i + 7 of a part of 2 `half` rotated channels (padding passes unchanged)
__device__ __forceinline__ void turn8(float (&v)[8], const float2* turn, int i, int half) {
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    if (i * 4 + e < half) {
      const float2 a = turn[i * 4 + e];
      const float x = v[2 * e], y = v[2 * e + 1];
      v[2 * e] = x * a.x - y * a.y;
      v[2 * e + 1] = y * a.x + x * a.y;
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(128)
latent_rows_kernel(const LatentRows p) {
  __shared__ float sh[64];
  const long t = blockIdx.x;
  const float2* turn = reinterpret_cast<const float2*>(p.turns) + t * (p.rot / 2);
  const int half = p.rot / 2, hc = p.dim_p + p.rot_p, rv = (p.rot + 7) / 8;
  if (p.q) {
    T* row = static_cast<T*>(p.q) + t * p.ldq;
    for (int i = threadIdx.x; i < p.H * rv; i += 128) {
      const int h = i / rv, c = i - h * rv;
      T* q = row + h * hc + p.dim_p + 8 * c;
      float v[8];
      load8<T>(q, v);
      turn8(v, turn, c, half);
      store8<T>(q, v);
    }
  }
  if (p.z == nullptr && p.qc == nullptr) return;
  const T* z = static_cast<const T*>(p.z) + t * p.ldz;
  T* qc = static_cast<T*>(p.qc) + t * p.ldqc;
  float ss[2] = {0.f, 0.f};
  auto add = [&](const T* src, int n, float& sum) {
    for (int i = threadIdx.x; i < n / 8; i += 128) {
      float v[8];
      load8<T>(src + 8 * i, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) sum = fmaf(v[e], v[e], sum);
    }
  };
  if (p.z) add(z, p.rank_p, ss[0]);
  if (p.qc) add(qc, p.q_rank_p, ss[1]);
  block_sum<2>(ss, sh);
  if (p.qc) {
    const float s = rms_scale(ss[1], p.q_rank, p.eps);
    for (int i = threadIdx.x; i < p.q_rank_p / 8; i += 128) {
      float v[8];
      load8<T>(qc + 8 * i, v);
      scale_gain8(v, s, p.q_norm, 1, 8 * i);
      store8<T>(qc + 8 * i, v);
    }
  }
  if (p.z == nullptr) return;
  const float s = rms_scale(ss[0], p.rank, p.eps);
  const long slot = p.slots[t];
  if (slot >= p.num_slots && p.status && threadIdx.x == 0) atomicCAS(p.status, 0, (int)ERR_BOUNDS);
  if (slot < 0 || slot >= p.num_slots) return;
  T* page = static_cast<T*>(p.pages) + slot * (p.rank_p + p.rot_p);
  for (int i = threadIdx.x; i < (p.rank_p + p.rot_p) / 8; i += 128) {
    float v[8];
    load8<T>(z + 8 * i, v);
    if (8 * i < p.rank_p) scale_gain8(v, s, p.norm, 1, 8 * i);
    else turn8(v, turn, i - p.rank_p / 8, half);
    store8<T>(page + 8 * i, v);
  }
}

// out[t, c] *= sigmoid(gate[t, c])
template <typename T>
__global__ void __launch_bounds__(256)
gate_channels_kernel(T* __restrict__ out, long ldo, const T* __restrict__ gate, long ldg, long rows, int n) {
  const int chunks = n / 8;
  const long total = rows * chunks;
  for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x) {
    const long r = i / chunks;
    const int c = (int)(i - r * chunks) * 8;
    float v[8], g[8];
    load8<T>(out + r * ldo + c, v);
    load8<T>(gate + r * ldg + c, g);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= 1.0f / (1.0f + expf(-g[e]));
    store8<T>(out + r * ldo + c, v);
  }
}

// members: (sequence, first row of the output) pairs closed by (-1, rows); key_start[s]: row of the output that position 0 of
// sequence s has or would have (negative where a window leaves its first positions out); 16-byte pieces.
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ pages, int row16, const int* __restrict__ tables, int bt_stride, int block_size,
                     int num_blocks, const int* __restrict__ members, int n_members, const int* __restrict__ key_start,
                     uint4* __restrict__ out, long rows) {
  const long total = rows * row16;
  for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x) {
    const int r = (int)(i / row16), c = (int)(i - (long)r * row16);
    int lo = 0, hi = n_members - 1;                          // the last member that starts at or before r
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (members[2 * mid + 1] <= r) lo = mid; else hi = mid - 1;
    }
    const int seq = members[2 * lo], pos = r - key_start[seq];
    int pg = tables[(long)seq * bt_stride + pos / block_size];
    pg = min(max(pg, 0), num_blocks - 1);
    out[i] = pages[((long)pg * block_size + pos % block_size) * row16 + c];
  }
}

// -------------------------------------------------------------------------- one product per head
struct HeadGemm {
  const bf16* A; long a_row, a_head; const int* a_rows;     // A[(a_rows[m] or m) * a_row + h * a_head + k]
  const bf16* W;                                            // [H, N, K]
  bf16* C; long c_row, c_head; const int* c_rows;
  const bf16* gate; long g_row;                             // logits at the row of C and head, or nullptr
  int M, N, K, H, rows_a, rows_c;
  long g_head; int g_col;                                   // pitch of heads; 1: one logit per channel, 0: one per head
};

__device__ __forceinline__ void mma_bf16(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0,
                                         uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
               "{%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

// A block: 16 rows of one head, 32 outputs; its four warps take every fourth 32-channel chunk of the contraction, so
// that the loads of a short contraction are all in flight at once.  Lane group j of a quad owns channels 8 j .. 8 j + 7
// of a chunk in both operands (the contraction is permuted alike), so all loads are 16 bytes.
__global__ void __launch_bounds__(128)
head_gemm_kernel(const HeadGemm p) {
  __shared__ __align__(16) float part[4][16][36];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, j = lane & 3;
  const int h = blockIdx.y, n0 = blockIdx.x * 32, m0 = blockIdx.z * 16;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  const bf16* a[2];
  bool live[2];
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int r = m0 + u * 8 + g;
    live[u] = r < p.M;
    int row = live[u] ? (p.a_rows ? p.a_rows[r] : r) : 0;
    row = min(max(row, 0), p.rows_a - 1);
    a[u] = p.A + row * p.a_row + h * p.a_head + j * 8;
  }
  const bf16* w = p.W + ((long)h * p.N + n0 + g) * p.K + j * 8;
  float acc[4][4] = {};
#pragma unroll 4
  for (int k = warp * 32; k < p.K; k += 128) {
    const bool in = k + j * 8 < p.K;                        // K is a multiple of 16
    const uint4 x = in && live[0] ? *reinterpret_cast<const uint4*>(a[0] + k) : zero;
    const uint4 y = in && live[1] ? *reinterpret_cast<const uint4*>(a[1] + k) : zero;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const uint4 b = in && n0 + n * 8 < p.N ? *reinterpret_cast<const uint4*>(w + (long)n * 8 * p.K + k) : zero;
      mma_bf16(acc[n], x.x, y.x, x.y, y.y, b.x, b.y);
      mma_bf16(acc[n], x.z, y.z, x.w, y.w, b.z, b.w);
    }
  }
#pragma unroll
  for (int n = 0; n < 4; ++n)
#pragma unroll
    for (int u = 0; u < 2; ++u)
      *reinterpret_cast<float2*>(&part[warp][u * 8 + g][n * 8 + j * 2]) = make_float2(acc[n][2 * u], acc[n][2 * u + 1]);
  __syncthreads();
  const int r = threadIdx.x >> 3, c = (threadIdx.x & 7) * 4;
  if (m0 + r >= p.M || n0 + c >= p.N) return;
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int q = 0; q < 4; ++q) {
    const float4 v = *reinterpret_cast<const float4*>(&part[q][r][c]);
    o.x += v.x; o.y += v.y; o.z += v.z; o.w += v.w;
  }
  int row = p.c_rows ? p.c_rows[m0 + r] : m0 + r;
  row = min(max(row, 0), p.rows_c - 1);
  if (p.gate) {
    const bf16* z = p.gate + row * p.g_row + h * p.g_head + (n0 + c) * p.g_col;
    auto open = [](bf16 v) { return 1.0f / (1.0f + __expf(-(float)v)); };
    const float f = open(z[0]);
    o.x *= f;
    o.y *= p.g_col ? open(z[1]) : f;
    o.z *= p.g_col ? open(z[2]) : f;
    o.w *= p.g_col ? open(z[3]) : f;
  }
  *reinterpret_cast<uint2*>(p.C + row * p.c_row + h * p.c_head + n0 + c) = make_uint2(pack_bf16(o.x, o.y), pack_bf16(o.z, o.w));
}

// ---------------------------------------------------------------------------------- decode
struct LatentDecode {
  const bf16* q_lat;                   // [n, H, rank_p]
  const bf16* proj; long ldp; int head_cols, dim_p;         // rotated query part: proj[row * ldp + h * head_cols + dim_p]
  const bf16* pages; int rank_p, rot_p;
  const int* block_tables; int bt_stride, block_size, num_blocks;
  const int* rows; int n;              // batch rows served
  const int* row_seq; const int* q_start; const int* context; int num_seqs, T;
  float scale;
  bf16* out;                           // [n, H, rank_p]
  int H, splits;
  float* part_o; float* part_ml;       // [n, H, splits, rank_p], [n, H, splits, 2]
  int* status;
  int window;                          // a row sees its last `window` positions; <= 0: all
};

constexpr int LD_KEYS = 32, LD_ROWS = 16, LD_MAX_STAGES = 8;
constexpr float LD_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float ld_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// contiguous bytes to shared memory, counted on an mbarrier (both addresses and the size: multiples of 16)
__device__ __forceinline__ void ld_bulk(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes),
               "r"(bar)
               : "memory");
}
__device__ __forceinline__ void ld_m4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ld_m4t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}

// shared memory of one block: the key ring, the queries, and per group of warps the weights (bf16) and four partial
// score tiles (fp32)
constexpr int LD_GROUP_BYTES = LD_ROWS * (LD_KEYS * 2 + 16) + 4 * LD_ROWS * (LD_KEYS + 4) * 4;
constexpr int LD_LIMIT = 226 * 1024;

inline int latent_decode_stages(int row_ch, bool wide) {
  const int pitch = row_ch * 2 + 16;
  const int n = (LD_LIMIT - 2 * LD_GROUP_BYTES - (wide ? 2 : 1) * LD_ROWS * pitch) / (LD_KEYS * pitch);
  return n < LD_MAX_STAGES ? n : LD_MAX_STAGES;
}

// CPW: 16-channel slices of the weighted sum per warp (rank_p <= 128 CPW).  WIDE: more than 16 heads, the two groups of
// warps own 16 heads each and share every tile; otherwise they own the same heads and take tiles in turn.
template <int CPW, bool WIDE>
__global__ void __launch_bounds__(544, 1)
latent_decode_kernel(const LatentDecode p, const int stages) {
  constexpr int SP = LD_KEYS + 4, pp = LD_KEYS * 2 + 16, QROWS = WIDE ? 2 * LD_ROWS : LD_ROWS;
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ __align__(8) uint64_t k_full[LD_MAX_STAGES], k_empty[LD_MAX_STAGES];
  __shared__ float s_alpha[2][LD_ROWS], s_m[2][LD_ROWS], s_l[2][LD_ROWS];
  __shared__ int s_abort;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h0 = blockIdx.y * QROWS, split = blockIdx.z;
  const int row = min(max(p.rows[blockIdx.x], 0), p.T - 1);
  const int seq = min(max(p.row_seq[row], 0), p.num_seqs - 1);
  const int pos = p.context[seq] + row - p.q_start[seq];
  const int first = p.window > 0 ? max(0, pos - p.window + 1) : 0;         // keys are counted from the first visible one
  const int n_vis = pos - first + 1;
  const int tiles_all = (n_vis + LD_KEYS - 1) / LD_KEYS;
  const int per = (tiles_all + p.splits - 1) / p.splits;
  const int t0 = min(tiles_all, split * per), n_tiles = min(tiles_all, t0 + per) - t0;
  const int ch = p.rank_p + p.rot_p, pitch = ch * 2 + 16;
  const uint32_t sK = smem_u32(smem), sQ = sK + stages * LD_KEYS * pitch, sG = sQ + QROWS * pitch;

  if (tid == 0) {
    s_abort = 0;
    for (int i = 0; i < stages; ++i) {
      mbar_init(smem_u32(&k_full[i]), 1);
      mbar_init(smem_u32(&k_empty[i]), WIDE ? 16 : 8);       // warps that read a tile
    }
    fence_mbar_init();
  }
  // queries: latent part, rotated part; rows past the last head are zero
  for (int i = tid; i < QROWS * (ch / 8); i += 544) {
    const int r = i / (ch / 8), c = (i - r * (ch / 8)) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (h0 + r < p.H) {
      const bf16* src = c < p.rank_p ? p.q_lat + ((long)blockIdx.x * p.H + h0 + r) * p.rank_p + c
                                     : p.proj + (long)row * p.ldp + (long)(h0 + r) * p.head_cols + p.dim_p + (c - p.rank_p);
      v = *reinterpret_cast<const uint4*>(src);
    }
    st_shared_v4(sQ + r * pitch + c * 2, v);
  }
  __syncthreads();

  const int grp = (warp >> 3) & 1, gw = warp & 7, gt = tid & 255;
  float acc[CPW][2][4];
#pragma unroll
  for (int c = 0; c < CPW; ++c)
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[c][n][i] = 0.f;

  if (warp == 16) {
    // ------------------------------------------- producer: a lane copies one key row, pages are looked up a tile ahead
    const int* bt = p.block_tables + (long)seq * p.bt_stride;
    auto src_row = [&](int t) {
      const int j = first + min((t0 + t) * LD_KEYS + lane, n_vis - 1);     // past the end: a valid key, masked below
      const int pg = min(max(bt[j / p.block_size], 0), p.num_blocks - 1);
      return p.pages + ((long)pg * p.block_size + j % p.block_size) * ch;
    };
    const bf16* next = n_tiles > 0 ? src_row(0) : nullptr;
    int st = 0;
    uint32_t ph = 1;
    for (int t = 0; t < n_tiles; ++t) {
      const bf16* src = next;
      if (t + 1 < n_tiles) next = src_row(t + 1);
      const uint32_t bar = smem_u32(&k_full[st]);
      mbar_wait(smem_u32(&k_empty[st]), ph, &s_abort, p.status, ERR_WAIT_EMPTY);
      if (lane == 0) mbar_expect_tx(bar, (uint32_t)(LD_KEYS * ch * 2));
      __syncwarp();
      ld_bulk(sK + (st * LD_KEYS + lane) * pitch, src, (uint32_t)(ch * 2), bar);
      if (++st == stages) {
        st = 0;
        ph ^= 1;
      }
    }
  } else {
    const uint32_t sP = sG + grp * LD_GROUP_BYTES;
    float* sS = reinterpret_cast<float*>(smem + (sP - sK) + LD_ROWS * pp);                 // [4][LD_ROWS][SP]
    const uint32_t q0 = sQ + (WIDE ? grp * LD_ROWS * pitch : 0);
    const int quarter = gw >> 1, kg = gw & 1;                // score product: channel quarter, group of 16 keys
    const int steps = ch / 16, k_lo = steps * quarter / 4, k_hi = steps * (quarter + 1) / 4;
    const int srow = gt >> 4, sk0 = (gt & 15) * 2;           // softmax: row and first of two keys of this thread
    float m_run = -INFINITY, l_run = 0.f;
    const float mul = p.scale * LD_LOG2E;
    auto group_sync = [&]() { asm volatile("bar.sync %0, 256;" ::"r"(1 + grp) : "memory"); };
    for (int t = WIDE ? 0 : grp; t < n_tiles; t += WIDE ? 1 : 2) {
      const int st = t % stages;
      mbar_wait(smem_u32(&k_full[st]), (t / stages) & 1, &s_abort, p.status, ERR_WAIT_FULL);
      const uint32_t kt = sK + st * LD_KEYS * pitch;
      {
        float s[2][4] = {};
        // K matrices: keys 0-7 ch 0-7 | keys 0-7 ch 8-15 | keys 8-15 ch 0-7 | keys 8-15 ch 8-15
        const uint32_t ka = kt + (kg * 16 + (lane & 7) + ((lane >> 4) << 3)) * pitch + ((lane >> 3) & 1) * 16;
        // Q matrices: rows 0-7 ch 0-7 | rows 8-15 ch 0-7 | rows 0-7 ch 8-15 | rows 8-15 ch 8-15
        const uint32_t qa = q0 + ((lane & 7) + (((lane >> 3) & 1) << 3)) * pitch + (lane >> 4) * 16;
#pragma unroll 5
        for (int k = k_lo; k < k_hi; ++k) {
          uint32_t a[4], b[4];
          ld_m4(ka + k * 32, b);
          ld_m4(qa + k * 32, a);
          mma_bf16(s[0], a[0], a[1], a[2], a[3], b[0], b[1]);
          mma_bf16(s[1], a[0], a[1], a[2], a[3], b[2], b[3]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int u = 0; u < 2; ++u)
            *reinterpret_cast<float2*>(sS + (quarter * LD_ROWS + u * 8 + (lane >> 2)) * SP + kg * 16 + n * 8 + (lane & 3) * 2) =
                make_float2(s[n][2 * u], s[n][2 * u + 1]);
      }
      group_sync();
      {
        float2 y = make_float2(0.f, 0.f);
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const float2 v = *reinterpret_cast<const float2*>(sS + (q * LD_ROWS + srow) * SP + sk0);
          y.x += v.x;
          y.y += v.y;
        }
        const int left = n_vis - (t0 + t) * LD_KEYS - sk0;   // keys of this thread that are visible
        y.x = left > 0 ? y.x * mul : -INFINITY;
        y.y = left > 1 ? y.y * mul : -INFINITY;
        float mx = fmaxf(y.x, y.y);
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float m_new = fmaxf(m_run, mx);                // finite: a tile holds at least one visible key
        const float alpha = ld_ex2(m_run - m_new);
        y.x = ld_ex2(y.x - m_new);
        y.y = ld_ex2(y.y - m_new);
        l_run = fmaf(l_run, alpha, y.x + y.y);               // this thread's keys only; summed at the end
        m_run = m_new;
        if ((gt & 15) == 0) s_alpha[grp][srow] = alpha;
        asm volatile("st.shared.b32 [%0], %1;" ::"r"(sP + srow * pp + sk0 * 2), "r"(pack_bf16(y.x, y.y)) : "memory");
      }
      group_sync();
      const float a0 = s_alpha[grp][lane >> 2], a1 = s_alpha[grp][8 + (lane >> 2)];
      if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
        for (int c = 0; c < CPW; ++c)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            acc[c][n][0] *= a0; acc[c][n][1] *= a0;
            acc[c][n][2] *= a1; acc[c][n][3] *= a1;
          }
      }
      const uint32_t pa = sP + ((lane & 7) + (((lane >> 3) & 1) << 3)) * pp + (lane >> 4) * 16;
      // V matrices, transposed: keys 0-7 ch 0-7 | keys 8-15 ch 0-7 | keys 0-7 ch 8-15 | keys 8-15 ch 8-15
      const uint32_t va = kt + ((lane & 7) + (((lane >> 3) & 1) << 3)) * pitch + (lane >> 4) * 16;
#pragma unroll
      for (int k = 0; k < LD_KEYS / 16; ++k) {
        uint32_t a[4];
        ld_m4(pa + k * 32, a);
#pragma unroll
        for (int c = 0; c < CPW; ++c) {
          const int sl = c * 8 + gw;
          if (sl * 16 < p.rank_p) {
            uint32_t b[4];
            ld_m4t(va + k * 16 * pitch + sl * 32, b);
            mma_bf16(acc[c][0], a[0], a[1], a[2], a[3], b[0], b[1]);
            mma_bf16(acc[c][1], a[0], a[1], a[2], a[3], b[2], b[3]);
          }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&k_empty[st]));
    }
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, o);
    if ((gt & 15) == 0) {
      s_m[grp][srow] = m_run;
      s_l[grp][srow] = l_run;
    }
  }
  __syncthreads();                                           // every tile is read
  if (s_abort) {
    // a wait ran out: give copies in flight time to finish before their memory goes
    const unsigned long long t_end = globaltimer_ns() + 200000ull;
    while (globaltimer_ns() < t_end) {
    }
  }
  if (!WIDE) {
    // the second group's sums join the first's through the ring's memory
    float* other = reinterpret_cast<float*>(smem);           // [LD_ROWS][rank_p]
    if (warp < 16 && grp == 1) {
#pragma unroll
      for (int c = 0; c < CPW; ++c)
        if ((c * 8 + gw) * 16 < p.rank_p)
#pragma unroll
          for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int u = 0; u < 2; ++u)
              *reinterpret_cast<float2*>(other + (u * 8 + (lane >> 2)) * p.rank_p + (c * 8 + gw) * 16 + n * 8 + (lane & 3) * 2) =
                  make_float2(acc[c][n][2 * u], acc[c][n][2 * u + 1]);
    }
    __syncthreads();
  }
  if (warp == 16 || (!WIDE && grp == 1)) return;
  const float* other = reinterpret_cast<const float*>(smem);
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int r = u * 8 + (lane >> 2), h = h0 + (WIDE ? grp * LD_ROWS : 0) + r;
    if (h >= p.H) continue;
    const long hi = (long)blockIdx.x * p.H + h;
    float m = s_m[grp][r], l = s_l[grp][r], f0 = 1.f, f1 = 0.f;
    if (!WIDE) {                                             // group 0 has a tile wherever group 1 has one
      const float m1 = s_m[1][r];
      const float top = fmaxf(m, m1);
      f0 = m == -INFINITY ? 0.f : ld_ex2(m - top);
      f1 = m1 == -INFINITY ? 0.f : ld_ex2(m1 - top);
      l = l * f0 + s_l[1][r] * f1;
      m = top;
    }
#pragma unroll
    for (int c = 0; c < CPW; ++c) {
      const int sl = c * 8 + gw;
      if (sl * 16 >= p.rank_p) continue;
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const int col = sl * 16 + n * 8 + (lane & 3) * 2;
        float x = acc[c][n][2 * u], y = acc[c][n][2 * u + 1];
        if (!WIDE) {
          const float2 o = *reinterpret_cast<const float2*>(other + r * p.rank_p + col);
          x = x * f0 + o.x * f1;
          y = y * f0 + o.y * f1;
        }
        if (p.splits == 1) {
          const float f = 1.0f / l;
          *reinterpret_cast<uint32_t*>(p.out + hi * p.rank_p + col) = pack_bf16(x * f, y * f);
        } else {
          *reinterpret_cast<float2*>(p.part_o + (hi * p.splits + split) * p.rank_p + col) = make_float2(x, y);
        }
      }
    }
    if (p.splits > 1 && gw == 0 && (lane & 3) == 0) {
      p.part_ml[2 * (hi * p.splits + split)] = m;
      p.part_ml[2 * (hi * p.splits + split) + 1] = l;
    }
  }
}

__global__ void __launch_bounds__(128)
latent_merge_kernel(const LatentDecode p) {
  const long base = (long)blockIdx.x * p.splits;            // blockIdx.x: (row, head)
  float top = -INFINITY;
  for (int s = 0; s < p.splits; ++s) top = fmaxf(top, p.part_ml[2 * (base + s)]);
  float den = 0.f;
  for (int s = 0; s < p.splits; ++s) {
    const float ms = p.part_ml[2 * (base + s)];
    den += ms == -INFINITY ? 0.f : p.part_ml[2 * (base + s) + 1] * ld_ex2(ms - top);
  }
  const float f = 1.0f / den;
  for (int c = threadIdx.x * 4; c < p.rank_p; c += 512) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < p.splits; ++s) {
      const float ms = p.part_ml[2 * (base + s)];
      if (ms == -INFINITY) continue;
      const float a = ld_ex2(ms - top) * f;
      const float4 v = *reinterpret_cast<const float4*>(p.part_o + (base + s) * p.rank_p + c);
      o.x = fmaf(v.x, a, o.x); o.y = fmaf(v.y, a, o.y); o.z = fmaf(v.z, a, o.z); o.w = fmaf(v.w, a, o.w);
    }
    *reinterpret_cast<uint2*>(p.out + (long)blockIdx.x * p.rank_p + c) = make_uint2(pack_bf16(o.x, o.y), pack_bf16(o.z, o.w));
  }
}

template <int CPW, bool WIDE>
static int launch_latent_decode(const LatentDecode& p, cudaStream_t st) {
  static unsigned long long prep = 0;
  if (int e = ensure_dynamic_smem((const void*)latent_decode_kernel<CPW, WIDE>, LD_LIMIT, prep)) return e;
  const int heads = WIDE ? 2 * LD_ROWS : LD_ROWS, ch = p.rank_p + p.rot_p, stages = latent_decode_stages(ch, WIDE);
  const int smem = (stages * LD_KEYS + heads) * (ch * 2 + 16) + 2 * LD_GROUP_BYTES;
  latent_decode_kernel<CPW, WIDE><<<dim3(p.n, (p.H + heads - 1) / heads, p.splits), 544, smem, st>>>(p, stages);
  return (int)cudaGetLastError();
}

template <int CPW>
static int pick_latent_decode(const LatentDecode& p, bool wide, cudaStream_t st) {
  return wide ? launch_latent_decode<CPW, true>(p, st) : launch_latent_decode<CPW, false>(p, st);
}

}  // namespace omni

using namespace omni;

extern "C" int omni_latent_rows(const LatentRows* args, int is_bf16, void* stream) {
  const LatentRows& p = *args;
  if (p.T <= 0) return RC_OK;
  if (p.H < 0 || p.rot < 0 || (p.rot & 1) || p.rot > p.rot_p || (p.dim_p & 15) || (p.rot_p & 15) || (p.q && (p.ldq & 7))) return RC_BAD_ARG;
  if ((p.q || p.z) && p.turns == nullptr) return RC_BAD_ARG;
  if (p.z && (p.pages == nullptr || p.norm == nullptr || p.slots == nullptr || (p.rank_p & 15) || (p.ldz & 7) || p.rank <= 0 ||
              p.rank > p.rank_p || p.num_slots <= 0))
    return RC_BAD_ARG;
  if (p.qc && (p.q_norm == nullptr || (p.q_rank_p & 7) || (p.ldqc & 7) || p.q_rank <= 0 || p.q_rank > p.q_rank_p)) return RC_BAD_ARG;
  if (is_bf16) latent_rows_kernel<bf16><<<p.T, 128, 0, (cudaStream_t)stream>>>(p);
  else latent_rows_kernel<float><<<p.T, 128, 0, (cudaStream_t)stream>>>(p);
  return (int)cudaGetLastError();
}

extern "C" int omni_latent_gather(const void* pages, int row_bytes, const int* tables, int bt_stride, int block_size, int num_blocks,
                                  const int* members, int n_members, const int* key_start, void* out, long rows, void* stream) {
  if (rows <= 0) return RC_OK;
  if (key_start == nullptr || (row_bytes & 15) || row_bytes <= 0 || n_members <= 0 || block_size <= 0 || num_blocks <= 0) return RC_BAD_ARG;
  long blocks = (rows * (row_bytes / 16) + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  latent_gather_kernel<<<(unsigned)blocks, 256, 0, (cudaStream_t)stream>>>((const uint4*)pages, row_bytes / 16, tables, bt_stride,
                                                                          block_size, num_blocks, members, n_members, key_start, (uint4*)out,
                                                                          rows);
  return (int)cudaGetLastError();
}

extern "C" int omni_gate_channels(void* out, long ldo, const void* gate, long ldg, long rows, int n, int is_bf16, void* stream) {
  if (rows <= 0 || n <= 0) return RC_OK;
  if ((n & 7) || (ldo & 7) || (ldg & 7)) return RC_BAD_ARG;
  long blocks = (rows * (n / 8) + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  cudaStream_t st = (cudaStream_t)stream;
  if (is_bf16) gate_channels_kernel<bf16><<<(unsigned)blocks, 256, 0, st>>>((bf16*)out, ldo, (const bf16*)gate, ldg, rows, n);
  else gate_channels_kernel<float><<<(unsigned)blocks, 256, 0, st>>>((float*)out, ldo, (const float*)gate, ldg, rows, n);
  return (int)cudaGetLastError();
}

extern "C" int omni_head_gemm(const HeadGemm* args, void* stream) {
  const HeadGemm& p = *args;
  if (p.M <= 0 || p.H <= 0) return RC_OK;
  if ((p.N & 15) || (p.K & 15) || p.N <= 0 || p.K <= 0 || (p.a_row & 7) || (p.a_head & 7) || (p.c_row & 3) || (p.c_head & 3) ||
      p.H > 65535 || p.rows_a <= 0 || p.rows_c <= 0)
    return RC_BAD_ARG;
  if ((p.M + 15) / 16 > 65535) return RC_BAD_ARG;
  head_gemm_kernel<<<dim3((p.N + 31) / 32, p.H, (p.M + 15) / 16), 128, 0, (cudaStream_t)stream>>>(p);
  return (int)cudaGetLastError();
}

// 0: the sizes do not fit the decode kernel; otherwise the heads a block serves.
extern "C" int omni_latent_decode_heads(int heads, int rank_p, int rot_p) {
  if (rank_p > 512 || rank_p <= 0 || rot_p < 0) return 0;
  if (heads > LD_ROWS && latent_decode_stages(rank_p + rot_p, true) >= 2) return 2 * LD_ROWS;
  return latent_decode_stages(rank_p + rot_p, false) >= 2 ? LD_ROWS : 0;
}

extern "C" int omni_latent_decode(const LatentDecode* args, void* stream) {
  const LatentDecode& p = *args;
  if (p.n <= 0) return RC_OK;
  const int heads = p.H > 0 ? omni_latent_decode_heads(p.H, p.rank_p, p.rot_p) : 0;
  if (heads == 0 || (p.rank_p & 15) || (p.rot_p & 15) || (p.ldp & 7) || (p.head_cols & 7) || (p.dim_p & 7) || p.splits < 1 ||
      p.splits > 65535 || p.block_size <= 0 || p.num_blocks <= 0 || p.num_seqs <= 0 || p.T <= 0)
    return RC_BAD_ARG;
  if (p.splits > 1 && (!p.part_o || !p.part_ml)) return RC_BAD_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  const bool wide = heads > LD_ROWS;
  const int rc = p.rank_p <= 128 ? pick_latent_decode<1>(p, wide, st)
                                 : (p.rank_p <= 256 ? pick_latent_decode<2>(p, wide, st) : pick_latent_decode<4>(p, wide, st));
  if (rc || p.splits == 1) return rc;
  latent_merge_kernel<<<(unsigned)(p.n * p.H), 128, 0, st>>>(p);
  return (int)cudaGetLastError();
}
