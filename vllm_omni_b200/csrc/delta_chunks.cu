// Delta-rule recurrences of prompt portions in chunks of 16 or 32 tokens on tensor cores (delta_rule.cuh says what is computed).
//
// Within a chunk the recurrence is a triangular system.  With G_t the chunk's decays through token t (scalars, or one per
// key channel), S the state before the chunk, and rows over tokens:
//   gated     (I + A) U = b V - b e^G K S,  A_ts = b_t k_t.k_s e^(G_t - G_s) below the diagonal
//             O = e^G Q S + P U,  P_ts = q_t.k_s e^(G_t - G_s) up to the diagonal
//             S <- e^G_last S + (e^(G_last - G) K)^T U
//   channel   (I + A) Y = B0 S + M V,  B0_t = u_t e^G_(t-1),  A_ts, M_ts = B0_t . (a_s u_s, k_s) e^-G_s below the diagonal
//             O = R0 S + N V - L Y,  R0_t = r_t e^G_t,  N_ts, L_ts = R0_t . (k_s, a_s u_s) e^-G_s up to the diagonal
//             S <- e^G_last S + (e^(G_last - G) k)^T V - (e^(G_last - G) a u)^T Y
//
//   prepare   a warp per 16 tokens of a (chunk, head), all chunks at once: the lower tiles (16 x 16) of the matrices and of
//             T = (I + A)^-1, left in memory as tensor-core operands; gated: the tokens' factors; channel: the decayed rows
//   sequence  one block per (portion, head, 32 or 16 value columns); a warp (or two, see there) owns eight columns of the
//             state, in registers from the first chunk to the last, and walks the chunks; operands come through a ring of
//             TMA copies that the block shares.  Every wait is bounded
//
// Everything that is not a GEMM's or convolution's bf16 result keeps fp32 precision on the way through the tensor cores: such
// an operand is two bf16 numbers, high and low part, and a product of two of them three products (16 bits and more of
// each operand count).  Raw q, k, v are bf16 as they are.  A step of the sequence is a chain of small dependent products
// with the state as operand, so warp-level products (no staging through tensor memory) are the ones that fit.
#include "delta_rule.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

constexpr int DC_TOK = 16;             // tokens of a tile; a chunk is one or two tiles
constexpr int DC_WARPS = 4;            // of the sequence kernel (and one that copies, where two share columns)

__device__ __forceinline__ void dc_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "
               "{%0, %1, %2, %3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void dc_ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void dc_ldsm4_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void dc_ldsm2_t(uint32_t addr, uint32_t& a, uint32_t& b) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];" : "=r"(a), "=r"(b) : "r"(addr) : "memory");
}
// transpose of an 8 x 8 tile of 16-bit numbers spread over the warp
__device__ __forceinline__ uint32_t dc_trans(uint32_t x) {
  uint32_t y;
  asm("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
  return y;
}
__device__ __forceinline__ void dc_copy16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void dc_bulk(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes),
               "r"(bar)
               : "memory");
}
// two numbers as pairs of bf16: high parts, and what the high parts leave
__device__ __forceinline__ void dc_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(a, b);
  const float2 f = unpack_bf16(hi);
  lo = pack_bf16(a - f.x, b - f.y);
}

// Operands of the products: B tile (k x 8) from a result tile (rows = k), high and low parts
struct SplitB {
  uint32_t h0, h1, l0, l1;
  __device__ __forceinline__ void from(const float (&c)[4]) {
    uint32_t a, b, x, y;
    dc_split(c[0], c[1], a, x);
    dc_split(c[2], c[3], b, y);
    h0 = dc_trans(a);
    h1 = dc_trans(b);
    l0 = dc_trans(x);
    l1 = dc_trans(y);
  }
};

// 16 x 16 matrix from result tiles (columns 0-7, 8-15), stored as an A operand: high parts, then low parts, 512 bytes each
__device__ __forceinline__ void dc_store_mat(uint4* dst, int lane, const float (&a)[4], const float (&b)[4]) {
  uint4 hi, lo;
  dc_split(a[0], a[1], hi.x, lo.x);
  dc_split(a[2], a[3], hi.y, lo.y);
  dc_split(b[0], b[1], hi.z, lo.z);
  dc_split(b[2], b[3], hi.w, lo.w);
  dst[lane] = hi;
  dst[32 + lane] = lo;
}

// T = (I + A)^-1 for a strictly lower triangular A [16][20] in shared memory, which T replaces.  A lane owns a column.
__device__ __forceinline__ void dc_invert(float (*a)[20], int lane) {
  float x[DC_TOK];
  const int c = lane & 15;
#pragma unroll
  for (int t = 0; t < DC_TOK; ++t) {
    float s0 = t == c ? 1.f : 0.f, s1 = 0.f;
#pragma unroll
    for (int s = 0; s < t; ++s) {
      if (s & 1) s1 = fmaf(-a[t][s], x[s], s1);
      else s0 = fmaf(-a[t][s], x[s], s0);
    }
    x[t] = s0 + s1;
  }
  __syncwarp();
  if (lane < 16)
#pragma unroll
    for (int t = 0; t < DC_TOK; ++t) a[t][c] = x[t];
  __syncwarp();
}

__device__ __forceinline__ void dc_read_tiles(const float (*a)[20], int lane, float (&c0)[4], float (&c1)[4]) {
  const int g = lane >> 2, j2 = (lane & 3) * 2;
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    c0[e] = a[g + (e >> 1) * 8][j2 + (e & 1)];
    c1[e] = a[g + (e >> 1) * 8][8 + j2 + (e & 1)];
  }
}

// Lower left tile of the inverse, -T1 A10 T0, from the tile A10 (result layout) and the inverses of the two diagonal tiles
__device__ __forceinline__ void dc_corner(const float (&a0)[4], const float (&a1)[4], const float (*t0)[20], const float (*t1)[20],
                                          int lane, float (&c0)[4], float (&c1)[4]) {
  auto product = [&](const float (&x0)[4], const float (&x1)[4], const float (&y0)[4], const float (&y1)[4], float (&r0)[4],
                     float (&r1)[4]) {
    uint32_t h[4], l[4];
    dc_split(x0[0], x0[1], h[0], l[0]);
    dc_split(x0[2], x0[3], h[1], l[1]);
    dc_split(x1[0], x1[1], h[2], l[2]);
    dc_split(x1[2], x1[3], h[3], l[3]);
    SplitB b;
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      float (&r)[4] = n ? r1 : r0;
      b.from(n ? y1 : y0);
#pragma unroll
      for (int e = 0; e < 4; ++e) r[e] = 0.f;
      dc_mma(r, h, b.h0, b.h1);
      dc_mma(r, h, b.l0, b.l1);
      dc_mma(r, l, b.h0, b.h1);
    }
  };
  float x0[4], x1[4], w0[4], w1[4];
  dc_read_tiles(t0, lane, x0, x1);
  product(a0, a1, x0, x1, w0, w1);
  dc_read_tiles(t1, lane, x0, x1);
  product(x0, x1, w0, w1, c0, c1);
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    c0[e] = -c0[e];
    c1[e] = -c1[e];
  }
}

// rows of a chunk
struct ChunkRows {
  int seq, n;
  long row0;
};
template <int M>
__device__ __forceinline__ ChunkRows dc_chunk(const DeltaRule& p, int i) {
  const int4 c = *reinterpret_cast<const int4*>(p.chunks + 4 * i);
  ChunkRows r;
  r.seq = min(max(c.x, 0), p.num_seqs - 1);
  r.n = min(max(c.z, 1), DC_TOK * M);
  r.row0 = p.q_start[r.seq] + c.y;
  return r;
}

// Matrices of a (chunk, head): `kinds` kinds of the lower tiles, in the order (0, 0), (1, 0), (1, 1); 64 uint4 each
template <int M> __host__ __device__ constexpr int dc_tiles() { return M * (M + 1) / 2; }
__device__ __forceinline__ int dc_tile(int m, int n) { return m * (m + 1) / 2 + n; }

// ------------------------------------------------------------------------------ prepare: gated
template <int M>
__global__ void __launch_bounds__(128)
delta_prepare_gated_kernel(const DeltaRule p) {
  constexpr int HEADS = 4 / M, C = DC_TOK * M, NT = dc_tiles<M>();
  __shared__ float s_a[4][DC_TOK][20], s_tok[HEADS][3][C];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, j = lane & 3;
  const int m = warp % M, slot = warp / M;                   // token tile, head of the block
  const bool live = blockIdx.y * HEADS + slot < p.H;
  const int h = min((int)blockIdx.y * HEADS + slot, p.H - 1);
  const ChunkRows ch = dc_chunk<M>(p, blockIdx.x);
  float* s_G = s_tok[slot][0];         // cumulative log decay
  float* s_b = s_tok[slot][1];
  float* s_ik = s_tok[slot][2];
  const int hk = h / (p.H / p.G);
  // rows g and g + 8 of a tile: 8 channels per lane and turn, the same order in both operands
  const bf16* u = static_cast<const bf16*>(p.u) + hk * p.dp;
  const int ko = p.G * p.dp;
  auto row = [&](int tile, int r) { return (ch.row0 + min(tile * DC_TOK + r, ch.n - 1)) * p.ldu; };
  const long ra = row(m, g), rb = row(m, g + 8);
  float kk[M][2][4] = {}, qk[M][2][4] = {};
  float ss[4] = {};                    // sums of squares: k rows g, g + 8, q rows g, g + 8
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  auto load = [&](long at) { return *reinterpret_cast<const uint4*>(u + at); };
  for (int c = j * 8; c < p.dp + j * 8; c += 32) {
    const bool in = c < p.dp;
    const uint4 ka = in ? load(ra + ko + c) : zero, kb = in ? load(rb + ko + c) : zero;
    const uint4 qa = in ? load(ra + c) : zero, qb = in ? load(rb + c) : zero;
    const uint32_t kf[2][4] = {{ka.x, kb.x, ka.y, kb.y}, {ka.z, kb.z, ka.w, kb.w}};
    const uint32_t qf[2][4] = {{qa.x, qb.x, qa.y, qb.y}, {qa.z, qb.z, qa.w, qb.w}};
    uint32_t cf[2][4];                 // keys of the first tile
    if (M == 2 && m == 1) {
      const uint4 a = in ? load(row(0, g) + ko + c) : zero, b = in ? load(row(0, g + 8) + ko + c) : zero;
      cf[0][0] = a.x; cf[0][1] = b.x; cf[0][2] = a.y; cf[0][3] = b.y;
      cf[1][0] = a.z; cf[1][1] = b.z; cf[1][2] = a.w; cf[1][3] = b.w;
    }
#pragma unroll
    for (int s = 0; s < 2; ++s) {
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        dc_mma(kk[0][n], kf[s], kf[s][n], kf[s][n + 2]);
        dc_mma(qk[0][n], qf[s], kf[s][n], kf[s][n + 2]);
        if (M == 2 && m == 1) {
          dc_mma(kk[M - 1][n], kf[s], cf[s][n], cf[s][n + 2]);
          dc_mma(qk[M - 1][n], qf[s], cf[s][n], cf[s][n + 2]);
        }
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 fk = unpack_bf16(kf[s][e]), fq = unpack_bf16(qf[s][e]);
        ss[e & 1] = fmaf(fk.x, fk.x, fmaf(fk.y, fk.y, ss[e & 1]));
        ss[2 + (e & 1)] = fmaf(fq.x, fq.x, fmaf(fq.y, fq.y, ss[2 + (e & 1)]));
      }
    }
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    ss[e] += __shfl_xor_sync(0xffffffffu, ss[e], 1);
    ss[e] += __shfl_xor_sync(0xffffffffu, ss[e], 2);
  }
  const float ik[2] = {1.0f / sqrtf(ss[0] + p.unit_eps), 1.0f / sqrtf(ss[1] + p.unit_eps)};
  const float iq[2] = {p.q_mul / sqrtf(ss[2] + p.unit_eps), p.q_mul / sqrtf(ss[3] + p.unit_eps)};
  if (j == 0) {
    s_ik[m * DC_TOK + g] = ik[0];
    s_ik[m * DC_TOK + g + 8] = ik[1];
  }
  // a lane per token: step size, cumulative log decay
  const int t = lane & (C - 1);
  const bf16* pr = static_cast<const bf16*>(p.proj) + (ch.row0 + min(t, ch.n - 1)) * p.ldp;
  const float beta = t < ch.n ? dr_sigmoid((float)pr[p.b_col + h]) : 0.f;
  float G = t < ch.n ? p.rate[h] * dr_softplus((float)pr[p.a_col + h] + p.dt_bias[h]) : 0.f;
#pragma unroll
  for (int o = 1; o < C; o <<= 1) {
    const float v = __shfl_up_sync(0xffffffffu, G, o, C);
    if (t >= o) G += v;
  }
  const float G_last = __shfl_sync(0xffffffffu, G, C - 1, C);
  if (m == 0 && lane < C) {
    s_G[t] = G;
    s_b[t] = beta;
  }
  __syncthreads();
  const long at = (long)blockIdx.x * p.H + h;
  uint4* mats = static_cast<uint4*>(p.mats) + at * (2 * NT * 64);
  float* coef = p.coef + at * (4 * C + 4);
  // tile (m, n) of the system and of the output matrix
  auto finish = [&](int n, float (&a)[2][4], float (&q)[2][4]) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = m * DC_TOK + g + (e >> 1) * 8;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int s = n * DC_TOK + half * 8 + j * 2 + (e & 1);
        const float d = r >= s ? expf(s_G[r] - s_G[s]) * s_ik[s] : 0.f;
        a[half][e] *= r > s ? s_b[r] * ik[e >> 1] * d : 0.f;
        q[half][e] *= iq[e >> 1] * d;
      }
    }
    if (live) dc_store_mat(mats + (NT + dc_tile(m, n)) * 64, lane, q[0], q[1]);
  };
  finish(m, kk[0], qk[0]);
  if (M == 2 && m == 1) finish(0, kk[M - 1], qk[M - 1]);
#pragma unroll
  for (int e = 0; e < 4; ++e)
#pragma unroll
    for (int half = 0; half < 2; ++half) s_a[warp][g + (e >> 1) * 8][half * 8 + j * 2 + (e & 1)] = kk[0][half][e];
  if (live && j == 0) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = m * DC_TOK + g + 8 * half;
      const float e = expf(s_G[r]);
      const float4 c = make_float4(s_b[r], -s_b[r] * e * ik[half], e * iq[half], r < ch.n ? expf(G_last - s_G[r]) * ik[half] : 0.f);
      *reinterpret_cast<float4*>(coef + 4 * r) = c;
    }
  }
  if (live && m == 0 && lane == 0) *reinterpret_cast<float4*>(coef + 4 * C) = make_float4(expf(G_last), 0.f, 0.f, 0.f);
  __syncwarp();
  dc_invert(s_a[warp], lane);
  float c0[4], c1[4];
  dc_read_tiles(s_a[warp], lane, c0, c1);
  if (live) dc_store_mat(mats + dc_tile(m, m) * 64, lane, c0, c1);
  if (M == 2) {
    __syncthreads();                                         // the first tile's inverse is there
    if (m == 1) {
      dc_corner(kk[M - 1][0], kk[M - 1][1], s_a[warp - 1], s_a[warp], lane, c0, c1);
      if (live) dc_store_mat(mats + dc_tile(1, 0) * 64, lane, c0, c1);
    }
  }
}

// ---------------------------------------------------------------------------- prepare: channel
constexpr int PC_PITCH = 64 * 2 + 16;  // bytes of a row of 64 channels

template <int M>
__global__ void __launch_bounds__(32 * M)
delta_prepare_channel_kernel(const DeltaRule p) {
  constexpr int C = DC_TOK * M, NT = dc_tiles<M>();
  constexpr int ROW32 = PC_PITCH / 4, ARR32 = C * ROW32;
  __shared__ __align__(16) uint32_t s_rows[8 * ARR32];       // decayed rows: b0, r0, k / G, a u / G (high, low)
  __shared__ float s_a[M][DC_TOK][20];
  __shared__ float2 s_tot[M][32];                            // log decay of a tile's tokens
  __shared__ float s_ik[M][DC_TOK];                          // one over the length of a key
  const int m = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, j = lane & 3;
  const int h = blockIdx.y;
  const ChunkRows ch = dc_chunk<M>(p, blockIdx.x);
  const bf16* proj = static_cast<const bf16*>(p.proj) + (long)h * p.dp;
  const bf16* z = static_cast<const bf16*>(p.z) + (long)h * p.dp;
  const long at = (long)blockIdx.x * p.H + h;
  const int pitch = p.dp / 2 + 4, tile = C * pitch;          // channel pairs of a row (padded as in shared memory), of an operand
  uint32_t* tiles = static_cast<uint32_t*>(p.tiles) + at * (8 * tile);
  uint4* mats = static_cast<uint4*>(p.mats) + at * (4 * NT * 64);
  const uint32_t base = smem_u32(s_rows);
  constexpr uint32_t ARR = C * PC_PITCH;
  // the raw rows of 64 channels, where the operands k / G and a u / G take their places channel by channel: r, k, a, z
  auto fetch = [&](int cb) {
    for (int x = threadIdx.x; x < 4 * C * 8; x += 32 * M) {
      const int arr = x / (C * 8), t = x / 8 % C, c = cb + x % 8 * 8;
      const bf16* src = arr == 3 ? z : proj + (arr == 0 ? p.q_col : (arr == 1 ? p.k_col : p.a_col));
      const long ld = arr == 3 ? p.ldz : p.ldp;
      if (c < p.dp) dc_copy16(base + (4 + arr) * ARR + t * PC_PITCH + x % 8 * 16, src + (ch.row0 + min(t, ch.n - 1)) * ld + c);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0);
  // lengths of the keys: two lanes per token
  {
    const int t = lane & 15;
    const bf16* k = proj + p.k_col + (ch.row0 + min(m * DC_TOK + t, ch.n - 1)) * p.ldp;
    float ss = 0.f;
    for (int c = (lane >> 4) * 8; c < p.dp; c += 16) {
      float v[8];
      load8<bf16>(k + c, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
    }
    ss += __shfl_xor_sync(0xffffffffu, ss, 16);
    if (lane < 16) s_ik[m][t] = 1.0f / sqrtf(ss + p.unit_eps);
    __syncwarp();
  }
  float am[M][2][4] = {}, mm[M][2][4] = {}, nm[M][2][4] = {}, lm[M][2][4] = {};      // [0]: diagonal tile, [1]: left of it
  for (int cb = 0; cb < p.dp; cb += 64) {
    if (cb > 0) {
      __syncthreads();                                       // the products of the last 64 channels are done
      fetch(cb);
    }
    const int c = cb + lane * 2;
    const bool in = c < p.dp;
    const int cc = in ? c : 0;
    const float2 db = *reinterpret_cast<const float2*>(p.decay_bias + h * p.dp + cc);
    const float2 rb = *reinterpret_cast<const float2*>(p.removal_bias + h * p.dp + cc);
    const int nt = min(max(ch.n - m * DC_TOK, 0), DC_TOK);   // tokens of the tile
    auto log_decay = [&](uint32_t w) {
      const float2 f = unpack_bf16(w);
      return make_float2(p.decay_scale * __fdividef(1.0f, 1.0f + __expf(-(f.x + db.x))),
                         p.decay_scale * __fdividef(1.0f, 1.0f + __expf(-(f.y + db.y))));
    };
    auto raw = [&](int arr, int t) { return s_rows[(4 + arr) * ARR32 + (m * DC_TOK + t) * ROW32 + lane]; };
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    float2 sum = make_float2(0.f, 0.f);
#pragma unroll 8
    for (int t = 0; t < DC_TOK; ++t) {
      const float2 l = log_decay(raw(3, t));
      if (t < nt) {
        sum.x += l.x;
        sum.y += l.y;
      }
    }
    s_tot[m][lane] = sum;
    __syncthreads();
    float2 G = make_float2(0.f, 0.f), total = s_tot[0][lane];               // cumulative log decay
    if (M == 2) {
      if (m == 1) G = total;
      total.x += s_tot[M - 1][lane].x;
      total.y += s_tot[M - 1][lane].y;
    }
    const float tx = __expf(total.x), ty = __expf(total.y);
    float e0 = __expf(G.x), e1 = __expf(G.y);                // decays so far
#pragma unroll 4
    for (int t = 0; t < DC_TOK; ++t) {
      const uint32_t rw = raw(0, t), kw = raw(1, t), aw = raw(2, t), zw = raw(3, t);
      float2 b0 = make_float2(0.f, 0.f), r0 = b0, ki = b0, ai = b0;
      if (t < nt && in) {
        const float2 r = unpack_bf16(rw), k = unpack_bf16(kw), a = unpack_bf16(aw), l = log_decay(zw);
        const float ik = s_ik[m][t];
        b0 = make_float2(k.x * ik * e0, k.y * ik * e1);
        G.x += l.x;
        G.y += l.y;
        e0 = __expf(G.x);
        e1 = __expf(G.y);
        r0 = make_float2(r.x * e0, r.y * e1);
        ki = make_float2(k.x * __expf(-G.x), k.y * __expf(-G.y));
        ai = make_float2(__fdividef(ik, 1.0f + __expf(-(a.x + rb.x))) * ki.x, __fdividef(ik, 1.0f + __expf(-(a.y + rb.y))) * ki.y);
      }
      const int tok = m * DC_TOK + t;
      uint32_t hi, lo;
      uint32_t* dst = s_rows + tok * ROW32 + lane;
      uint32_t* out = tiles + tok * pitch + c / 2;
      auto put = [&](int x, float2 v, bool shared, int global) {           // a pair of channels of operand x, high and low parts
        dc_split(v.x, v.y, hi, lo);
        if (shared) {
          dst[x * ARR32] = hi;
          dst[(x + 1) * ARR32] = lo;
        }
        if (in && global >= 0) {
          out[global * tile] = hi;
          out[(global + 1) * tile] = lo;
        }
      };
      put(0, b0, true, 0);
      put(2, r0, true, 2);
      put(4, ki, true, -1);
      put(6, ai, true, -1);
      put(0, make_float2(ki.x * tx, ki.y * ty), false, 4);
      put(0, make_float2(-ai.x * tx, -ai.y * ty), false, 6);
    }
    if (in && m == 0) *reinterpret_cast<float2*>(p.coef + at * p.dp + c) = make_float2(tx, ty);
    __syncthreads();
    const uint32_t a0 = base + ((lane & 7) + ((lane >> 3) & 1) * 8) * PC_PITCH + (lane >> 4) * 16, mine = a0 + m * DC_TOK * PC_PITCH;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      if (cb + k * 16 >= p.dp) break;
      uint32_t x[4][4];                                      // b0, r0 of this tile
#pragma unroll
      for (int i = 0; i < 4; ++i) dc_ldsm4(mine + i * ARR + k * 32, x[i]);
#pragma unroll
      for (int n = 0; n < M; ++n) {                          // columns: this tile, then the one before
        if (n > m) continue;
        uint32_t y[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) dc_ldsm4((n ? a0 : mine) + (4 + i) * ARR + k * 32, y[i]);
        // high high, high low, low high
        auto product = [&](float (&r)[2][4], int i, int q) {
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            dc_mma(r[half], x[i], y[q][half], y[q][half + 2]);
            dc_mma(r[half], x[i], y[q + 1][half], y[q + 1][half + 2]);
            dc_mma(r[half], x[i + 1], y[q][half], y[q][half + 2]);
          }
        };
        product(am[n], 0, 2);
        product(mm[n], 0, 0);
        product(nm[n], 2, 0);
        product(lm[n], 2, 2);
      }
    }
  }
#pragma unroll
  for (int n = 0; n < 2; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = g + (e >> 1) * 8, s = n * 8 + j * 2 + (e & 1);
      s_a[m][r][s] = r > s ? am[0][n][e] : 0.f;
      if (r <= s) mm[0][n][e] = 0.f;
      if (r < s) nm[0][n][e] = 0.f;
      lm[0][n][e] = r < s ? 0.f : -lm[0][n][e];
      if (M == 2) lm[M - 1][n][e] = m == 1 ? -lm[M - 1][n][e] : lm[M - 1][n][e];
    }
#pragma unroll
  for (int n = 0; n < M; ++n) {
    if (n > m) continue;
    const int i = dc_tile(m, m - n);
    dc_store_mat(mats + (NT + i) * 64, lane, mm[n][0], mm[n][1]);
    dc_store_mat(mats + (2 * NT + i) * 64, lane, nm[n][0], nm[n][1]);
    dc_store_mat(mats + (3 * NT + i) * 64, lane, lm[n][0], lm[n][1]);
  }
  __syncwarp();
  dc_invert(s_a[m], lane);
  float c0[4], c1[4];
  dc_read_tiles(s_a[m], lane, c0, c1);
  dc_store_mat(mats + dc_tile(m, m) * 64, lane, c0, c1);
  if (M == 2) {
    __syncthreads();                                         // the first tile's inverse is there
    if (m == 1) {
      dc_corner(am[M - 1][0], am[M - 1][1], s_a[0], s_a[M - 1], lane, c0, c1);
      dc_store_mat(mats + dc_tile(1, 0) * 64, lane, c0, c1);
    }
  }
}

// ----------------------------------------------------------------------------------- sequence
// Bytes of a stage: rows of the operands, values, matrices, factors.  Gated: k, then q, in boxes of 64 channels of all
// tokens, 128-byte swizzle.  Channel: eight operands as prepared, rows of `pitch` bytes (an odd multiple of 16:
// conflict-free ldmatrix).
struct DeltaStage {
  int pitch, arr, values, mats, coef, bytes;
};
template <bool CHANNEL, int M, int COLS>
__host__ __device__ __forceinline__ DeltaStage delta_stage(int dp) {
  DeltaStage s;
  s.pitch = CHANNEL ? dp * 2 + 16 : 128;
  s.arr = M * DC_TOK * (CHANNEL ? s.pitch : (dp + 63) / 64 * 128);
  s.values = ((CHANNEL ? 8 : 2) * s.arr + 127) / 128 * 128;
  s.mats = s.values + M * DC_TOK * COLS * 2;
  s.coef = s.mats + (CHANNEL ? 4 : 2) * dc_tiles<M>() * 1024;
  s.bytes = (s.coef + (CHANNEL ? dp * 4 : (4 * M * DC_TOK + 4) * 4) + 1023) / 1024 * 1024;
  return s;
}

// KS: 16-channel steps of the key channels that the state's registers hold.  EXACT: dp = 16 KS, so that a chunk's products
// are straight-line code; otherwise dp <= 16 KS.  M: tiles of 16 tokens in a chunk.  SPLIT = 2: two warps share eight
// columns, each has half of the key channels; they add up what the state answers in shared memory, and each finishes the
// output of one token tile.  For few portions and heads, where the chain of a chunk's products is what takes the time.
template <bool CHANNEL, int KS, bool EXACT, int M, int SPLIT>
__global__ void __launch_bounds__(32 * (DC_WARPS + SPLIT - 1), SPLIT == 1 && KS <= 8 ? 4 : 1)
delta_sequence_kernel(const __grid_constant__ CUtensorMap tmU, const __grid_constant__ CUtensorMap tmV,
                      const __grid_constant__ DeltaRule p, const int stages) {
  constexpr int C = M * DC_TOK, NT = dc_tiles<M>(), GROUPS = DC_WARPS / SPLIT, COLS = 8 * GROUPS, VPITCH = COLS * 2;
  constexpr int KW = KS / SPLIT, NM = (CHANNEL ? 4 : 2) * NT * 64;
  static_assert(SPLIT == 1 || (SPLIT == 2 && M == 2), "a warp of a pair finishes one tile");
  extern __shared__ uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t full[3], empty[3];
  __shared__ __align__(16) float4 s_ex[SPLIT == 2 ? 2 : 1][DC_WARPS][3][SPLIT == 2 ? 32 : 1];
  __shared__ int s_abort;
  const int dp = EXACT ? 16 * KS : p.dp;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, j2 = (lane & 3) * 2;
  const int seq = min(max(p.long_list[2 * blockIdx.z], 0), p.num_seqs - 1), first = p.long_list[2 * blockIdx.z + 1];
  const int h = blockIdx.y, col0 = blockIdx.x * COLS, hk = h / (p.H / p.G);
  const long row0 = p.q_start[seq];
  const int n = (int)(p.q_start[seq + 1] - row0);
  const int n_chunks = min((n + C - 1) / C, p.n_chunks - first);
  const DeltaStage lay = delta_stage<CHANNEL, M, COLS>(dp);
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint8_t* smem = smem_raw + (base - smem_u32(smem_raw));
  if (tid == 0) {
    s_abort = 0;
    tma_prefetch_desc(&tmU);
    tma_prefetch_desc(&tmV);
    for (int i = 0; i < 3; ++i) {
      mbar_init(smem_u32(&full[i]), 1);
      mbar_init(smem_u32(&empty[i]), DC_WARPS);
    }
    fence_mbar_init();
  }
  __syncthreads();

  // the copies of chunk i (one thread); rows past the portion's end are another's or zero: finite, and their factors are zero
  auto copy = [&](int i) {
    const int slot = i % stages, boxes = (dp + 63) / 64, row = (int)row0 + i * C;
    const uint32_t bar = smem_u32(&full[slot]), dst = base + slot * lay.bytes;
    const uint32_t f_bytes = CHANNEL ? dp * 4 : (4 * C + 4) * 4;
    const long at = (long)(first + i) * p.H + h;
    mbar_wait(smem_u32(&empty[slot]), ((i / stages) & 1) ^ 1, &s_abort, p.status, ERR_WAIT_EMPTY);
    mbar_expect_tx(bar, (CHANNEL ? 8 : 2) * lay.arr + C * VPITCH + NM * 16 + f_bytes);
    if (CHANNEL) {
      dc_bulk(dst, static_cast<const uint8_t*>(p.tiles) + at * (8 * lay.arr), 8 * lay.arr, bar);
    } else {
      for (int x = 0; x < boxes; ++x) tma_load_2d(dst + x * C * 128, &tmU, bar, (p.G + hk) * dp + 64 * x, row);
      for (int x = 0; x < boxes; ++x) tma_load_2d(dst + lay.arr + x * C * 128, &tmU, bar, hk * dp + 64 * x, row);
    }
    tma_load_2d(dst + lay.values, &tmV, bar, h * p.vp + col0, row);
    dc_bulk(dst + lay.mats, static_cast<const uint4*>(p.mats) + at * NM, NM * 16, bar);
    dc_bulk(dst + lay.coef, reinterpret_cast<const uint8_t*>(p.coef) + at * f_bytes, f_bytes, bar);
  };

  if (SPLIT == 2 && warp == DC_WARPS) {                      // a warp of its own where the chain of products counts
    if (elect_one())
      for (int i = 0; i < n_chunks; ++i) copy(i);
  } else {
    if (SPLIT == 1 && warp == 0 && elect_one())
      for (int i = 0; i < min(stages - 1, n_chunks); ++i) copy(i);
    __syncwarp();
    int sin, sout;
    delta_rows(p, seq, sin, sout);
    const int grp = warp % GROUPS, kh = warp / GROUPS, k0 = kh * KW;
    const int col = col0 + grp * 8;                          // this warp's columns
    const bool used = col < p.vp;
    float S[KW][4];                                          // rows g, g + 8 of 16 key channels, columns j2, j2 + 1
    {
      const float* src = p.state + ((long)sin * p.H + h) * dp * p.vp + col + j2;
      const bool have = used && p.context[seq] > 0;
#pragma unroll
      for (int k = 0; k < KW; ++k)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = (k0 + k) * 16 + g + 8 * e;
          const float2 v = have && (EXACT || (k0 + k) * 16 < dp) ? *reinterpret_cast<const float2*>(src + (long)r * p.vp) : make_float2(0.f, 0.f);
          S[k][2 * e] = v.x;
          S[k][2 * e + 1] = v.y;
        }
    }
    bf16* out = static_cast<bf16*>(p.raw) + row0 * p.H * p.vp + (long)h * p.vp + col + j2;
    // where a lane's 16 bytes of a 16 x 16 operand are: tokens x channels, and channels x tokens (transposed on the way)
    const uint32_t a_row = ((lane & 7) + ((lane >> 3) & 1) * 8) * lay.pitch, t_row = ((lane & 7) + (lane >> 4) * 8) * lay.pitch;
    const uint32_t a_vec = (CHANNEL ? lane >> 4 : (lane >> 4) ^ (lane & 7)) * 16;
    const uint32_t t_vec = (CHANNEL ? (lane >> 3) & 1 : ((lane >> 3) & 1) ^ (lane & 7)) * 16;
    auto place = [&](uint32_t row, uint32_t vec, int arr, int m, int k) {
      const uint32_t at = row + arr * lay.arr + m * DC_TOK * lay.pitch;
      k += k0;
      return CHANNEL ? at + vec + k * 32 : at + (k >> 2) * (C * 128) + (vec ^ ((k & 3) * 32));
    };
    auto at_a = [&](int arr, int m, int k) { return place(a_row, a_vec, arr, m, k); };
    auto at_t = [&](int arr, int m, int k) { return place(t_row, t_vec, arr, m, k); };
    int stage = 0;
    uint32_t ph = 0;
    for (int i = 0; i < n_chunks; ++i) {
      mbar_wait(smem_u32(&full[stage]), ph, &s_abort, p.status, ERR_WAIT_FULL);
      const int so = stage * lay.bytes;
      const uint32_t bar = smem_u32(&empty[stage]);
      if (++stage == stages) {
        stage = 0;
        ph ^= 1;
      }
      if (!used) {
        if (lane == 0) mbar_arrive(bar);
        continue;
      }
      const uint32_t st = base + so;
      const uint4* mats = reinterpret_cast<const uint4*>(smem + so + lay.mats) + lane;
      // what the state gives for the chunk's keys (x) and queries (o)
      float x[M][2][4] = {}, o[M][2][4] = {};
      SplitB s[KW];
      auto queries = [&](int k) {
#pragma unroll
        for (int m = 0; m < M; ++m) {
          uint32_t a[4];
          dc_ldsm4(st + at_a(CHANNEL ? 2 : 1, m, k), a);
          dc_mma(o[m][0], a, s[k].h0, s[k].h1);
          dc_mma(o[m][1], a, s[k].l0, s[k].l1);
          if (CHANNEL) {
            dc_ldsm4(st + at_a(3, m, k), a);
            dc_mma(o[m][1], a, s[k].h0, s[k].h1);
          }
        }
      };
#pragma unroll
      for (int k = 0; k < KW; ++k) {
        if (!EXACT && (k0 + k) * 16 >= dp) break;
        s[k].from(S[k]);
#pragma unroll
        for (int m = 0; m < M; ++m) {
          uint32_t a[4];
          dc_ldsm4(st + at_a(0, m, k), a);
          dc_mma(x[m][0], a, s[k].h0, s[k].h1);
          dc_mma(x[m][1], a, s[k].l0, s[k].l1);
          if (CHANNEL) {
            dc_ldsm4(st + at_a(1, m, k), a);
            dc_mma(x[m][1], a, s[k].h0, s[k].h1);
          }
        }
        if (SPLIT == 2) queries(k);                          // more chains side by side; with one warp they fill later gaps
      }
      if (SPLIT == 1)
#pragma unroll
        for (int k = 0; k < KW; ++k) {
          if (!EXACT && (k0 + k) * 16 >= dp) break;
          queries(k);
        }
#pragma unroll
      for (int m = 0; m < M; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          x[m][0][e] += x[m][1][e];
          o[m][0][e] += o[m][1][e];
          x[m][1][e] = o[m][1][e] = 0.f;
        }
      if constexpr (SPLIT == 2) {                            // what the other half of the key channels gives
        auto as4 = [](const float (&v)[4]) { return make_float4(v[0], v[1], v[2], v[3]); };
        auto plus = [](float (&v)[4], const float4& a) {
          v[0] += a.x;
          v[1] += a.y;
          v[2] += a.z;
          v[3] += a.w;
        };
        float4(*mine)[32] = s_ex[i & 1][warp], (*other)[32] = s_ex[i & 1][warp ^ GROUPS];
        mine[0][lane] = as4(x[0][0]);
        mine[1][lane] = as4(x[1][0]);
        mine[2][lane] = kh ? as4(o[0][0]) : as4(o[1][0]);
        asm volatile("bar.sync %0, 64;" ::"r"(1 + grp) : "memory");
        plus(x[0][0], other[0][lane]);
        plus(x[1][0], other[1][lane]);
        const float4 c = other[2][lane];                     // only one of the two tiles is finished here
        plus(o[0][0], c);
        plus(o[1][0], c);
      }
      if (SPLIT == 1 && warp == 0) {                         // into the place of chunk i - 1
        if (elect_one() && i + stages - 1 < n_chunks) copy(i + stages - 1);
        __syncwarp();
      }
      const bool has[2] = {SPLIT == 1 || kh == 0, SPLIT == 1 || kh == 1};     // token tiles whose output this warp finishes
      // r += tile (m, n) of matrix `kind` times split rows, or times bf16 rows
      auto times = [&](float (&r)[4], int kind, int m, int n, const SplitB& b) {
        const uint4 h4 = mats[(kind * NT + dc_tile(m, n)) * 64], l4 = mats[(kind * NT + dc_tile(m, n)) * 64 + 32];
        const uint32_t hi[4] = {h4.x, h4.y, h4.z, h4.w}, lo[4] = {l4.x, l4.y, l4.z, l4.w};
        dc_mma(r, hi, b.h0, b.h1);
        dc_mma(r, hi, b.l0, b.l1);
        dc_mma(r, lo, b.h0, b.h1);
      };
      auto times_raw = [&](float (&r)[4], int kind, int m, int n, const uint32_t (&b)[2]) {
        const uint4 h4 = mats[(kind * NT + dc_tile(m, n)) * 64], l4 = mats[(kind * NT + dc_tile(m, n)) * 64 + 32];
        const uint32_t hi[4] = {h4.x, h4.y, h4.z, h4.w}, lo[4] = {l4.x, l4.y, l4.z, l4.w};
        dc_mma(r, hi, b[0], b[1]);
        dc_mma(r, lo, b[0], b[1]);
      };
      float y[M][4] = {}, y2[4] = {};                        // y2: the lower left tile's share, a chain of its own
      SplitB b[M];
      if (CHANNEL) {
        uint32_t v[M][2];
#pragma unroll
        for (int m = 0; m < M; ++m) dc_ldsm2_t(st + lay.values + (m * DC_TOK + (lane & 15)) * VPITCH + grp * 16, v[m][0], v[m][1]);
#pragma unroll
        for (int m = 0; m < M; ++m) {
#pragma unroll
          for (int q = 0; q <= m; ++q) times_raw(x[m][1], 1, m, q, v[q]);
#pragma unroll
          for (int e = 0; e < 4; ++e) x[m][0][e] += x[m][1][e];
          b[m].from(x[m][0]);
        }
#pragma unroll
        for (int m = 0; m < M; ++m) times(y[m], 0, m, m, b[m]);
        if (M == 2) times(y2, 0, 1, 0, b[0]);
#pragma unroll
        for (int m = 0; m < M; ++m) {
          if (m == 1)
#pragma unroll
            for (int e = 0; e < 4; ++e) y[m][e] += y2[e];
          b[m].from(y[m]);
        }
        const float* decay = reinterpret_cast<const float*>(smem + so + lay.coef) + k0 * 16 + g;
#pragma unroll
        for (int k = 0; k < KW; ++k) {
          if (!EXACT && (k0 + k) * 16 >= dp) break;
          const float d0 = decay[k * 16], d1 = decay[k * 16 + 8];
          S[k][0] *= d0;
          S[k][1] *= d0;
          S[k][2] *= d1;
          S[k][3] *= d1;
#pragma unroll
          for (int m = 0; m < M; ++m) {
            uint32_t a[4];
            dc_ldsm4_t(st + at_t(4, m, k), a);
            dc_mma(S[k], a, v[m][0], v[m][1]);
            dc_ldsm4_t(st + at_t(5, m, k), a);
            dc_mma(S[k], a, v[m][0], v[m][1]);
            dc_ldsm4_t(st + at_t(6, m, k), a);
            dc_mma(S[k], a, b[m].h0, b[m].h1);
            dc_mma(S[k], a, b[m].l0, b[m].l1);
            dc_ldsm4_t(st + at_t(7, m, k), a);
            dc_mma(S[k], a, b[m].h0, b[m].h1);
          }
        }
#pragma unroll
        for (int m = 0; m < M; ++m) {
          if (!has[m]) continue;
#pragma unroll
          for (int q = 0; q <= m; ++q) {
            times_raw(o[m][0], 2, m, q, v[q]);
            times(o[m][1], 3, m, q, b[q]);
          }
#pragma unroll
          for (int e = 0; e < 4; ++e) o[m][0][e] += o[m][1][e];
        }
      } else {
        const float* coef = reinterpret_cast<const float*>(smem + so + lay.coef);
        float4 ca[M], cb[M];                                 // factors of rows g, g + 8
#pragma unroll
        for (int m = 0; m < M; ++m) {
          ca[m] = *reinterpret_cast<const float4*>(coef + 4 * (m * DC_TOK + g));
          cb[m] = *reinterpret_cast<const float4*>(coef + 4 * (m * DC_TOK + g + 8));
          const uint8_t* vp = smem + so + lay.values + (m * DC_TOK + g) * VPITCH + (grp * 8 + j2) * 2;
          const float2 va = unpack_bf16(*reinterpret_cast<const uint32_t*>(vp)), vb = unpack_bf16(*reinterpret_cast<const uint32_t*>(vp + 8 * VPITCH));
          float (&x0)[4] = x[m][0];
          x0[0] = fmaf(ca[m].y, x0[0], ca[m].x * va.x);
          x0[1] = fmaf(ca[m].y, x0[1], ca[m].x * va.y);
          x0[2] = fmaf(cb[m].y, x0[2], cb[m].x * vb.x);
          x0[3] = fmaf(cb[m].y, x0[3], cb[m].x * vb.y);
          b[m].from(x0);
        }
#pragma unroll
        for (int m = 0; m < M; ++m) times(y[m], 0, m, m, b[m]);
        if (M == 2) times(y2, 0, 1, 0, b[0]);
        SplitB w[M];                                         // what is written, with the decays to the chunk's end
#pragma unroll
        for (int m = 0; m < M; ++m) {
          if (m == 1)
#pragma unroll
            for (int e = 0; e < 4; ++e) y[m][e] += y2[e];
          const float u[4] = {y[m][0] * ca[m].w, y[m][1] * ca[m].w, y[m][2] * cb[m].w, y[m][3] * cb[m].w};
          w[m].from(u);
        }
        const float decay = coef[4 * C];
#pragma unroll
        for (int k = 0; k < KW; ++k) {
          if (!EXACT && (k0 + k) * 16 >= dp) break;
#pragma unroll
          for (int e = 0; e < 4; ++e) S[k][e] *= decay;
#pragma unroll
          for (int m = 0; m < M; ++m) {
            uint32_t a[4];
            dc_ldsm4_t(st + at_t(0, m, k), a);
            dc_mma(S[k], a, w[m].h0, w[m].h1);
            dc_mma(S[k], a, w[m].l0, w[m].l1);
          }
        }
#pragma unroll
        for (int m = 0; m < M; ++m) {
          b[m].from(y[m]);
          o[m][0][0] *= ca[m].z;
          o[m][0][1] *= ca[m].z;
          o[m][0][2] *= cb[m].z;
          o[m][0][3] *= cb[m].z;
        }
#pragma unroll
        for (int m = 0; m < M; ++m) {
          if (!has[m]) continue;
#pragma unroll
          for (int q = 0; q <= m; ++q) times(o[m][0], 1, m, q, b[q]);
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(bar);
#pragma unroll
      for (int m = 0; m < M; ++m) {
        if (!has[m]) continue;
        const int t = i * C + m * DC_TOK + g;
        if (t < n) *reinterpret_cast<uint32_t*>(out + (long)t * p.H * p.vp) = pack_bf16(o[m][0][0], o[m][0][1]);
        if (t + 8 < n) *reinterpret_cast<uint32_t*>(out + (long)(t + 8) * p.H * p.vp) = pack_bf16(o[m][0][2], o[m][0][3]);
      }
    }
    if (used && sout >= 0) {
      float* dst = p.state + ((long)sout * p.H + h) * dp * p.vp + col + j2;
#pragma unroll
      for (int k = 0; k < KW; ++k)
#pragma unroll
        for (int e = 0; e < 2; ++e)
          if (EXACT || (k0 + k) * 16 < dp)
            *reinterpret_cast<float2*>(dst + (long)((k0 + k) * 16 + g + 8 * e) * p.vp) = make_float2(S[k][2 * e], S[k][2 * e + 1]);
    }
  }
  __syncthreads();
  if (s_abort) {
    // a wait ran out: give copies in flight time to finish before their memory goes
    const unsigned long long t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) {
    }
  }
}

// [rows, cols] bf16 as boxes of box_rows x box_cols without swizzle
static int rows_tmap(CUtensorMap* out, const void* ptr, uint64_t rows, uint64_t cols, uint64_t pitch, uint32_t box_rows, uint32_t box_cols) {
  EncodeTiledFn enc = get_encode_tiled();
  if (!enc) return RC_NO_DRIVER;
  if ((reinterpret_cast<uintptr_t>(ptr) & 15) || (pitch & 15)) return RC_BAD_ARG;
  cuuint64_t gdim[2] = {cols, rows}, gstr[1] = {pitch};
  cuuint32_t box[2] = {box_cols, box_rows}, estr[2] = {1, 1};
  const CUresult r = enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(ptr), gdim, gstr, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                         CU_TENSOR_MAP_SWIZZLE_NONE, CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? RC_OK : RC_TMAP;
}

template <bool CHANNEL, int KS, bool EXACT, int M, int SPLIT>
static int launch_sequence(const DeltaRule& p, cudaStream_t st) {
  constexpr int COLS = 8 * DC_WARPS / SPLIT;
  const DeltaStage lay = delta_stage<CHANNEL, M, COLS>(p.dp);
  const int limit = 212 * 1024;                              // less the exchange and the barriers
  const dim3 grid((p.vp + COLS - 1) / COLS, p.H, p.n_long);
  // two stages leave room for more blocks on an SM, three hide more of a fetch
  const int stages = (long)grid.x * grid.y * grid.z <= sm_count() && 3 * lay.bytes <= limit ? 3 : 2;
  const int smem = stages * lay.bytes + 1024;
  if (smem > limit) return RC_TOO_LARGE;
  CUtensorMap tu, tv;
  const bf16* v = CHANNEL ? static_cast<const bf16*>(p.proj) + p.v_col : static_cast<const bf16*>(p.u) + 2 * p.G * p.dp;
  const uint64_t ldv = (uint64_t)(CHANNEL ? p.ldp : p.ldu) * 2;
  if (int rc = rows_tmap(&tv, v, p.T, p.H * p.vp, ldv, M * DC_TOK, COLS)) return rc;
  tu = tv;
  if (!CHANNEL)
    if (int rc = make_tmap_2d(&tu, p.u, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, p.T, 2 * p.G * p.dp, (uint64_t)p.ldu * 2, M * DC_TOK, 64)) return rc;
  static unsigned long long prep = 0;
  if (int e = ensure_dynamic_smem((const void*)delta_sequence_kernel<CHANNEL, KS, EXACT, M, SPLIT>, limit, prep)) return e;
  delta_sequence_kernel<CHANNEL, KS, EXACT, M, SPLIT><<<grid, 32 * (DC_WARPS + SPLIT - 1), smem, st>>>(tu, tv, p, stages);
  return (int)cudaGetLastError();
}

template <bool CHANNEL, int KS>
static int launch_exact(const DeltaRule& p, cudaStream_t st) {
  // few blocks: two warps to eight columns
  const long blocks = (long)((p.vp + 4 * DC_WARPS - 1) / (4 * DC_WARPS)) * p.H * p.n_long;
  return blocks <= (CHANNEL ? 1l : 2l) * sm_count() ? launch_sequence<CHANNEL, KS, true, 2, 2>(p, st) : launch_sequence<CHANNEL, KS, true, 2, 1>(p, st);
}

template <bool CHANNEL, int M>
static int launch_chunks(const DeltaRule& p, cudaStream_t st) {
  if constexpr (CHANNEL) delta_prepare_channel_kernel<M><<<dim3(p.n_chunks, p.H), 32 * M, 0, st>>>(p);
  else delta_prepare_gated_kernel<M><<<dim3(p.n_chunks, (p.H * M + 3) / 4), 128, 0, st>>>(p);
  if (int e = (int)cudaGetLastError()) return e;
  if constexpr (M == 1) {
    return launch_sequence<CHANNEL, 16, false, 1, 1>(p, st);
  } else {
    switch (p.dp) {
      case 64: return launch_exact<CHANNEL, 4>(p, st);
      case 96: return launch_exact<CHANNEL, 6>(p, st);
      case 128: return launch_exact<CHANNEL, 8>(p, st);
      default: break;
    }
    if (p.dp <= 128) return launch_sequence<CHANNEL, 8, false, 2, 1>(p, st);
    if constexpr (CHANNEL) return RC_TOO_LARGE;
    else return launch_sequence<CHANNEL, 16, false, 2, 1>(p, st);
  }
}

}  // namespace omni

using namespace omni;

// Portions of more than one row (`chunks` of 32 tokens, channel also 16; `long_list`); results before their norm go to `raw`.
extern "C" int omni_delta_chunks(const DeltaRule* args, int channel, int chunk, void* stream) {
  const DeltaRule& p = *args;
  if (p.n_chunks <= 0 || p.n_long <= 0) return RC_OK;
  if (!delta_args_ok(p, channel) || !p.chunks || !p.long_list || !p.raw || !p.mats || !p.coef || p.dp > 256 || p.n_long > 65535 ||
      (chunk != 32 && !(channel && chunk == 16 && p.dp > 128)) || (channel && chunk == 32 && p.dp > 128))
    return RC_BAD_ARG;
  if (channel ? !p.tiles : (!p.u || (p.ldu & 7) || p.ldu < 2l * p.G * p.dp + (long)p.H * p.vp)) return RC_BAD_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  if (!channel) return launch_chunks<false, 2>(p, st);
  return chunk == 16 ? launch_chunks<true, 1>(p, st) : launch_chunks<true, 2>(p, st);
}
