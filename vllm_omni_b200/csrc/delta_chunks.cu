// Delta-rule recurrences of prompt portions in chunks of 16 tokens on tensor cores (delta_rule.cuh says what is computed).
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
//   prepare   one warp per (chunk, head), all chunks at once: the 16 x 16 matrices and the inverse T of I + A, left in memory
//             as tensor-core operands; gated: the tokens' factors; channel: the decayed rows
//   sequence  one block per (portion, head, 32 value columns); a warp owns eight columns of the state, in registers from the
//             first chunk to the last, and walks the chunks without talking to the others; operands come through a
//             cp.async ring that the block shares
//
// Everything that is not a GEMM's or convolution's bf16 result keeps fp32 precision on the way through the tensor cores: such
// an operand is two bf16 numbers, high and low part, and a product of two of them three products (16 bits and more of
// each operand count).  Raw q, k, v are bf16 as they are.  A step of the sequence is a chain of small dependent products
// with the state as operand, so warp-level products (no staging through tensor memory) are the ones that fit.
#include "delta_rule.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

constexpr int DC_TOK = 16;
constexpr int DC_COLS = 32;            // value columns per block of the sequence kernel
constexpr int DC_WARPS = 4;

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

// rows of a chunk
struct ChunkRows {
  int seq, n;
  long row0;
};
__device__ __forceinline__ ChunkRows dc_chunk(const DeltaRule& p, int i) {
  const int4 c = *reinterpret_cast<const int4*>(p.chunks + 4 * i);
  ChunkRows r;
  r.seq = min(max(c.x, 0), p.num_seqs - 1);
  r.n = min(max(c.z, 1), DC_TOK);
  r.row0 = p.q_start[r.seq] + c.y;
  return r;
}

// ------------------------------------------------------------------------------ prepare: gated
__global__ void __launch_bounds__(128)
delta_prepare_gated_kernel(const DeltaRule p) {
  __shared__ float s_a[4][DC_TOK][20], s_tok[4][4][DC_TOK];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, j = lane & 3;
  const int h = blockIdx.y * 4 + warp;
  if (h >= p.H) return;
  const ChunkRows ch = dc_chunk(p, blockIdx.x);
  float* s_G = s_tok[warp][0];         // cumulative log decay
  float* s_b = s_tok[warp][1];
  float* s_ik = s_tok[warp][2];
  const bf16* proj = static_cast<const bf16*>(p.proj);
  const int hk = h / (p.H / p.G);
  // q and k of rows g and g + 8: 8 channels per lane and turn, the same order in both operands
  const bf16* u = static_cast<const bf16*>(p.u);
  const long ra = (ch.row0 + min(g, ch.n - 1)) * p.ldu + hk * p.dp, rb = (ch.row0 + min(g + 8, ch.n - 1)) * p.ldu + hk * p.dp;
  const int ko = p.G * p.dp;
  float kk0[4] = {}, kk1[4] = {}, qk0[4] = {}, qk1[4] = {};
  float ss[4] = {};                    // sums of squares: k rows g, g + 8, q rows g, g + 8
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
  for (int c = j * 8; c < p.dp + j * 8; c += 32) {
    const bool in = c < p.dp;
    const uint4 ka = in ? *reinterpret_cast<const uint4*>(u + ra + ko + c) : zero, kb = in ? *reinterpret_cast<const uint4*>(u + rb + ko + c) : zero;
    const uint4 qa = in ? *reinterpret_cast<const uint4*>(u + ra + c) : zero, qb = in ? *reinterpret_cast<const uint4*>(u + rb + c) : zero;
    const uint32_t kf[2][4] = {{ka.x, kb.x, ka.y, kb.y}, {ka.z, kb.z, ka.w, kb.w}};
    const uint32_t qf[2][4] = {{qa.x, qb.x, qa.y, qb.y}, {qa.z, qb.z, qa.w, qb.w}};
#pragma unroll
    for (int s = 0; s < 2; ++s) {
      dc_mma(kk0, kf[s], kf[s][0], kf[s][2]);
      dc_mma(kk1, kf[s], kf[s][1], kf[s][3]);
      dc_mma(qk0, qf[s], kf[s][0], kf[s][2]);
      dc_mma(qk1, qf[s], kf[s][1], kf[s][3]);
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
    s_ik[g] = ik[0];
    s_ik[g + 8] = ik[1];
  }
  // a lane per token: step size, cumulative log decay
  const int t = lane & 15;
  const bool live = t < ch.n;
  const bf16* pr = proj + (ch.row0 + min(t, ch.n - 1)) * p.ldp;
  const float beta = live ? dr_sigmoid((float)pr[p.b_col + h]) : 0.f;
  float G = live ? p.rate[h] * dr_softplus((float)pr[p.a_col + h] + p.dt_bias[h]) : 0.f;
#pragma unroll
  for (int o = 1; o < 16; o <<= 1) {
    const float v = __shfl_up_sync(0xffffffffu, G, o, 16);
    if (t >= o) G += v;
  }
  const float G_last = __shfl_sync(0xffffffffu, G, 15, 16);
  if (lane < 16) {
    s_G[t] = G;
    s_b[t] = beta;
  }
  __syncwarp();
  const long at = (long)blockIdx.x * p.H + h;
  uint4* mats = static_cast<uint4*>(p.mats) + at * 128;
  float* coef = p.coef + at * (4 * DC_TOK + 4);
  float p0[4], p1[4];
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int r = g + (e >> 1) * 8;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int s = half * 8 + j * 2 + (e & 1);
      const float d = r >= s ? expf(s_G[r] - s_G[s]) * s_ik[s] : 0.f;
      s_a[warp][r][s] = r > s ? s_b[r] * ik[e >> 1] * (half ? kk1[e] : kk0[e]) * d : 0.f;
      (half ? p1[e] : p0[e]) = iq[e >> 1] * (half ? qk1[e] : qk0[e]) * d;
    }
  }
  dc_store_mat(mats + 64, lane, p0, p1);
  if (j == 0) {
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = g + 8 * half;
      const float e = expf(s_G[r]);
      const float4 c = make_float4(s_b[r], -s_b[r] * e * ik[half], e * iq[half], r < ch.n ? expf(G_last - s_G[r]) * ik[half] : 0.f);
      *reinterpret_cast<float4*>(coef + 4 * r) = c;
    }
  }
  if (lane == 0) *reinterpret_cast<float4*>(coef + 4 * DC_TOK) = make_float4(expf(G_last), 0.f, 0.f, 0.f);
  __syncwarp();
  dc_invert(s_a[warp], lane);
  float c0[4], c1[4];
  dc_read_tiles(s_a[warp], lane, c0, c1);
  dc_store_mat(mats, lane, c0, c1);
}

// ---------------------------------------------------------------------------- prepare: channel
constexpr int PC_WARPS = 2, PC_PITCH = 64 * 2 + 16;          // bytes of a row of 64 channels
constexpr int PC_WARP_BYTES = 8 * DC_TOK * PC_PITCH;

__global__ void __launch_bounds__(32 * PC_WARPS)
delta_prepare_channel_kernel(const DeltaRule p) {
  __shared__ __align__(16) uint8_t s_rows[PC_WARPS][PC_WARP_BYTES];      // decayed rows: b0, r0, k / G, a u / G (high, low)
  __shared__ float s_a[PC_WARPS][DC_TOK][20];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, j = lane & 3;
  const int h = blockIdx.y * PC_WARPS + warp;
  if (h >= p.H) return;
  const ChunkRows ch = dc_chunk(p, blockIdx.x);
  const bf16* proj = static_cast<const bf16*>(p.proj) + (long)h * p.dp;
  const bf16* z = static_cast<const bf16*>(p.z) + (long)h * p.dp;
  const long at = (long)blockIdx.x * p.H + h;
  uint32_t* tiles = static_cast<uint32_t*>(p.tiles) + at * (8 * DC_TOK * (p.dp / 2));
  uint4* mats = static_cast<uint4*>(p.mats) + at * 256;
  const int tile = DC_TOK * (p.dp / 2);                      // channel pairs of an operand
  auto pair = [&](const bf16* base, long ld, int t, int c) {  // two channels of token t
    return unpack_bf16(*reinterpret_cast<const uint32_t*>(base + (ch.row0 + t) * ld + c));
  };
  // lengths of the keys
  float ik[DC_TOK];
#pragma unroll
  for (int t = 0; t < DC_TOK; ++t) {
    ik[t] = 0.f;
    if (t < ch.n)
      for (int c = lane * 2; c < p.dp; c += 64) {
        const float2 k = pair(proj + p.k_col, p.ldp, t, c);
        ik[t] = fmaf(k.x, k.x, fmaf(k.y, k.y, ik[t]));
      }
  }
#pragma unroll
  for (int t = 0; t < DC_TOK; ++t) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ik[t] += __shfl_xor_sync(0xffffffffu, ik[t], o);
    ik[t] = 1.0f / sqrtf(ik[t] + p.unit_eps);
  }
  float am[2][4] = {}, mm[2][4] = {}, nm[2][4] = {}, lm[2][4] = {};
  const uint32_t base = smem_u32(s_rows[warp]);
  uint32_t* rows = reinterpret_cast<uint32_t*>(s_rows[warp]);
  constexpr int ROW32 = PC_PITCH / 4, ARR32 = DC_TOK * ROW32;
  for (int cb = 0; cb < p.dp; cb += 64) {
    const int c = cb + lane * 2;
    const bool in = c < p.dp;
    const int cc = in ? c : 0;
    const float2 db = *reinterpret_cast<const float2*>(p.decay_bias + h * p.dp + cc);
    const float2 rb = *reinterpret_cast<const float2*>(p.removal_bias + h * p.dp + cc);
    float e0 = 1.f, e1 = 1.f, G0 = 0.f, G1 = 0.f;            // decays so far
    float kx[DC_TOK], ky[DC_TOK], ax[DC_TOK], ay[DC_TOK];    // k / G, a u / G
    __syncwarp();                                            // the products of the last 64 channels are done
#pragma unroll
    for (int t = 0; t < DC_TOK; ++t) {
      float2 b0 = make_float2(0.f, 0.f), r0 = b0;
      kx[t] = ky[t] = ax[t] = ay[t] = 0.f;
      if (t < ch.n && in) {
        const float2 r = pair(proj + p.q_col, p.ldp, t, c), k = pair(proj + p.k_col, p.ldp, t, c);
        const float2 a = pair(proj + p.a_col, p.ldp, t, c), zz = pair(z, p.ldz, t, c);
        b0 = make_float2(k.x * ik[t] * e0, k.y * ik[t] * e1);
        G0 = fmaf(p.decay_scale, __fdividef(1.0f, 1.0f + __expf(-(zz.x + db.x))), G0);
        G1 = fmaf(p.decay_scale, __fdividef(1.0f, 1.0f + __expf(-(zz.y + db.y))), G1);
        e0 = __expf(G0);
        e1 = __expf(G1);
        r0 = make_float2(r.x * e0, r.y * e1);
        const float i0 = __expf(-G0), i1 = __expf(-G1);
        kx[t] = k.x * i0;
        ky[t] = k.y * i1;
        ax[t] = __fdividef(ik[t], 1.0f + __expf(-(a.x + rb.x))) * kx[t];
        ay[t] = __fdividef(ik[t], 1.0f + __expf(-(a.y + rb.y))) * ky[t];
      }
      uint32_t hi, lo;
      uint32_t* dst = rows + t * ROW32 + lane;
      uint32_t* out = tiles + t * (p.dp / 2) + c / 2;
      dc_split(b0.x, b0.y, hi, lo);
      dst[0] = hi;
      dst[ARR32] = lo;
      if (in) { out[0] = hi; out[tile] = lo; }
      dc_split(r0.x, r0.y, hi, lo);
      dst[2 * ARR32] = hi;
      dst[3 * ARR32] = lo;
      if (in) { out[2 * tile] = hi; out[3 * tile] = lo; }
      dc_split(kx[t], ky[t], hi, lo);
      dst[4 * ARR32] = hi;
      dst[5 * ARR32] = lo;
      dc_split(ax[t], ay[t], hi, lo);
      dst[6 * ARR32] = hi;
      dst[7 * ARR32] = lo;
    }
    if (in) {
      *reinterpret_cast<float2*>(p.coef + at * p.dp + c) = make_float2(e0, e1);
#pragma unroll
      for (int t = 0; t < DC_TOK; ++t) {
        uint32_t hi, lo;
        uint32_t* out = tiles + 4 * tile + t * (p.dp / 2) + c / 2;
        dc_split(kx[t] * e0, ky[t] * e1, hi, lo);
        out[0] = hi;
        out[tile] = lo;
        dc_split(-ax[t] * e0, -ay[t] * e1, hi, lo);
        out[2 * tile] = hi;
        out[3 * tile] = lo;
      }
    }
    __syncwarp();
    const uint32_t a0 = base + ((lane & 7) + ((lane >> 3) & 1) * 8) * PC_PITCH + (lane >> 4) * 16;
    constexpr uint32_t ARR = DC_TOK * PC_PITCH;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      if (cb + k * 16 >= p.dp) break;
      uint32_t f[8][4];
#pragma unroll
      for (int x = 0; x < 8; ++x) dc_ldsm4(a0 + x * ARR + k * 32, f[x]);
      // rows x (0: b0, 2: r0) times columns y (4: k / G, 6: a u / G): high high, high low, low high
      auto product = [&](float (&c)[2][4], int x, int y) {
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          dc_mma(c[n], f[x], f[y][n], f[y][n + 2]);
          dc_mma(c[n], f[x], f[y + 1][n], f[y + 1][n + 2]);
          dc_mma(c[n], f[x + 1], f[y][n], f[y][n + 2]);
        }
      };
      product(am, 0, 6);
      product(mm, 0, 4);
      product(nm, 2, 4);
      product(lm, 2, 6);
    }
  }
#pragma unroll
  for (int n = 0; n < 2; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int r = g + (e >> 1) * 8, s = n * 8 + j * 2 + (e & 1);
      s_a[warp][r][s] = r > s ? am[n][e] : 0.f;
      if (r <= s) mm[n][e] = 0.f;
      if (r < s) nm[n][e] = 0.f;
      lm[n][e] = r < s ? 0.f : -lm[n][e];
    }
  dc_store_mat(mats + 64, lane, mm[0], mm[1]);
  dc_store_mat(mats + 128, lane, nm[0], nm[1]);
  dc_store_mat(mats + 192, lane, lm[0], lm[1]);
  __syncwarp();
  dc_invert(s_a[warp], lane);
  float c0[4], c1[4];
  dc_read_tiles(s_a[warp], lane, c0, c1);
  dc_store_mat(mats, lane, c0, c1);
}

// ----------------------------------------------------------------------------------- sequence
// Bytes of a stage: rows of the operands (gated: k, q; channel: eight), values, matrices, factors
struct DeltaStage {
  int pitch, arr, values, mats, coef, bytes;
};
__host__ __device__ __forceinline__ DeltaStage delta_stage(int dp, bool channel) {
  DeltaStage s;
  s.pitch = dp * 2 + 16;               // an odd multiple of 16 bytes: conflict-free ldmatrix
  s.arr = DC_TOK * s.pitch;
  s.values = (channel ? 8 : 2) * s.arr;
  s.mats = s.values + DC_TOK * (DC_COLS * 2 + 16);
  s.coef = s.mats + (channel ? 4096 : 2048);
  s.bytes = s.coef + (channel ? dp * 4 : (4 * DC_TOK + 4) * 4);
  return s;
}
constexpr int DC_VPITCH = DC_COLS * 2 + 16;

// KS: 16-channel steps of the key channels that the state's registers hold (dp <= 16 KS)
template <bool CHANNEL, int KS>
__global__ void __launch_bounds__(32 * DC_WARPS)
delta_sequence_kernel(const DeltaRule p, const int stages) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, j2 = (lane & 3) * 2;
  const int seq = min(max(p.long_list[2 * blockIdx.z], 0), p.num_seqs - 1), first = p.long_list[2 * blockIdx.z + 1];
  const int h = blockIdx.y, col0 = blockIdx.x * DC_COLS, hk = h / (p.H / p.G);
  const long row0 = p.q_start[seq];
  const int n = (int)(p.q_start[seq + 1] - row0);
  const int n_chunks = min((n + DC_TOK - 1) / DC_TOK, p.n_chunks - first);
  const DeltaStage lay = delta_stage(p.dp, CHANNEL);
  const uint32_t base = smem_u32(smem);
  const int vecs = p.dp / 8, v_vecs = min(DC_COLS, p.vp - col0) / 8;

  auto fetch = [&](int i) {
    const uint32_t st = base + (i % stages) * lay.bytes;
    const long at = (long)(first + i) * p.H + h;
    auto row = [&](int t) { return row0 + min(i * DC_TOK + t, n - 1); };       // past the end: finite, its factors are zero
    if (CHANNEL) {
      const uint4* src = static_cast<const uint4*>(p.tiles) + at * (8 * DC_TOK * vecs);
      for (int x = tid; x < 8 * DC_TOK * vecs; x += 32 * DC_WARPS) dc_copy16(st + (x / vecs) * lay.pitch + (x % vecs) * 16, src + x);
    } else {
      const bf16* u = static_cast<const bf16*>(p.u) + hk * p.dp;
      for (int x = tid; x < 2 * DC_TOK * vecs; x += 32 * DC_WARPS) {
        const int r = x / vecs, c = x - r * vecs;            // rows of k, then of q
        dc_copy16(st + r * lay.pitch + c * 16, u + row(r & 15) * p.ldu + (r < DC_TOK ? p.G * p.dp : 0) + c * 8);
      }
    }
    const bf16* v = CHANNEL ? static_cast<const bf16*>(p.proj) + p.v_col : static_cast<const bf16*>(p.u) + 2 * p.G * p.dp;
    const long ldv = CHANNEL ? p.ldp : p.ldu;
    for (int x = tid; x < DC_TOK * v_vecs; x += 32 * DC_WARPS) {
      const int r = x / v_vecs, c = x - r * v_vecs;
      dc_copy16(st + lay.values + r * DC_VPITCH + c * 16, v + row(r) * ldv + (long)h * p.vp + col0 + c * 8);
    }
    const int nm = CHANNEL ? 256 : 128;
    for (int x = tid; x < nm; x += 32 * DC_WARPS) dc_copy16(st + lay.mats + x * 16, static_cast<const uint4*>(p.mats) + at * nm + x);
    const int nf = CHANNEL ? p.dp / 4 : DC_TOK + 1;
    for (int x = tid; x < nf; x += 32 * DC_WARPS) dc_copy16(st + lay.coef + x * 16, reinterpret_cast<const float4*>(p.coef) + at * nf + x);
  };

  int sin, sout;
  delta_rows(p, seq, sin, sout);
  const int col = col0 + warp * 8;                           // this warp's columns
  const bool used = col < p.vp;
  float S[KS][4];                                            // rows g, g + 8 of 16 key channels, columns j2, j2 + 1
  {
    const float* src = p.state + ((long)sin * p.H + h) * p.dp * p.vp + col + j2;
    const bool have = used && p.context[seq] > 0;
#pragma unroll
    for (int k = 0; k < KS; ++k)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int r = k * 16 + g + 8 * e;
        const float2 v = have && k * 16 < p.dp ? *reinterpret_cast<const float2*>(src + (long)r * p.vp) : make_float2(0.f, 0.f);
        S[k][2 * e] = v.x;
        S[k][2 * e + 1] = v.y;
      }
  }
  for (int i = 0; i < stages - 1; ++i) {
    if (i < n_chunks) fetch(i);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  bf16* raw = static_cast<bf16*>(p.raw) + (long)h * p.vp + col + j2;
  const uint32_t a_off = ((lane & 7) + ((lane >> 3) & 1) * 8) * lay.pitch + (lane >> 4) * 16;      // tokens x channels
  const uint32_t t_off = ((lane & 7) + (lane >> 4) * 8) * lay.pitch + ((lane >> 3) & 1) * 16;      // channels x tokens
  for (int i = 0; i < n_chunks; ++i) {
    if (stages == 4) asm volatile("cp.async.wait_group 2;" ::: "memory");
    else if (stages == 3) asm volatile("cp.async.wait_group 1;" ::: "memory");
    else asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                         // chunk i is here, chunk i - 1 is done with
    if (i + stages - 1 < n_chunks) fetch(i + stages - 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (!used) continue;
    const int so = (i % stages) * lay.bytes;
    const uint32_t st = base + so;
    const uint4* mats = reinterpret_cast<const uint4*>(smem + so + lay.mats) + lane;
    auto mat = [&](int m, uint32_t (&a)[4]) {
      const uint4 v = mats[32 * m];
      a[0] = v.x; a[1] = v.y; a[2] = v.z; a[3] = v.w;
    };
    // what the state gives for the chunk's keys (x) and queries (o)
    float x0[4] = {}, x1[4] = {}, o0[4] = {}, o1[4] = {};
    SplitB s[KS];
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      if (k * 16 >= p.dp) break;
      s[k].from(S[k]);
      uint32_t a[4];
      dc_ldsm4(st + a_off + k * 32, a);
      dc_mma(x0, a, s[k].h0, s[k].h1);
      dc_mma(x1, a, s[k].l0, s[k].l1);
      if (CHANNEL) {
        dc_ldsm4(st + lay.arr + a_off + k * 32, a);
        dc_mma(x1, a, s[k].h0, s[k].h1);
      }
    }
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      if (k * 16 >= p.dp) break;
      uint32_t a[4];
      dc_ldsm4(st + (CHANNEL ? 2 : 1) * lay.arr + a_off + k * 32, a);
      dc_mma(o0, a, s[k].h0, s[k].h1);
      dc_mma(o1, a, s[k].l0, s[k].l1);
      if (CHANNEL) {
        dc_ldsm4(st + 3 * lay.arr + a_off + k * 32, a);
        dc_mma(o1, a, s[k].h0, s[k].h1);
      }
    }
    float y[4] = {}, o[4];
    uint32_t mh[4], ml[4];
    // product of a 16 x 16 matrix with split rows
    auto times = [&](float (&c)[4], int m, const SplitB& b) {
      mat(m, mh);
      mat(m + 1, ml);
      dc_mma(c, mh, b.h0, b.h1);
      dc_mma(c, mh, b.l0, b.l1);
      dc_mma(c, ml, b.h0, b.h1);
    };
    SplitB b;
    if (CHANNEL) {
      uint32_t v0, v1;
      dc_ldsm2_t(st + lay.values + (lane & 15) * DC_VPITCH + warp * 16, v0, v1);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        x0[e] += x1[e];
        o[e] = o0[e] + o1[e];
      }
      mat(2, mh);
      mat(3, ml);
      dc_mma(x0, mh, v0, v1);
      dc_mma(x0, ml, v0, v1);
      b.from(x0);
      times(y, 0, b);
      b.from(y);
      mat(4, mh);
      mat(5, ml);
      dc_mma(o, mh, v0, v1);
      dc_mma(o, ml, v0, v1);
      times(o, 6, b);
      const float* decay = reinterpret_cast<const float*>(smem + so + lay.coef);
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        if (k * 16 >= p.dp) break;
        const float d0 = decay[k * 16 + g], d1 = decay[k * 16 + g + 8];
        S[k][0] *= d0;
        S[k][1] *= d0;
        S[k][2] *= d1;
        S[k][3] *= d1;
        uint32_t a[4];
        dc_ldsm4_t(st + 4 * lay.arr + t_off + k * 32, a);
        dc_mma(S[k], a, v0, v1);
        dc_ldsm4_t(st + 5 * lay.arr + t_off + k * 32, a);
        dc_mma(S[k], a, v0, v1);
        dc_ldsm4_t(st + 6 * lay.arr + t_off + k * 32, a);
        dc_mma(S[k], a, b.h0, b.h1);
        dc_mma(S[k], a, b.l0, b.l1);
        dc_ldsm4_t(st + 7 * lay.arr + t_off + k * 32, a);
        dc_mma(S[k], a, b.h0, b.h1);
      }
    } else {
      const float* coef = reinterpret_cast<const float*>(smem + so + lay.coef);
      const float4 ca = *reinterpret_cast<const float4*>(coef + 4 * g), cb = *reinterpret_cast<const float4*>(coef + 4 * (g + 8));
      const uint8_t* vp = smem + so + lay.values + g * DC_VPITCH + (warp * 8 + j2) * 2;
      const float2 va = unpack_bf16(*reinterpret_cast<const uint32_t*>(vp)), vb = unpack_bf16(*reinterpret_cast<const uint32_t*>(vp + 8 * DC_VPITCH));
      x0[0] = fmaf(ca.y, x0[0] + x1[0], ca.x * va.x);
      x0[1] = fmaf(ca.y, x0[1] + x1[1], ca.x * va.y);
      x0[2] = fmaf(cb.y, x0[2] + x1[2], cb.x * vb.x);
      x0[3] = fmaf(cb.y, x0[3] + x1[3], cb.x * vb.y);
      b.from(x0);
      times(y, 0, b);
      b.from(y);
      o[0] = ca.z * (o0[0] + o1[0]);
      o[1] = ca.z * (o0[1] + o1[1]);
      o[2] = cb.z * (o0[2] + o1[2]);
      o[3] = cb.z * (o0[3] + o1[3]);
      times(o, 2, b);
      y[0] *= ca.w;
      y[1] *= ca.w;
      y[2] *= cb.w;
      y[3] *= cb.w;
      b.from(y);
      const float decay = coef[4 * DC_TOK];
#pragma unroll
      for (int k = 0; k < KS; ++k) {
        if (k * 16 >= p.dp) break;
#pragma unroll
        for (int e = 0; e < 4; ++e) S[k][e] *= decay;
        uint32_t a[4];
        dc_ldsm4_t(st + t_off + k * 32, a);
        dc_mma(S[k], a, b.h0, b.h1);
        dc_mma(S[k], a, b.l0, b.l1);
      }
    }
    const int t = i * DC_TOK + g;
    if (t < n) *reinterpret_cast<uint32_t*>(raw + (row0 + t) * p.H * p.vp) = pack_bf16(o[0], o[1]);
    if (t + 8 < n) *reinterpret_cast<uint32_t*>(raw + (row0 + t + 8) * p.H * p.vp) = pack_bf16(o[2], o[3]);
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  if (!used || sout < 0) return;
  float* dst = p.state + ((long)sout * p.H + h) * p.dp * p.vp + col + j2;
#pragma unroll
  for (int k = 0; k < KS; ++k)
#pragma unroll
    for (int e = 0; e < 2; ++e)
      if (k * 16 < p.dp) *reinterpret_cast<float2*>(dst + (long)(k * 16 + g + 8 * e) * p.vp) = make_float2(S[k][2 * e], S[k][2 * e + 1]);
}

template <bool CHANNEL, int KS>
static int launch_sequence(const DeltaRule& p, cudaStream_t st) {
  const DeltaStage lay = delta_stage(p.dp, CHANNEL);
  const int limit = 226 * 1024;
  int stages = 4;
  while (stages > 2 && stages * lay.bytes > (stages == 4 ? 64 : 226) * 1024) --stages;
  const int smem = stages * lay.bytes;
  if (smem > limit) return RC_TOO_LARGE;
  static unsigned long long prep = 0;
  if (int e = ensure_dynamic_smem((const void*)delta_sequence_kernel<CHANNEL, KS>, limit, prep)) return e;
  delta_sequence_kernel<CHANNEL, KS><<<dim3((p.vp + DC_COLS - 1) / DC_COLS, p.H, p.n_long), 32 * DC_WARPS, smem, st>>>(p, stages);
  return (int)cudaGetLastError();
}

template <bool CHANNEL>
static int launch_chunks(const DeltaRule& p, cudaStream_t st) {
  if (CHANNEL) delta_prepare_channel_kernel<<<dim3(p.n_chunks, (p.H + PC_WARPS - 1) / PC_WARPS), 32 * PC_WARPS, 0, st>>>(p);
  else delta_prepare_gated_kernel<<<dim3(p.n_chunks, (p.H + 3) / 4), 128, 0, st>>>(p);
  if (int e = (int)cudaGetLastError()) return e;
  if (p.dp <= 64) return launch_sequence<CHANNEL, 4>(p, st);
  if (p.dp <= 128) return launch_sequence<CHANNEL, 8>(p, st);
  return launch_sequence<CHANNEL, 16>(p, st);
}

}  // namespace omni

using namespace omni;

// Portions of more than one row (`chunks`, `long_list`); results before their norm go to `raw`.
extern "C" int omni_delta_chunks(const DeltaRule* args, int channel, void* stream) {
  const DeltaRule& p = *args;
  if (p.n_chunks <= 0 || p.n_long <= 0) return RC_OK;
  if (!delta_args_ok(p, channel) || !p.chunks || !p.long_list || !p.raw || !p.mats || !p.coef || p.dp > 256 || p.n_long > 65535)
    return RC_BAD_ARG;
  if (channel ? !p.tiles : (!p.u || (p.ldu & 7) || p.ldu < 2l * p.G * p.dp + (long)p.H * p.vp)) return RC_BAD_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  return channel ? launch_chunks<true>(p, st) : launch_chunks<false>(p, st);
}
