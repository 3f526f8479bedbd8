// Row-wise steps of decoder-only language models whose residual stream is kept in fp32, for bf16
// activations (serving) and fp32 activations (exact mode):
//
//   omni_embed_norm     x = embed[id] (+ position table), xn = rms(x) * g            (one launch)
//   omni_add_norm       x += rms(y) * g_y, xn = rms(x) * g_n                          (one launch)
//   omni_poly_norm      a N(z) + b N(z^2) + c N(z^3) + e, N = division by the row's rms
//   omni_conv_heads     short causal convolution over time of the packed q/k/v projection, per-head
//                       RMS norm of q and k, growth of q with the position, mixing of v with an earlier
//                       layer's values, K/V rows written to their pages, convolution history written to
//                       the state pool
//   omni_rotary_heads   norm of whole query and key rows, rotation of the first channels of every head, norm of value heads,
//                       K/V rows written to their pages
//   omni_tanh_cols      tanh of some columns of a projection, packed
//   omni_logit_softcap  mult * logit, bounded to cap * tanh(. / cap) -> fp32
//
// Norm gains are fp32, either one number for the whole row (stride 0) or one per channel (stride 1).
// Rows are padded to a multiple of 8 channels; padding channels hold zeros and do not count in means.
#include "host_util.h"
#include "ptx_sm100.cuh"
#include "row_ops.cuh"

namespace omni {

// ------------------------------------------------------------------ embedding + first norm
template <typename T, int NV>
__global__ void __launch_bounds__(1024)
embed_norm_kernel(const long* __restrict__ ids, const long* __restrict__ pos, const T* __restrict__ embed, int vocab,
                  const T* __restrict__ pos_table, int max_pos, const T* __restrict__ overlay,
                  const unsigned char* __restrict__ overlay_mask, float* __restrict__ x, T* __restrict__ xn,
                  const float* __restrict__ g, int gs, int D, int Dp, int ld_embed, float eps) {
  __shared__ float sh[32];
  const long r = blockIdx.x;
  long id = ids[r];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  long p = pos_table ? pos[r] : 0;
  p = p < 0 ? 0 : (p >= max_pos ? max_pos - 1 : p);
  const bool over = overlay != nullptr && (overlay_mask == nullptr || overlay_mask[r]);
  const T* src = over ? overlay + r * ld_embed : embed + id * ld_embed;
  float v[NV][8];
  float ss[1] = {0.f};
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < Dp) {
      load8<T>(src + c, v[i]);
      if (pos_table) {
        float pe[8];
        load8<T>(pos_table + p * ld_embed + c, pe);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] += pe[e];
      }
      store8<float>(x + r * Dp + c, v[i]);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss[0] = fmaf(v[i][e], v[i][e], ss[0]);
    }
  }
  block_sum<1>(ss, sh);
  const float s = rms_scale(ss[0], D, eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < Dp) {
      scale_gain8(v[i], s, g, gs, c);
      store8<T>(xn + r * Dp + c, v[i]);
    }
  }
}

// ------------------------------------------------- residual add of a normed branch + next norm
// x += rms(y) * g_y; xn = rms(x) * g_n.  xn == nullptr: no second norm.
template <typename T, int NV>
__global__ void __launch_bounds__(1024)
add_norm_kernel(float* __restrict__ x, const T* __restrict__ y, int ldy, const float* __restrict__ gy, int gys,
                T* __restrict__ xn, const float* __restrict__ gn, int gns, int D, int Dp, float eps) {
  __shared__ float sh[32];
  const long r = blockIdx.x;
  float yv[NV][8], xv[NV][8];
  float ss[1] = {0.f};
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < Dp) {
      load8<T>(y + r * ldy + c, yv[i]);
      load8<float>(x + r * Dp + c, xv[i]);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss[0] = fmaf(yv[i][e], yv[i][e], ss[0]);
    }
  }
  block_sum<1>(ss, sh);
  const float sy = rms_scale(ss[0], D, eps);
  ss[0] = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < Dp) {
      scale_gain8(yv[i], sy, gy, gys, c);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        xv[i][e] += yv[i][e];
        ss[0] = fmaf(xv[i][e], xv[i][e], ss[0]);
      }
      store8<float>(x + r * Dp + c, xv[i]);
    }
  }
  if (xn == nullptr) return;
  block_sum<1>(ss, sh);
  const float sn = rms_scale(ss[0], D, eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < Dp) {
      scale_gain8(xv[i], sn, gn, gns, c);
      store8<T>(xn + r * Dp + c, xv[i]);
    }
  }
}

// --------------------------------------------------------------------------------- PolyNorm
// The row stays in registers as it was loaded (bf16 rows: half the registers of fp32 ones), so that blocks are small
// and several rows are in flight per SM.
template <typename T> struct Raw8;
template <> struct Raw8<__nv_bfloat16> { uint4 a; };
template <> struct Raw8<float> { uint4 a, b; };
template <typename T> __device__ __forceinline__ void unraw8(const Raw8<T>& r, float (&v)[8]) {
  load8<T>(reinterpret_cast<const T*>(&r), v);
}

template <typename T, int NV>
__global__ void __launch_bounds__(NV == 8 ? 1024 : 320)
poly_norm_kernel(const T* __restrict__ z, int ldz, T* __restrict__ out, int ldo, const float* __restrict__ coef, int F,
                 int Fp, float eps) {
  __shared__ float sh[96];
  const long r = blockIdx.x;
  Raw8<T> raw[NV];
  float ss[3] = {0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < Fp) raw[i] = *reinterpret_cast<const Raw8<T>*>(z + r * ldz + c);
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < Fp) {
      float v[8];
      unraw8<T>(raw[i], v);
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const float q = v[e] * v[e];
        ss[0] += q;
        ss[1] = fmaf(q, q, ss[1]);
        ss[2] = fmaf(q * q, q, ss[2]);
      }
    }
  }
  block_sum<3>(ss, sh);
  const float k1 = coef[0] * rms_scale(ss[0], F, eps), k2 = coef[1] * rms_scale(ss[1], F, eps);
  const float k3 = coef[2] * rms_scale(ss[2], F, eps), k0 = coef[3];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < Fp) {
      float v[8];
      unraw8<T>(raw[i], v);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = fmaf(v[e], fmaf(v[e], fmaf(v[e], k3, k2), k1), k0);
      store8<T>(out + r * ldo + c, v);
    }
  }
}

// ------------------------------------------ short convolution, head norms, value mixing, pages
// The packed projection has columns [q: H * dp | k: G * dp | v: GV * vp | ...], heads padded to dp / vp
// channels (multiples of 8).  A group of `lph` lanes owns one (row, head); a lane holds 8 channels.
// The history of a sequence (its last K-1 projected rows) comes from the state pool when it lies before
// the rows of this launch; pool rows are double-buffered (read index != write index), so the groups that
// read a sequence's old history never race with the one that writes its new one.
struct ConvHeads {
  const void* proj; long ldp;
  int T, H, G, dp, vp, d, taps;
  const float* conv;        // [taps, H * dp + G * dp + GV * vp] or nullptr
  const float* q_norm;      // [dp] or nullptr (no norm)
  const float* k_norm;
  float eps;
  const int* row_seq;       // [T] sequence of each row
  const int* q_start;       // [S + 1] first row of each sequence
  const int* context;       // [S] tokens of the sequence before its first row
  const int* slots;         // [T] page slot of each row, < 0: not written
  void* state;              // [pool rows, taps - 1, channels]
  const int* state_in;      // [S]
  const int* state_out;     // [S], < 0: not written
  void* q_out;              // [T, H * dp]
  void* k_cache; void* v_cache;     // [slots, G, dp], [slots, GV, vp]
  void* v_first;            // [T, GV * vp]
  int v_mode;               // 0: as they are, 1: also saved to v_first, 2: mixed with v_first
  const float* lambda;
  long num_slots;           // page slots of the caches / rows of the pool (bounds of the index operands)
  int num_state, num_seqs;
  int* status;
  int lph;                  // lanes per head: a power of two, 32 at most
  int GV;                   // value heads
  float q_coef;             // q grows by 1 + q_coef ln(floor((position + 1) / q_every) + 1); 0: not at all
  float q_every;
};

__device__ __forceinline__ float query_growth(const ConvHeads& p, int pos) {
  const float x = (float)(pos + 1);
  float n = floorf(__fdividef(x, p.q_every));             // off by one at most: put right by the products
  if (n * p.q_every > x) n -= 1.0f;
  else if ((n + 1.0f) * p.q_every <= x) n += 1.0f;
  return fmaf(p.q_coef, logf(n + 1.0f), 1.0f);
}

template <typename T, int IT>
__global__ void __launch_bounds__(256)
conv_heads_kernel(ConvHeads p) {
  const int lane = threadIdx.x & (p.lph - 1);
  const int t = blockIdx.x * (blockDim.x / p.lph) + threadIdx.x / p.lph;
  const int head = blockIdx.y;
  const bool live = t < p.T;
  const int row = live ? t : p.T - 1;                     // idle groups keep the shuffles company
  const int kind = head < p.H ? 0 : (head < p.H + p.G ? 1 : 2);
  const int width = kind == 2 ? p.vp : p.dp;
  const int hk = kind == 0 ? head : (kind == 1 ? head - p.H : head - p.H - p.G);
  const int C = (p.H + p.G) * p.dp + p.GV * p.vp;
  const int col0 = kind == 0 ? hk * p.dp : (kind == 1 ? (p.H + hk) * p.dp : (p.H + p.G) * p.dp + hk * p.vp);
  const T* proj = static_cast<const T*>(p.proj);
  T* state = static_cast<T*>(p.state);
  int seq = p.row_seq[row];
  seq = min(max(seq, 0), p.num_seqs - 1);
  const int q0 = p.q_start[seq], ctx = p.context[seq];
  const int off = row - q0;                               // row within the sequence's portion
  const int hist = p.taps - 1;
  int sin = 0, sout = -1;
  if (hist > 0) {
    sin = p.state_in[seq];
    sout = p.state_out[seq];
    if (sin < 0 || sin >= p.num_state || sout >= p.num_state) {
      if (p.status) atomicCAS(p.status, 0, (int)ERR_BOUNDS);
      sin = 0;
      sout = -1;
    }
  }
  float v[IT][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int c = (i * p.lph + lane) * 8;
#pragma unroll
    for (int e = 0; e < 8; ++e) v[i][e] = 0.f;
    if (c < width) {
      const int col = col0 + c;
      if (p.conv == nullptr) {
        load8<T>(proj + (long)row * p.ldp + col, v[i]);
      } else {
        for (int j = 0; j < p.taps; ++j) {
          const int b = off - hist + j;                   // row of the portion; negative: history
          float u[8], w[8];
          if (b >= 0) load8<T>(proj + (long)(q0 + b) * p.ldp + col, u);
          else if (ctx + b >= 0) load8<T>(state + ((long)sin * hist + hist + b) * C + col, u);
          else continue;
          load8<float>(p.conv + (long)j * C + col, w);
#pragma unroll
          for (int e = 0; e < 8; ++e) v[i][e] = fmaf(w[e], u[e], v[i][e]);
        }
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(v[i][e], v[i][e], ss);
    }
  }
  // new history: the group of the portion's last row writes all of it
  if (live && hist > 0 && sout >= 0 && row == p.q_start[seq + 1] - 1) {
    const int n = off + 1;
    for (int m = 0; m < hist; ++m) {
      const int b = n - hist + m;
#pragma unroll
      for (int i = 0; i < IT; ++i) {
        const int c = (i * p.lph + lane) * 8;
        if (c < width) {
          float u[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
          if (b >= 0) load8<T>(proj + (long)(q0 + b) * p.ldp + col0 + c, u);
          else if (ctx + b >= 0) load8<T>(state + ((long)sin * hist + hist + b) * C + col0 + c, u);
          store8<T>(state + ((long)sout * hist + m) * C + col0 + c, u);
        }
      }
    }
  }
  const float* nw = kind == 0 ? p.q_norm : (kind == 1 ? p.k_norm : nullptr);
  if (nw != nullptr) {                                    // uniform over the block (one head per block row)
    for (int o = p.lph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float s = rms_scale(ss, p.d, p.eps);
#pragma unroll
    for (int i = 0; i < IT; ++i) {
      const int c = (i * p.lph + lane) * 8;
      if (c < width) scale_gain8(v[i], s, nw, 1, c);
    }
  }
  if (!live) return;
  if (kind == 0 && p.q_coef != 0.f) {
    const float grow = query_growth(p, ctx + off);
#pragma unroll
    for (int i = 0; i < IT; ++i)
#pragma unroll
      for (int e = 0; e < 8; ++e) v[i][e] *= grow;
  }
  int slot = kind == 0 ? 0 : p.slots[row];
  if (slot >= p.num_slots && kind != 0) {
    if (p.status) atomicCAS(p.status, 0, (int)ERR_BOUNDS);
    slot = -1;
  }
  const float lam = p.v_mode == 2 ? p.lambda[0] : 0.f;
#pragma unroll
  for (int i = 0; i < IT; ++i) {
    const int c = (i * p.lph + lane) * 8;
    if (c >= width) continue;
    if (kind == 0) {
      store8<T>(static_cast<T*>(p.q_out) + (long)row * p.H * p.dp + col0 + c, v[i]);
    } else if (kind == 1) {
      if (slot >= 0) store8<T>(static_cast<T*>(p.k_cache) + ((long)slot * p.G + hk) * p.dp + c, v[i]);
    } else {
      T* vf = static_cast<T*>(p.v_first) + (long)row * p.GV * p.vp + hk * p.vp + c;
      if (p.v_mode == 1) store8<T>(vf, v[i]);
      if (p.v_mode == 2) {
        float f[8];
        load8<T>(vf, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[i][e] = (1.f - lam) * v[i][e] + lam * f[e];
      }
      if (slot >= 0) store8<T>(static_cast<T*>(p.v_cache) + ((long)slot * p.GV + hk) * p.vp + c, v[i]);
    }
  }
}

// The same for long batches: a group owns RUN consecutive rows of one head, holds the taps of its eight channels
// in registers and slides a window of projected rows along, so every projected value is loaded once (plus
// TAPS - 1 per run) and the weights once per run.
template <int TAPS, int RUN>
__global__ void __launch_bounds__(256)
conv_heads_run_kernel(ConvHeads p) {
  typedef __nv_bfloat16 T;
  constexpr int HIST = TAPS - 1;
  const int lane = threadIdx.x & (p.lph - 1);
  const int t0 = (blockIdx.x * (blockDim.x / p.lph) + threadIdx.x / p.lph) * RUN;
  const int head = blockIdx.y;
  const int kind = head < p.H ? 0 : (head < p.H + p.G ? 1 : 2);
  const int width = kind == 2 ? p.vp : p.dp;
  const int hk = kind == 0 ? head : (kind == 1 ? head - p.H : head - p.H - p.G);
  const int C = (p.H + p.G) * p.dp + p.GV * p.vp;
  const int c = lane * 8;
  const int col = (kind == 0 ? hk * p.dp : (kind == 1 ? (p.H + hk) * p.dp : (p.H + p.G) * p.dp + hk * p.vp)) + c;
  const bool in = c < width;
  const T* proj = static_cast<const T*>(p.proj) + col;
  T* state = static_cast<T*>(p.state) + col;
  uint4 raw[RUN];                                          // all loads of the run in flight at once
#pragma unroll
  for (int i = 0; i < RUN; ++i) {
    raw[i] = make_uint4(0u, 0u, 0u, 0u);
    if (in && t0 + i < p.T) raw[i] = *reinterpret_cast<const uint4*>(proj + (long)(t0 + i) * p.ldp);
  }
  float w[TAPS][8];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
#pragma unroll
    for (int e = 0; e < 8; ++e) w[j][e] = 0.f;
    if (in) load8<float>(p.conv + (long)j * C + col, w[j]);
  }
  const float* nw = kind == 0 ? p.q_norm : (kind == 1 ? p.k_norm : nullptr);
  const float lam = p.v_mode == 2 ? p.lambda[0] : 0.f;
  uint4 win[HIST > 0 ? HIST : 1];                          // the rows before the current one
  int prev_seq = -1, q0 = 0, ctx = 0, q1 = 0, sin = 0, sout = -1;
#pragma unroll
  for (int i = 0; i < RUN; ++i) {
    const int row = t0 + i;
    const bool live = row < p.T;
    const int seq = live ? min(max(p.row_seq[row], 0), p.num_seqs - 1) : prev_seq;
    if (live && seq != prev_seq) {                         // first row of the run or of a sequence: fetch its history
      prev_seq = seq;
      q0 = p.q_start[seq];
      q1 = p.q_start[seq + 1];
      ctx = p.context[seq];
      if (HIST > 0) {
        sin = p.state_in[seq];
        sout = p.state_out[seq];
        if (sin < 0 || sin >= p.num_state || sout >= p.num_state) {
          if (p.status) atomicCAS(p.status, 0, (int)ERR_BOUNDS);
          sin = 0;
          sout = -1;
        }
#pragma unroll
        for (int m = 0; m < HIST; ++m) {
          const int b = row - q0 - HIST + m;               // row of the portion; negative: history
          win[m] = make_uint4(0u, 0u, 0u, 0u);
          if (in && b >= 0) win[m] = *reinterpret_cast<const uint4*>(proj + (long)(q0 + b) * p.ldp);
          else if (in && ctx + b >= 0) win[m] = *reinterpret_cast<const uint4*>(state + ((long)sin * HIST + HIST + b) * C);
        }
      }
    }
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      float u[8];
      load8<T>(reinterpret_cast<const T*>(j < HIST ? &win[j] : &raw[i]), u);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = fmaf(w[j][e], u[e], v[e]);
    }
    if (HIST > 0) {
#pragma unroll
      for (int m = 0; m + 1 < HIST; ++m) win[m] = win[m + 1];
      win[HIST > 0 ? HIST - 1 : 0] = raw[i];
      // after its last row the window is the sequence's new history
      if (live && in && sout >= 0 && row == q1 - 1) {
#pragma unroll
        for (int m = 0; m < HIST; ++m) *reinterpret_cast<uint4*>(state + ((long)sout * HIST + m) * C) = win[m];
      }
    }
    if (nw != nullptr) {                                   // uniform over the block
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
      for (int o = p.lph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (in) scale_gain8(v, rms_scale(ss, p.d, p.eps), nw, 1, c);
    }
    if (!live || !in) continue;
    if (kind == 0) {
      if (p.q_coef != 0.f) {
        const float grow = query_growth(p, ctx + row - q0);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] *= grow;
      }
      store8<T>(static_cast<T*>(p.q_out) + (long)row * p.H * p.dp + col, v);
      continue;
    }
    int slot = p.slots[row];
    if (slot >= p.num_slots) {
      if (p.status) atomicCAS(p.status, 0, (int)ERR_BOUNDS);
      slot = -1;
    }
    if (kind == 1) {
      if (slot >= 0) store8<T>(static_cast<T*>(p.k_cache) + ((long)slot * p.G + hk) * p.dp + c, v);
    } else {
      T* vf = static_cast<T*>(p.v_first) + (long)row * p.GV * p.vp + hk * p.vp + c;
      if (p.v_mode == 1) store8<T>(vf, v);
      if (p.v_mode == 2) {
        float f[8];
        load8<T>(vf, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = (1.f - lam) * v[e] + lam * f[e];
      }
      if (slot >= 0) store8<T>(static_cast<T*>(p.v_cache) + ((long)slot * p.GV + hk) * p.vp + c, v);
    }
  }
}

// Without a convolution: a group owns RUN rows of one head, all loads of the run (rows, page slots, positions) in flight at
// once.
template <int RUN>
__global__ void __launch_bounds__(256)
heads_run_kernel(ConvHeads p) {
  typedef __nv_bfloat16 T;
  const int head = blockIdx.y;
  const int kind = head < p.H ? 0 : (head < p.H + p.G ? 1 : 2);
  const int width = kind == 2 ? p.vp : p.dp;
  const int lph = width <= 16 ? 2 : (width <= 32 ? 4 : (width <= 64 ? 8 : (width <= 128 ? 16 : 32)));
  const int lane = threadIdx.x & (lph - 1);
  const int groups = 256 / lph, t0 = blockIdx.x * groups * RUN + threadIdx.x / lph;   // rows t0 + i * groups
  if (blockIdx.x * groups * RUN >= p.T) return;             // the grid is made for the widest heads
  const int hk = kind == 0 ? head : (kind == 1 ? head - p.H : head - p.H - p.G);
  const int c = lane * 8;
  const int col = (kind == 0 ? hk * p.dp : (kind == 1 ? (p.H + hk) * p.dp : (p.H + p.G) * p.dp + hk * p.vp)) + c;
  const bool in = c < width;
  const T* proj = static_cast<const T*>(p.proj) + col;
  uint4 raw[RUN];
  int at[RUN];                                              // page slot of a row (k, v)
#pragma unroll
  for (int i = 0; i < RUN; ++i) {
    const int row = t0 + i * groups;
    raw[i] = make_uint4(0u, 0u, 0u, 0u);
    at[i] = -1;
    if (row >= p.T) continue;
    if (in) raw[i] = *reinterpret_cast<const uint4*>(proj + (long)row * p.ldp);
    if (kind != 0) at[i] = p.slots[row];
  }
  float grow[RUN];
#pragma unroll
  for (int i = 0; i < RUN; ++i) grow[i] = 1.f;
  if (kind == 0 && p.q_coef != 0.f) {                       // a lane computes one row's growth for all lanes of its group
    float mine[RUN];
#pragma unroll
    for (int i = 0; i < RUN; ++i) {
      const int row = t0 + (i * lph + lane) * groups;
      mine[i] = 1.f;
      if (i * lph >= RUN) break;
      if (i * lph + lane < RUN && row < p.T) {
        const int seq = min(max(p.row_seq[row], 0), p.num_seqs - 1);
        mine[i] = query_growth(p, max(p.context[seq] + row - p.q_start[seq], 0));
      }
    }
    const int first = threadIdx.x & 31 & ~(lph - 1);
#pragma unroll
    for (int i = 0; i < RUN; ++i) {
      float m = mine[0];
#pragma unroll
      for (int k = 1; k < RUN; ++k)
        if (i >= k * lph) m = mine[k];
      grow[i] = __shfl_sync(0xffffffffu, m, first + (i & (lph - 1)));
    }
  }
  const float* nw = kind == 0 ? p.q_norm : (kind == 1 ? p.k_norm : nullptr);
  float w[8];
  if (nw != nullptr && in) load8<float>(nw + c, w);
#pragma unroll
  for (int i = 0; i < RUN; ++i) {
    const int row = t0 + i * groups;
    float v[8];
    load8<T>(reinterpret_cast<const T*>(&raw[i]), v);
    if (nw != nullptr) {                                    // uniform over the block
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
      for (int o = lph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      const float s = rsqrtf(fmaf(ss, 1.0f / (float)p.d, p.eps)) * grow[i];
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] *= s * w[e];
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] *= grow[i];
    }
    if (row >= p.T || !in) continue;
    if (kind == 0) {
      store8<T>(static_cast<T*>(p.q_out) + (long)row * p.H * p.dp + col, v);
      continue;
    }
    if (at[i] >= p.num_slots) {
      if (p.status) atomicCAS(p.status, 0, (int)ERR_BOUNDS);
      continue;
    }
    if (at[i] < 0) continue;
    T* dst = kind == 1 ? static_cast<T*>(p.k_cache) + ((long)at[i] * p.G + hk) * p.dp : static_cast<T*>(p.v_cache) + ((long)at[i] * p.GV + hk) * p.vp;
    store8<T>(dst + c, v);
  }
}

// ------------------------------------------- row norms, rotation, value head norms, pages
// One block per row of the packed projection [q: H * dp | k: G * dp | v: G * vp | ...]; a thread holds NV vectors of eight
// channels.  Rotated pairs are neighbours, so a rotation stays within a vector.
struct RotaryHeads {
  const void* proj; long ldp;
  int T, H, G, dp, vp;
  int rot;                  // rotated channels of a q / k head, even
  const float* turns;       // [T, rot / 2, 2]: cos, sin
  const float* q_gain;      // [H * dp] or nullptr (no norm): norm over the whole row
  const float* k_gain;      // [G * dp] or nullptr
  int nq, nk, vdim;         // real channels of a query row, a key row, a value head
  int v_norm;               // every value head over its root mean square
  float v_mult, eps;
  const int* slots;         // [T] page slot of each row, < 0: not written
  void* q_out;              // [T, H * dp]
  void* k_cache; void* v_cache;     // [slots, G, dp], [slots, G, vp]
  long num_slots;
  int* status;
};

template <typename T, int NV>
__global__ void __launch_bounds__(256)
rotary_heads_kernel(const RotaryHeads p) {
  extern __shared__ float s_v[];                            // sums of squares of the value vectors
  __shared__ float sh[64];
  const long row = blockIdx.x;
  const int nq = p.H * p.dp, nk = p.G * p.dp, C = nq + nk + p.G * p.vp;
  const T* proj = static_cast<const T*>(p.proj) + row * p.ldp;
  Raw8<T> raw[NV];                                          // as loaded: half the registers for bf16
  int slot = p.slots[row];
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c < C) raw[i] = *reinterpret_cast<const Raw8<T>*>(proj + c);
  }
  float sq = 1.f, sk = 1.f;
  if (p.q_gain || p.k_gain || p.v_norm) {                   // uniform
    float ss[2] = {0.f, 0.f};                               // of the query row, of the key row
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = (i * blockDim.x + threadIdx.x) * 8;
      if (c >= C) continue;
      float v[8], s = 0.f;
      unraw8<T>(raw[i], v);
#pragma unroll
      for (int e = 0; e < 8; ++e) s = fmaf(v[e], v[e], s);
      if (c < nq) ss[0] += s;
      else if (c < nq + nk) ss[1] += s;
      else if (p.v_norm) s_v[(c - nq - nk) / 8] = s;
    }
    block_sum<2>(ss, sh);                                   // also: the value sums are in place
    sq = rms_scale(ss[0], p.nq, p.eps);
    sk = rms_scale(ss[1], p.nk, p.eps);
  }
  if (slot >= p.num_slots) {
    if (p.status) atomicCAS(p.status, 0, (int)ERR_BOUNDS);
    slot = -1;
  }
  const float* turns = p.turns + row * p.rot;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c >= C) continue;
    float v[8];
    unraw8<T>(raw[i], v);
    if (c >= nq + nk) {
      const int cv = c - nq - nk;
      float s = p.v_mult;
      if (p.v_norm) {
        const int per = p.vp / 8, first = cv / p.vp * per;
        float t = 0.f;
        for (int x = 0; x < per; ++x) t += s_v[first + x];
        s *= rms_scale(t, p.vdim, p.eps);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] *= s;
      if (slot >= 0) store8<T>(static_cast<T*>(p.v_cache) + (long)slot * p.G * p.vp + cv, v);
      continue;
    }
    const bool is_q = c < nq;
    const int ck = is_q ? c : c - nq;
    const float* gain = is_q ? p.q_gain : p.k_gain;
    if (gain) scale_gain8(v, is_q ? sq : sk, gain, 1, ck);
    const int in = ck % p.dp;
    if (in + 8 <= p.rot && (p.rot & 3) == 0) {              // rows of turns on 16 bytes
      float t[8];                                           // four pairs of cos and sin
      load8<float>(turns + in, t);
#pragma unroll
      for (int e = 0; e < 8; e += 2) {
        const float a = v[e], b = v[e + 1];
        v[e] = a * t[e] - b * t[e + 1];
        v[e + 1] = b * t[e] + a * t[e + 1];
      }
    } else {
#pragma unroll
      for (int e = 0; e < 8; e += 2) {
        if (in + e >= p.rot) break;
        const float a = v[e], b = v[e + 1], co = turns[in + e], si = turns[in + e + 1];
        v[e] = a * co - b * si;
        v[e + 1] = b * co + a * si;
      }
    }
    if (is_q) store8<T>(static_cast<T*>(p.q_out) + row * nq + ck, v);
    else if (slot >= 0) store8<T>(static_cast<T*>(p.k_cache) + (long)slot * nk + ck, v);
  }
}

// ------------------------------------------------------------------------------ tanh of columns
template <typename T>
__global__ void __launch_bounds__(256)
tanh_cols_kernel(const T* __restrict__ in, long ldi, T* __restrict__ out, long rows, int n) {
  const int vec = n / 8;
  for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < rows * vec; i += (long)gridDim.x * blockDim.x) {
    const long r = i / vec;
    const int c = (int)(i - r * vec) * 8;
    float v[8];
    load8<T>(in + r * ldi + c, v);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = tanhf(v[e]);
    store8<T>(out + r * n + c, v);
  }
}

// ------------------------------------------------------------------------------ logit cap
template <typename T>
__global__ void __launch_bounds__(256)
logit_softcap_kernel(const T* __restrict__ in, long ldi, float* __restrict__ out, long ldo, long rows, int V, float cap, float mult) {
  const long total = rows * V;
  for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x) {
    const long r = i / V;
    const int c = (int)(i - r * V);
    const float z = mult * (float)in[r * ldi + c];
    out[r * ldo + c] = cap > 0.f ? cap * tanhf(z / cap) : z;
  }
}

}  // namespace omni

using namespace omni;
typedef __nv_bfloat16 bf16;

#define OMNI_ROW_DISPATCH(KERNEL, ROWS, ...)                                                            \
  do {                                                                                                  \
    cudaStream_t st_ = (cudaStream_t)stream;                                                            \
    if (is_bf16) {                                                                                      \
      typedef bf16 T;                                                                                   \
      if (nv == 1) KERNEL<T, 1><<<(unsigned)(ROWS), threads, 0, st_>>>(__VA_ARGS__);                    \
      else if (nv == 2) KERNEL<T, 2><<<(unsigned)(ROWS), threads, 0, st_>>>(__VA_ARGS__);               \
      else KERNEL<T, 4><<<(unsigned)(ROWS), threads, 0, st_>>>(__VA_ARGS__);                            \
    } else {                                                                                            \
      typedef float T;                                                                                  \
      if (nv == 1) KERNEL<T, 1><<<(unsigned)(ROWS), threads, 0, st_>>>(__VA_ARGS__);                    \
      else if (nv == 2) KERNEL<T, 2><<<(unsigned)(ROWS), threads, 0, st_>>>(__VA_ARGS__);               \
      else KERNEL<T, 4><<<(unsigned)(ROWS), threads, 0, st_>>>(__VA_ARGS__);                            \
    }                                                                                                   \
  } while (0)

extern "C" int omni_embed_norm(const long* ids, const long* pos, const void* embed, int vocab, const void* pos_table,
                               int max_pos, const void* overlay, const void* overlay_mask, float* x, void* xn,
                               const float* g, int gs, int rows, int D, int Dp, int ld_embed, float eps, int is_bf16,
                               void* stream) {
  if (rows <= 0) return RC_OK;
  int threads, nv;
  if ((Dp & 7) || (ld_embed & 7) || D > Dp || vocab < 1 || !row_shape(Dp, threads, nv)) return RC_BAD_ARG;
  OMNI_ROW_DISPATCH(embed_norm_kernel, rows, ids, pos, (const T*)embed, vocab, (const T*)pos_table, max_pos,
                    (const T*)overlay, (const unsigned char*)overlay_mask, x, (T*)xn, g, gs, D, Dp, ld_embed, eps);
  return (int)cudaGetLastError();
}

extern "C" int omni_add_norm(float* x, const void* y, int ldy, const float* gy, int gys, void* xn, const float* gn,
                             int gns, int rows, int D, int Dp, float eps, int is_bf16, void* stream) {
  if (rows <= 0) return RC_OK;
  int threads, nv;
  if ((Dp & 7) || (ldy & 7) || D > Dp || !row_shape(Dp, threads, nv)) return RC_BAD_ARG;
  OMNI_ROW_DISPATCH(add_norm_kernel, rows, x, (const T*)y, ldy, gy, gys, (T*)xn, gn, gns, D, Dp, eps);
  return (int)cudaGetLastError();
}

extern "C" int omni_poly_norm(const void* z, int ldz, void* out, int ldo, const float* coef, int rows, int F, int Fp,
                              float eps, int is_bf16, void* stream) {
  if (rows <= 0) return RC_OK;
  int threads, nv;
  if (Fp <= 0 || (Fp & 7) || (ldz & 7) || (ldo & 7) || F > Fp || Fp > 65536) return RC_BAD_ARG;
  const int vec = Fp / 8;
  nv = vec <= 128 ? 1 : (vec <= 512 ? 2 : (vec <= 1280 ? 4 : 8));
  threads = ((vec + nv - 1) / nv + 31) / 32 * 32;
  cudaStream_t st = (cudaStream_t)stream;
#define OMNI_POLY(T, NV) poly_norm_kernel<T, NV><<<rows, threads, 0, st>>>((const T*)z, ldz, (T*)out, ldo, coef, F, Fp, eps)
#define OMNI_POLY_NV(T)           \
  do {                            \
    if (nv == 1) OMNI_POLY(T, 1); \
    else if (nv == 2) OMNI_POLY(T, 2); \
    else if (nv == 4) OMNI_POLY(T, 4); \
    else OMNI_POLY(T, 8);         \
  } while (0)
  if (is_bf16) OMNI_POLY_NV(bf16); else OMNI_POLY_NV(float);
#undef OMNI_POLY_NV
#undef OMNI_POLY
  return (int)cudaGetLastError();
}

extern "C" int omni_conv_heads(const ConvHeads* args, int is_bf16, void* stream) {
  ConvHeads p = *args;
  if (p.T <= 0) return RC_OK;
  if (p.num_seqs <= 0 || p.H <= 0 || p.G <= 0 || p.GV <= 0 || (p.q_coef != 0.f && !(p.q_every > 0)) || (p.dp & 7) || (p.vp & 7) || (p.ldp & 7) || p.d > p.dp || p.taps < 1)
    return RC_BAD_ARG;
  if ((p.conv == nullptr && p.taps != 1) || (p.taps > 1 && (p.state == nullptr || p.num_state <= 0))) return RC_BAD_ARG;
  if (p.v_mode != 0 && p.v_first == nullptr) return RC_BAD_ARG;
  const int lanes = (p.dp > p.vp ? p.dp : p.vp) / 8;
  if (lanes > 128) return RC_BAD_ARG;
  p.lph = 1;
  while (p.lph < lanes && p.lph < 32) p.lph *= 2;
  const int rows_per_cta = 256 / p.lph;
  dim3 grid((p.T + rows_per_cta - 1) / rows_per_cta, p.H + p.G + p.GV);
  cudaStream_t st = (cudaStream_t)stream;
  constexpr int RUN = 8;
  if (is_bf16 && lanes <= 32 && p.T >= 256 && p.taps <= 4 && p.conv != nullptr) {
    const int rows = rows_per_cta * RUN;
    dim3 rgrid((p.T + rows - 1) / rows, p.H + p.G + p.GV);
    switch (p.taps) {
      case 1: conv_heads_run_kernel<1, RUN><<<rgrid, 256, 0, st>>>(p); break;
      case 2: conv_heads_run_kernel<2, RUN><<<rgrid, 256, 0, st>>>(p); break;
      case 3: conv_heads_run_kernel<3, RUN><<<rgrid, 256, 0, st>>>(p); break;
      default: conv_heads_run_kernel<4, RUN><<<rgrid, 256, 0, st>>>(p); break;
    }
    return (int)cudaGetLastError();
  }
  if (is_bf16 && lanes <= 32 && p.T >= 256 && p.conv == nullptr && p.v_mode == 0) {
    const int rows = rows_per_cta * 4;
    heads_run_kernel<4><<<dim3((p.T + rows - 1) / rows, p.H + p.G + p.GV), 256, 0, st>>>(p);
    return (int)cudaGetLastError();
  }
  if (is_bf16) {
    if (lanes <= 32) conv_heads_kernel<bf16, 1><<<grid, 256, 0, st>>>(p);
    else conv_heads_kernel<bf16, 4><<<grid, 256, 0, st>>>(p);
  } else {
    if (lanes <= 32) conv_heads_kernel<float, 1><<<grid, 256, 0, st>>>(p);
    else conv_heads_kernel<float, 4><<<grid, 256, 0, st>>>(p);
  }
  return (int)cudaGetLastError();
}

extern "C" int omni_rotary_heads(const RotaryHeads* args, int is_bf16, void* stream) {
  const RotaryHeads& p = *args;
  if (p.T <= 0) return RC_OK;
  if (p.H <= 0 || p.G <= 0 || (p.dp & 7) || (p.vp & 7) || p.dp <= 0 || p.vp <= 0 || (p.ldp & 7) || (p.rot & 1) || p.rot < 0 ||
      p.rot > p.dp || (p.rot && !p.turns) || !p.slots || !p.q_out || !p.k_cache || !p.v_cache || p.nq <= 0 || p.nk <= 0 || p.vdim <= 0)
    return RC_BAD_ARG;
  const int C = (p.H + p.G) * p.dp + p.G * p.vp, vec = C / 8;
  if (C > p.ldp || vec > 256 * 16) return RC_BAD_ARG;
  const int nv = vec <= 256 ? 1 : (vec <= 512 ? 2 : (vec <= 1024 ? 4 : 16));
  const int threads = ((vec + nv - 1) / nv + 31) / 32 * 32;
  const int smem = p.v_norm ? p.G * p.vp / 8 * 4 : 0;
  if (smem > 47 * 1024) return RC_TOO_LARGE;
  cudaStream_t st = (cudaStream_t)stream;
#define OMNI_ROTARY(ELT)                                                              \
  do {                                                                                \
    if (nv == 1) rotary_heads_kernel<ELT, 1><<<p.T, threads, smem, st>>>(p);          \
    else if (nv == 2) rotary_heads_kernel<ELT, 2><<<p.T, threads, smem, st>>>(p);     \
    else if (nv == 4) rotary_heads_kernel<ELT, 4><<<p.T, threads, smem, st>>>(p);     \
    else rotary_heads_kernel<ELT, 16><<<p.T, threads, smem, st>>>(p);                 \
  } while (0)
  if (is_bf16) OMNI_ROTARY(bf16); else OMNI_ROTARY(float);
#undef OMNI_ROTARY
  return (int)cudaGetLastError();
}

extern "C" int omni_tanh_cols(const void* in, long ldi, void* out, long rows, int n, int is_bf16, void* stream) {
  if (rows <= 0 || n <= 0) return RC_OK;
  if ((n & 7) || (ldi & 7) || ldi < n || (reinterpret_cast<uintptr_t>(in) & 15)) return RC_BAD_ARG;
  long blocks = (rows * (n / 8) + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  cudaStream_t st = (cudaStream_t)stream;
  if (is_bf16) tanh_cols_kernel<bf16><<<(unsigned)blocks, 256, 0, st>>>((const bf16*)in, ldi, (bf16*)out, rows, n);
  else tanh_cols_kernel<float><<<(unsigned)blocks, 256, 0, st>>>((const float*)in, ldi, (float*)out, rows, n);
  return (int)cudaGetLastError();
}

extern "C" int omni_logit_softcap(const void* in, long ldi, float* out, long ldo, long rows, int V, float cap, float mult,
                                  int is_bf16, void* stream) {
  if (rows <= 0) return RC_OK;
  long blocks = (rows * V + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  cudaStream_t st = (cudaStream_t)stream;
  if (is_bf16) logit_softcap_kernel<bf16><<<(unsigned)blocks, 256, 0, st>>>((const bf16*)in, ldi, out, ldo, rows, V, cap, mult);
  else logit_softcap_kernel<float><<<(unsigned)blocks, 256, 0, st>>>((const float*)in, ldi, out, ldo, rows, V, cap, mult);
  return (int)cudaGetLastError();
}
