// Operands of the delta-rule recurrences (delta_rule.cu, delta_chunks.cu).  A head's state S [dp, vp] is fp32.
//
//   gated     q, k, v: causal convolution of the projection, silu; q, k over their length (sum of squares + unit_eps), q times
//             q_mul; ln g = rate softplus(a + dt_bias), b = sigmoid(b);  S <- g S, u = b (v - S^T k), S <- S + k u^T, o = S^T q
//   channel   u = k over its length, ln w = decay_scale sigmoid(z + decay_bias), a = sigmoid(a + removal_bias) per key channel;
//             S <- diag(w) S - (a u) (u^T S) + k v^T (both terms read the old S), o = S^T r
//
// Result: o / sqrt(<o^2> + eps) * gain * act(gate), act silu (gated) or sigmoid (channel).  Heads are padded to dp / vp
// channels, multiples of 16, with zeros.  State and history come from their pools where the position says that there are
// any; pool rows are double-buffered (read row != write row).
#pragma once
#include "host_util.h"
#include "row_ops.cuh"

namespace omni {

struct DeltaRule {
  const void* proj; long ldp;
  int T, H, G, dp, vp, d, dv, taps;             // d, dv: real channels
  int q_col, k_col, v_col, g_col, b_col, a_col;
  const float* conv;                            // gated: [taps, 2 G dp + H vp]
  const float* rate; const float* dt_bias;      // gated: [H]
  const void* z; long ldz;                      // channel: decay logits [T, H dp]
  const float* decay_bias; const float* removal_bias;       // channel: [H dp]
  float decay_scale, q_mul, eps, unit_eps;
  const float* gain; long gain_hs;              // [H, vp] at pitch gain_hs (0: shared by the heads)
  const int* row_seq; const int* q_start; const int* context;
  const int* state_in; const int* state_out;    // [S] rows of the pools; out < 0: not written
  void* hist; float* state;                     // [num_state, taps - 1, 2 G dp + H vp], [num_state, H, dp, vp]
  int num_state, num_seqs;
  const int* seq_list; int n_list;              // token by token: sequences to run, nullptr: all
  void* out; long ldo;                          // [T, H vp]
  void* raw;                                    // [T, H vp]: o before its norm
  // chunked kernels
  const int* chunks; int n_chunks;              // [n, 4] (sequence, first row of the portion, rows, -)
  const int* long_list; int n_long;             // [n, 2] (sequence, its first chunk)
  const void* u; long ldu;                      // gated: convolved rows q | k | v
  void* mats;                                   // per (chunk, head): 16 x 16 matrices as tensor-core operands, high and low parts
  float* coef;                                  // gated: per (chunk, head) 16 x 4 factors of the tokens, decay of the chunk;
                                                // channel: decay of the chunk per key channel
  void* tiles;                                  // channel: per (chunk, head) eight [16, dp] operands
  int* status;
};

__device__ __forceinline__ float dr_sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
// for results that are rounded to bf16 next
__device__ __forceinline__ float dr_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float dr_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float dr_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// pool rows of a sequence, checked; a bad index is reported and not used
__device__ __forceinline__ void delta_rows(const DeltaRule& p, int seq, int& sin, int& sout) {
  sin = p.state_in[seq];
  sout = p.state_out[seq];
  if (sin < 0 || sin >= p.num_state || sout >= p.num_state) {
    if (p.status) atomicCAS(p.status, 0, (int)ERR_BOUNDS);
    sin = 0;
    sout = -1;
  }
}

inline bool delta_args_ok(const DeltaRule& p, bool channel) {
  if (p.H <= 0 || p.G <= 0 || p.H % p.G || p.dp <= 0 || p.vp <= 0 || (p.dp & 15) || (p.vp & 15) || p.d > p.dp || p.dv > p.vp || p.d <= 0 ||
      p.dv <= 0 || p.taps < 1 || (p.ldp & 7) || (p.ldo & 7) || p.num_seqs <= 0 || p.num_state <= 0 || p.H > 65535)
    return false;
  if (!p.proj || !p.out || !p.state || !p.gain || !p.q_start || !p.context || !p.state_in || !p.state_out) return false;
  if ((reinterpret_cast<uintptr_t>(p.proj) & 15) || (reinterpret_cast<uintptr_t>(p.out) & 15)) return false;
  if (channel) return p.taps == 1 && p.G == p.H && p.dp == p.vp && p.z && (p.ldz & 7) == 0 && p.decay_bias && p.removal_bias;
  return p.conv && p.rate && p.dt_bias && (p.taps == 1 || p.hist);
}

}  // namespace omni
