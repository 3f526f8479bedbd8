// Operands and per-element math of the gated linear recurrence (gated_scan.cu, gated_scan_sm100.cu).
//
// Per channel: u_t = conv_b + sum_j conv[j] x_(t - taps + 1 + j); per part of `part` channels z^g_t = W^g u_t + b^g for
// the decay gate r = sigmoid(z^0) and the input gate i = sigmoid(z^1); ln a_t = decay r_t;
// S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t; out_t = S_t gelu(y_t).  proj holds y (columns [0, C)) and x ([C, 2 C)).
// x before the rows of a launch comes from the history pool, S from the state pool, where the position says that there
// is any; pool rows are double-buffered (read row != write row), so readers of a sequence's old state never race with
// the writer of its new one.
#pragma once
#include "host_util.h"
#include "row_ops.cuh"

namespace omni {

struct GatedScan {
  const void* proj; long ldp;
  int T, C, blocks, part, taps;
  const float* conv; const float* conv_b;       // [taps, C], [C]
  const void* gates; const float* gates_b;      // [2, blocks, part, part] ([out, in]), [2, C]
  const float* decay;                           // [C], <= 0
  const int* row_seq; const int* q_start; const int* context;
  const int* state_in; const int* state_out;    // [S] rows of the pools; out < 0: not written
  void* hist; float* state;                     // [num_state, taps - 1, C], [num_state, C]
  int num_state, num_seqs;
  const int* seq_list; int n_list;              // sequences with exactly one row
  const int* runs; int n_runs;                  // (sequence, first row of the portion, rows, first run of the sequence)
  float* sums;                                  // [n_runs, 2, C]: product of a, state from zero
  void* u; float* z;                            // [T, C] fp32 (plain kernels) or bf16; [2, T, C] (plain kernels)
  void* out;                                    // [T, C]
  int* status;
};

__device__ __forceinline__ float gs_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float gs_rcp(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float gs_sqrt(float x) {
  float y;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

constexpr float GS_LOG2E = 1.4426950408889634f, GS_LN2 = 0.6931471805599453f;

// One token of one channel for bf16 rows: la2 = log2 a, a, and the input term.  nbr, nbi: gate biases times -log2 e;
// decay2 = decay log2 e.
__device__ __forceinline__ void gate_step(float zr, float zi, float nbr, float nbi, float u, float decay2, float& la2, float& a,
                                          float& add) {
  // both sigmoids from one reciprocal; the clamp keeps the product of the denominators finite
  const float er = 1.0f + gs_ex2(fminf(fmaf(zr, -GS_LOG2E, nbr), 60.f)), ei = 1.0f + gs_ex2(fminf(fmaf(zi, -GS_LOG2E, nbi), 60.f));
  const float k = gs_rcp(er * ei);
  la2 = decay2 * (k * ei);
  a = gs_ex2(la2);
  // 1 - e^x for x = 2 ln a <= 0: the series near zero, where 1 - a^2 would cancel
  const float x = 2.0f * GS_LN2 * la2;
  const float series = -x * fmaf(0.5f * x, fmaf(x, 1.f / 3.f, 1.f), 1.f);
  const float d = x > -0.03f ? series : fmaf(-a, a, 1.0f);
  add = gs_sqrt(d) * (k * er) * u;
}

// gelu with the tanh form, as z * sigmoid(2 sqrt(2 / pi) (z + 0.044715 z^3))
__device__ __forceinline__ float gelu_short(float z) {
  constexpr float A = -1.5957691216057308f * GS_LOG2E, B = A * 0.044715f;
  return z * gs_rcp(1.0f + gs_ex2(fminf(z * fmaf(B, z * z, A), 126.f)));
}

// pool rows of a sequence, checked; a bad index is reported and not used
__device__ __forceinline__ void scan_rows(const GatedScan& p, int seq, int& sin, int& sout) {
  sin = p.state_in[seq];
  sout = p.state_out[seq];
  if (sin < 0 || sin >= p.num_state || sout >= p.num_state) {
    if (p.status) atomicCAS(p.status, 0, (int)ERR_BOUNDS);
    sin = 0;
    sout = -1;
  }
}

inline bool scan_args_ok(const GatedScan& p) {
  return p.C > 0 && p.blocks > 0 && p.part > 0 && p.part * p.blocks == p.C && (p.part & 15) == 0 && p.taps >= 1 && (p.ldp & 7) == 0 &&
         p.ldp >= 2l * p.C && p.num_seqs > 0 && p.num_state > 0 && p.state && p.state_in && p.state_out && (p.taps == 1 || p.hist);
}

}  // namespace omni
