// Short causal convolution over time of a mixed batch's bf16 rows, per channel, with an optional bias and silu:
// out_t = act(bias + sum_j conv[j] x_(t - taps + 1 + j)).  Rows before a portion come from the history pool where the
// position says that there are any, zeros otherwise; the portion's last rows become the sequence's new history.  Pool rows
// are double-buffered (read row != write row), so readers of the old history never race with the writer of the new one.
// A thread slides over eight rows of four channels; with up to four taps weights and earlier rows stay in registers.
#include "f32x2.cuh"
#include "host_util.h"
#include "row_ops.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

struct ConvRows {
  const void* x; long ldx;
  int T, C, taps;
  const float* conv;                            // [taps, C]
  const float* bias;                            // [C] or nullptr
  int act;                                      // 0 none, 1 silu
  int skip_single;                              // sequences with one row: their history is another kernel's
  const int* row_seq; const int* q_start; const int* context;
  const int* state_in; const int* state_out;    // [S] rows of the pool; out < 0: not written
  void* hist;                                   // [num_state, taps - 1, C]
  int num_state, num_seqs;
  void* out;                                    // [T, C]
  int* status;
};

__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// four channels of a row
__device__ __forceinline__ void unpack4(const uint2& q, uint64_t (&v)[2]) {
  const float2 a = unpack_bf16(q.x), b = unpack_bf16(q.y);
  v[0] = pack2(a.x, a.y);
  v[1] = pack2(b.x, b.y);
}

template <int TAPS>
__global__ void __launch_bounds__(128)
conv_rows_kernel(const ConvRows p) {
  constexpr int RUN = 8, H = TAPS > 1 ? TAPS - 1 : 1;
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4;
  const long r0 = (long)blockIdx.y * RUN;
  if (c >= p.C) return;
  const int taps = TAPS > 0 ? TAPS : p.taps, h = taps - 1;
  const bf16* x = static_cast<const bf16*>(p.x) + c;
  bf16* hist = static_cast<bf16*>(p.hist) + c;
  bf16* out = static_cast<bf16*>(p.out) + c;
  int seq = -1, q0 = 0, q1 = 0, ctx = 0, sin = 0, sout = -1;
  auto row_x = [&](long row) { return __ldg(reinterpret_cast<const uint2*>(x + row * p.ldx)); };
  auto past = [&](int b) {                                   // row b < 0 of the portion
    return ctx + b >= 0 ? *reinterpret_cast<const uint2*>(hist + ((long)sin * h + h + b) * p.C) : make_uint2(0u, 0u);
  };
  auto raw_x = [&](int b) { return b >= 0 ? row_x(q0 + b) : past(b); };
  auto enter = [&](int s) {                                  // a sequence's numbers
    seq = s;
    q0 = p.q_start[seq];
    q1 = p.q_start[seq + 1];
    ctx = p.context[seq];
    if (h > 0) {
      sin = p.state_in[seq];
      sout = p.state_out[seq];
      if (sin < 0 || sin >= p.num_state || sout >= p.num_state) {
        if (p.status) atomicCAS(p.status, 0, (int)ERR_BOUNDS);
        sin = 0;
        sout = -1;
      }
    }
  };
  auto seq_of = [&](long row) { return min(max(p.row_seq[row], 0), p.num_seqs - 1); };
  auto finish = [&](const uint64_t (&v)[2], long row) {
    float o[4];
    unpack2(v[0], o[0], o[1]);
    unpack2(v[1], o[2], o[3]);
    if (p.act == 1) {
#pragma unroll
      for (int e = 0; e < 4; ++e) o[e] *= rcp_approx(1.0f + ex2_approx(-1.4426950408889634f * o[e]));
    }
    *reinterpret_cast<uint2*>(out + row * p.C) = make_uint2(pack_bf16(o[0], o[1]), pack_bf16(o[2], o[3]));
  };
  auto new_history = [&](long row) {                         // after the portion's last row
    if (row == q1 - 1 && sout >= 0 && !(p.skip_single && q1 - q0 == 1))
      for (int m = 0; m < h; ++m)
        *reinterpret_cast<uint2*>(hist + ((long)sout * h + m) * p.C) = raw_x((int)(row - q0) + 1 - h + m);
  };
  uint64_t bias[2] = {0ull, 0ull};
  auto load_pairs = [&](const float* src, uint64_t (&v)[2]) {
    const float4 f = *reinterpret_cast<const float4*>(src);
    v[0] = pack2(f.x, f.y);
    v[1] = pack2(f.z, f.w);
  };
  if (p.bias) load_pairs(p.bias + c, bias);
  if constexpr (TAPS == 0) {
    for (long row = r0; row < min(r0 + RUN, (long)p.T); ++row) {
      const int s = seq_of(row);
      if (s != seq) enter(s);
      uint64_t o[2] = {bias[0], bias[1]};
      for (int j = 0; j < taps; ++j) {
        uint64_t f[2], w[2];
        unpack4(raw_x((int)(row - q0) - h + j), f);
        load_pairs(p.conv + (long)j * p.C + c, w);
        o[0] = fma2(w[0], f[0], o[0]);
        o[1] = fma2(w[1], f[1], o[1]);
      }
      finish(o, row);
      new_history(row);
    }
  } else {
    // all loads of the run in flight at once, the rows before it as if the portion began earlier
    uint2 raw[RUN], before[H];
#pragma unroll
    for (int i = 0; i < RUN; ++i) raw[i] = row_x(min(r0 + i, (long)p.T - 1));
#pragma unroll
    for (int m = 0; m < H; ++m) before[m] = row_x(max(r0 - H + m, 0l));
    uint64_t w[TAPS][2], win[TAPS][2];                       // win: rows t - taps + 1 .. t, row t at t % TAPS
#pragma unroll
    for (int j = 0; j < TAPS; ++j) load_pairs(p.conv + (long)j * p.C + c, w[j]);
    // portions are contiguous: rows that begin and end in the same one need no look at those between
    const int s_first = seq_of(r0);
    const bool same = s_first == seq_of(min(r0 + RUN, (long)p.T) - 1);
#pragma unroll
    for (int i = 0; i < RUN; ++i) {
      const long row = r0 + i;
      if (row >= p.T) break;
      const int s = i == 0 || same ? s_first : seq_of(row);
      if (s != seq) {                                        // first row of the run or of a sequence
        enter(s);
        if (TAPS > 1) {
#pragma unroll
          for (int m = 0; m < H; ++m) {
            const int b = (int)(row - q0) - H + m;
            unpack4(b < 0 ? past(b) : (i == 0 ? before[m] : row_x(row - H + m)), win[(i + m + 1) % TAPS]);
          }
        }
      }
      unpack4(raw[i], win[i % TAPS]);
      uint64_t o[2] = {bias[0], bias[1]};
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        o[0] = fma2(w[j][0], win[(i + j + 1) % TAPS][0], o[0]);
        o[1] = fma2(w[j][1], win[(i + j + 1) % TAPS][1], o[1]);
      }
      finish(o, row);
      new_history(row);
    }
  }
}

}  // namespace omni

using namespace omni;

extern "C" int omni_conv_rows(const ConvRows* args, void* stream) {
  const ConvRows& p = *args;
  if (p.T <= 0) return RC_OK;
  if (p.C <= 0 || (p.C & 7) || (p.ldx & 7) || p.ldx < p.C || p.taps < 1 || !p.conv || !p.x || !p.out || !p.row_seq || p.num_seqs <= 0 ||
      (reinterpret_cast<uintptr_t>(p.x) & 15) || (p.taps > 1 && (!p.hist || !p.state_in || !p.state_out || p.num_state <= 0)))
    return RC_BAD_ARG;
  const dim3 blocks((p.C / 4 + 127) / 128, (p.T + 7) / 8);
  if (blocks.y > 65535) return RC_TOO_LARGE;
  cudaStream_t st = (cudaStream_t)stream;
  switch (p.taps) {
    case 1: conv_rows_kernel<1><<<blocks, 128, 0, st>>>(p); break;
    case 2: conv_rows_kernel<2><<<blocks, 128, 0, st>>>(p); break;
    case 3: conv_rows_kernel<3><<<blocks, 128, 0, st>>>(p); break;
    case 4: conv_rows_kernel<4><<<blocks, 128, 0, st>>>(p); break;
    default: conv_rows_kernel<0><<<blocks, 128, 0, st>>>(p); break;
  }
  return (int)cudaGetLastError();
}
