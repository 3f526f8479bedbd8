// Gated linear recurrence (gated_scan.cuh says what is computed).
//
//   omni_scan_step    sequences with one new token, bf16, everything in one launch: a block owns 16 tokens and 32
//                     channels of one part; convolution to shared memory, both gates on 16 x 8 x 16 tensor-core
//                     products (weights straight from global memory, each byte read once per 16 tokens), state
//                     update and output in the epilogue
//   omni_scan_conv    convolution to fp32 and the new history \ plain kernels, bf16 or fp32: the exact mode, and
//   omni_scan_plain   scan, one thread per channel            / sizes the other kernels do not take
#include "gated_scan.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

// x of a channel at row b of a sequence's portion (negative: history, zero before the start)
template <typename T>
__device__ __forceinline__ float scan_x(const GatedScan& p, int q0, int ctx, int sin, int b, int c) {
  if (b >= 0) return (float)static_cast<const T*>(p.proj)[(long)(q0 + b) * p.ldp + p.C + c];
  if (ctx + b < 0) return 0.f;
  return (float)static_cast<const T*>(p.hist)[((long)sin * (p.taps - 1) + p.taps - 1 + b) * p.C + c];
}

// new history of a channel after the portion's last row (row `last`)
template <typename T>
__device__ __forceinline__ void scan_write_hist(const GatedScan& p, int q0, int ctx, int sin, int sout, int last, int c) {
  const int h = p.taps - 1;
  for (int m = 0; m < h; ++m)
    static_cast<T*>(p.hist)[((long)sout * h + m) * p.C + c] = (T)scan_x<T>(p, q0, ctx, sin, last + 1 - h + m, c);
}

template <typename T>
__global__ void __launch_bounds__(256)
scan_conv_kernel(const GatedScan p) {
  const long n = (long)p.T * p.C;
  for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long)gridDim.x * blockDim.x) {
    const int t = (int)(i / p.C), c = (int)(i - (long)t * p.C);
    const int seq = min(max(p.row_seq[t], 0), p.num_seqs - 1);
    const int q0 = p.q_start[seq], ctx = p.context[seq], off = t - q0;
    int sin, sout;
    scan_rows(p, seq, sin, sout);
    float s = p.conv_b[c];
    for (int j = 0; j < p.taps; ++j) s = fmaf(p.conv[(long)j * p.C + c], scan_x<T>(p, q0, ctx, sin, off - p.taps + 1 + j, c), s);
    static_cast<float*>(p.u)[i] = s;
    if (sout >= 0 && t == p.q_start[seq + 1] - 1) scan_write_hist<T>(p, q0, ctx, sin, sout, off, c);
  }
}

template <typename T>
__global__ void __launch_bounds__(128)
scan_plain_kernel(const GatedScan p) {
  const int c = blockIdx.x * 128 + threadIdx.x, seq = blockIdx.y;
  if (c >= p.C) return;
  int sin, sout;
  scan_rows(p, seq, sin, sout);
  float S = p.context[seq] > 0 ? p.state[(long)sin * p.C + c] : 0.f;
  const float decay = p.decay[c];
  for (long t = p.q_start[seq]; t < p.q_start[seq + 1]; ++t) {
    const float r = 1.0f / (1.0f + expf(-p.z[t * p.C + c])), g = 1.0f / (1.0f + expf(-p.z[((long)p.T + t) * p.C + c]));
    const float la = decay * r;
    S = expf(la) * S + sqrtf(-expm1f(2.0f * la)) * g * static_cast<const float*>(p.u)[t * p.C + c];
    const float y = (float)static_cast<const T*>(p.proj)[t * p.ldp + c];
    const float th = tanhf(0.7978845608028654f * (y + 0.044715f * y * y * y));
    static_cast<T*>(p.out)[t * p.C + c] = (T)(S * (0.5f * y * (1.0f + th)));
  }
  if (sout >= 0) p.state[(long)sout * p.C + c] = S;
}

// ---------------------------------------------------------------------------- one token each
constexpr int SS_CH = 32;       // channels per block

__global__ void __launch_bounds__(128)
scan_step_kernel(const GatedScan p) {
  extern __shared__ __align__(16) uint8_t smem[];           // u: [16][part * 2 + 16 bytes]
  __shared__ int s_row[16], s_ctx[16], s_in[16], s_out[16];
  const int slices = (p.part + SS_CH - 1) / SS_CH;
  const int blk = blockIdx.x / slices, n_base = (blockIdx.x % slices) * SS_CH;
  const int l0 = blockIdx.y * 16, nt = min(16, p.n_list - l0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, j = lane & 3;
  const int c0 = blk * p.part, pitch = p.part * 2 + 16, h = p.taps - 1;
  if (tid < 16) {
    const int seq = min(max(p.seq_list[l0 + min(tid, nt - 1)], 0), p.num_seqs - 1);
    s_row[tid] = p.q_start[seq];
    s_ctx[tid] = p.context[seq];
    int a, b;
    scan_rows(p, seq, a, b);
    s_in[tid] = a;
    s_out[tid] = tid < nt ? b : -1;
  }
  __syncthreads();
  const bf16* proj = static_cast<const bf16*>(p.proj);
  const bf16* hist = static_cast<const bf16*>(p.hist);
  const int vecs = p.part / 8;
  for (int i = tid; i < 16 * vecs; i += 128) {
    const int t = i / vecs, c = c0 + (i - t * vecs) * 8;
    float s[8], x[8], w[8];
    load8<float>(p.conv_b + c, s);
    for (int q = 0; q < p.taps; ++q) {
      const int b = q - h;                                   // 0: the new token; negative: history
      if (b == 0) load8<bf16>(proj + (long)s_row[t] * p.ldp + p.C + c, x);
      else if (s_ctx[t] + b >= 0) load8<bf16>(hist + ((long)s_in[t] * h + h + b) * p.C + c, x);
      else continue;
      load8<float>(p.conv + (long)q * p.C + c, w);
#pragma unroll
      for (int e = 0; e < 8; ++e) s[e] = fmaf(w[e], x[e], s[e]);
    }
    store8<bf16>(reinterpret_cast<bf16*>(smem + t * pitch + (i - t * vecs) * 16), s);
  }
  // new history of this block's channels
  if (h > 0) {
    const int nv = min(SS_CH, p.part - n_base) / 8;
    for (int i = tid; i < nt * h * nv; i += 128) {
      const int t = i / (h * nv), m = (i / nv) % h, c = c0 + n_base + (i % nv) * 8;
      if (s_out[t] < 0) continue;
      const int b = m + 1 - h;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (b == 0) v = *reinterpret_cast<const uint4*>(proj + (long)s_row[t] * p.ldp + p.C + c);
      else if (s_ctx[t] + b >= 0) v = *reinterpret_cast<const uint4*>(hist + ((long)s_in[t] * h + h + b) * p.C + c);
      *reinterpret_cast<uint4*>(static_cast<bf16*>(p.hist) + ((long)s_out[t] * h + m) * p.C + c) = v;
    }
  }
  __syncthreads();
  const int n0 = n_base + warp * 8;                          // this warp's eight channels
  if (n0 >= p.part) return;
  float acc[2][4] = {};
  const bf16* w = static_cast<const bf16*>(p.gates) + ((long)blk * p.part + n0 + g) * p.part + j * 8;
  const long gate_stride = (long)p.blocks * p.part * p.part;
  const uint8_t* ua = smem + g * pitch + j * 16;
  const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
#pragma unroll 8
  for (int k = 0; k < p.part; k += 32) {
    const bool in = k + j * 8 < p.part;
    const uint4 br = in ? *reinterpret_cast<const uint4*>(w + k) : zero;
    const uint4 bi = in ? *reinterpret_cast<const uint4*>(w + gate_stride + k) : zero;
    const uint4 a0 = in ? *reinterpret_cast<const uint4*>(ua + k * 2) : zero;
    const uint4 a1 = in ? *reinterpret_cast<const uint4*>(ua + 8 * pitch + k * 2) : zero;
#define OMNI_SS_MMA(ACC, B0, B1, A0, A1, A2, A3)                                                                             \
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, "          \
               "{%0, %1, %2, %3};"                                                                                           \
               : "+f"(ACC[0]), "+f"(ACC[1]), "+f"(ACC[2]), "+f"(ACC[3])                                                      \
               : "r"(A0), "r"(A1), "r"(A2), "r"(A3), "r"(B0), "r"(B1))
    OMNI_SS_MMA(acc[0], br.x, br.y, a0.x, a1.x, a0.y, a1.y);
    OMNI_SS_MMA(acc[0], br.z, br.w, a0.z, a1.z, a0.w, a1.w);
    OMNI_SS_MMA(acc[1], bi.x, bi.y, a0.x, a1.x, a0.y, a1.y);
    OMNI_SS_MMA(acc[1], bi.z, bi.w, a0.z, a1.z, a0.w, a1.w);
#undef OMNI_SS_MMA
  }
  const int cl = n0 + j * 2, c = c0 + cl;                    // this thread's two channels
  const float2 b0 = *reinterpret_cast<const float2*>(p.gates_b + c), b1 = *reinterpret_cast<const float2*>(p.gates_b + p.C + c);
  const float2 dec = *reinterpret_cast<const float2*>(p.decay + c);
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const int t = u * 8 + g;
    if (t >= nt) continue;
    const long row = s_row[t];
    const float2 x = unpack_bf16(*reinterpret_cast<const uint32_t*>(smem + t * pitch + cl * 2));
    const float2 y = unpack_bf16(*reinterpret_cast<const uint32_t*>(proj + row * p.ldp + c));
    float2 S = make_float2(0.f, 0.f);
    if (s_ctx[t] > 0) S = *reinterpret_cast<const float2*>(p.state + (long)s_in[t] * p.C + c);
    float la, a, add;
    gate_step(acc[0][2 * u], acc[1][2 * u], -GS_LOG2E * b0.x, -GS_LOG2E * b1.x, x.x, dec.x * GS_LOG2E, la, a, add);
    S.x = fmaf(a, S.x, add);
    gate_step(acc[0][2 * u + 1], acc[1][2 * u + 1], -GS_LOG2E * b0.y, -GS_LOG2E * b1.y, x.y, dec.y * GS_LOG2E, la, a, add);
    S.y = fmaf(a, S.y, add);
    if (s_out[t] >= 0) *reinterpret_cast<float2*>(p.state + (long)s_out[t] * p.C + c) = S;
    *reinterpret_cast<uint32_t*>(static_cast<bf16*>(p.out) + row * p.C + c) = pack_bf16(S.x * gelu_short(y.x), S.y * gelu_short(y.y));
  }
}

}  // namespace omni

using namespace omni;

extern "C" int omni_scan_conv(const GatedScan* args, int is_bf16, void* stream) {
  const GatedScan& p = *args;
  if (p.T <= 0) return RC_OK;
  if (!scan_args_ok(p) || !p.u || !p.row_seq) return RC_BAD_ARG;
  long blocks = ((long)p.T * p.C + 255) / 256;
  if (blocks > 148 * 16) blocks = 148 * 16;
  if (is_bf16) scan_conv_kernel<bf16><<<(unsigned)blocks, 256, 0, (cudaStream_t)stream>>>(p);
  else scan_conv_kernel<float><<<(unsigned)blocks, 256, 0, (cudaStream_t)stream>>>(p);
  return (int)cudaGetLastError();
}

extern "C" int omni_scan_plain(const GatedScan* args, int is_bf16, void* stream) {
  const GatedScan& p = *args;
  if (p.T <= 0) return RC_OK;
  if (!scan_args_ok(p) || !p.u || !p.z || p.num_seqs > 65535) return RC_BAD_ARG;
  dim3 grid((p.C + 127) / 128, p.num_seqs);
  if (is_bf16) scan_plain_kernel<bf16><<<grid, 128, 0, (cudaStream_t)stream>>>(p);
  else scan_plain_kernel<float><<<grid, 128, 0, (cudaStream_t)stream>>>(p);
  return (int)cudaGetLastError();
}

extern "C" int omni_scan_step(const GatedScan* args, void* stream) {
  const GatedScan& p = *args;
  if (p.n_list <= 0) return RC_OK;
  if (!scan_args_ok(p) || !p.seq_list || p.part > 1024 || (p.n_list + 15) / 16 > 65535) return RC_BAD_ARG;
  dim3 grid(p.blocks * ((p.part + SS_CH - 1) / SS_CH), (p.n_list + 15) / 16);
  scan_step_kernel<<<grid, 128, 16 * (p.part * 2 + 16), (cudaStream_t)stream>>>(p);
  return (int)cudaGetLastError();
}
