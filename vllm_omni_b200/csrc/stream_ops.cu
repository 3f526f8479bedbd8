// Steps of decoders whose fp32 residual stream takes scaled branches, for bf16 activations (serving) and fp32
// activations (exact mode):
//
//   omni_stream_step    x += mult * branch, then the rows the next GEMM reads (one launch).  The branch is a row or the
//                       weighted sum of a token's expert rows plus a shared expert's row (times the sigmoid of one
//                       logit per token, where given); with a gain per channel either is divided by its rms first.
//                       Or x starts as mult * an embedding row, or as a row that replaces it.  Output: nothing, x in the activations' type,
//                       w tanh(alpha x) + b, or x divided by its rms times w.
//   omni_rotary_rows    magnitude * cos / sin of position * frequency, angles reduced in fp64
//   omni_gelu_lookup    z = gelu(z) * a token's row of a table
//
// Rows are padded to a multiple of 8 channels with zeros; padding does not count in means.
#include "host_util.h"
#include "row_ops.cuh"

namespace omni {

enum StreamSource : int { SRC_EMBED = 0, SRC_ROW = 1, SRC_NORMED = 2, SRC_EXPERTS = 3, SRC_EXPERTS_NORMED = 4 };
enum StreamOut : int { OUT_NONE = 0, OUT_CAST = 1, OUT_TANH = 2, OUT_RMS = 3 };

struct StreamStep {
  float* x;
  int rows, D, Dp;
  int source, out_mode;
  float mult, eps;
  const void* y; long ldy, y_rows;     // branch rows; expert rows: y_rows of them
  const float* gain;                   // [Dp]
  const int* row_of_pair;              // [rows * k] row of (token, choice) in y, or nullptr: pair order
  const float* weights; int k;         // [rows, k]
  const void* shared; long lds;        // [rows, Dp] or nullptr
  const long* ids; const void* embed; int vocab;    // [rows], [vocab, Dp]
  const void* overlay; const unsigned char* overlay_mask;
  void* out;                           // [rows, Dp]
  const float* alpha; const float* w; const float* b;
  int* status;
  const void* shared_gate; long ldsg;  // [rows] logits at this pitch, or nullptr
  float out_eps;                       // OUT_RMS
};

// tanh for values that are rounded to bf16 next: absolute error about 1e-7
__device__ __forceinline__ float tanh_short(float z) { return 1.0f - __fdividef(2.0f, __expf(2.0f * fminf(z, 40.f)) + 1.0f); }
template <typename T> __device__ __forceinline__ float tanh_for(float z);
template <> __device__ __forceinline__ float tanh_for<float>(float z) { return tanhf(z); }
template <> __device__ __forceinline__ float tanh_for<__nv_bfloat16>(float z) { return tanh_short(z); }

template <typename T, int SRC, int NV>
__global__ void __launch_bounds__(1024)
stream_step_kernel(const StreamStep p) {
  constexpr bool EXPERTS = SRC == SRC_EXPERTS || SRC == SRC_EXPERTS_NORMED;
  constexpr bool NORMED = SRC == SRC_NORMED || SRC == SRC_EXPERTS_NORMED;
  __shared__ float sh[32];
  const long r = blockIdx.x;
  float xv[NV][8], yv[NV][8];
  float ss[1] = {0.f};
  const T* src = nullptr;
  float scale = p.mult;
  if (SRC == SRC_EMBED) {
    long id = p.ids[r];
    id = id < 0 ? 0 : (id >= p.vocab ? p.vocab - 1 : id);
    const bool over = p.overlay != nullptr && (p.overlay_mask == nullptr || p.overlay_mask[r]);
    if (over) scale = 1.f;
    src = over ? static_cast<const T*>(p.overlay) + r * p.Dp : static_cast<const T*>(p.embed) + id * p.Dp;
  } else if (!EXPERTS) {
    src = static_cast<const T*>(p.y) + r * p.ldy;
  }
  float sg = 1.f;
  if (EXPERTS && p.shared_gate) sg = 1.0f / (1.0f + expf(-(float)static_cast<const T*>(p.shared_gate)[r * p.ldsg]));
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c >= p.Dp) continue;
    if (EXPERTS) {
      if (p.shared) {
        load8<T>(static_cast<const T*>(p.shared) + r * p.lds + c, yv[i]);
#pragma unroll
        for (int e = 0; e < 8; ++e) yv[i][e] *= sg;
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) yv[i][e] = 0.f;
      }
      for (int j = 0; j < p.k; ++j) {
        const long pair = r * p.k + j;
        const long row = p.row_of_pair ? p.row_of_pair[pair] : pair;
        if (row < 0 || row >= p.y_rows) {
          if (p.status) atomicCAS(p.status, 0, (int)ERR_BOUNDS);
          continue;
        }
        const float wt = p.weights[pair];
        float v[8];
        load8<T>(static_cast<const T*>(p.y) + row * p.ldy + c, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) yv[i][e] = fmaf(wt, v[e], yv[i][e]);
      }
    } else {
      load8<T>(src + c, yv[i]);
    }
    if (SRC != SRC_EMBED) load8<float>(p.x + r * p.Dp + c, xv[i]);
    if (NORMED) {
#pragma unroll
      for (int e = 0; e < 8; ++e) ss[0] = fmaf(yv[i][e], yv[i][e], ss[0]);
    }
  }
  if (NORMED) {
    block_sum<1>(ss, sh);
    scale = p.mult * rms_scale(ss[0], p.D, p.eps);
  }
  const float alpha = p.out_mode == OUT_TANH ? p.alpha[0] : 0.f;
  float so[1] = {0.f};
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c >= p.Dp) continue;
    if (SRC == SRC_EMBED) {
#pragma unroll
      for (int e = 0; e < 8; ++e) xv[i][e] = scale * yv[i][e];
    } else if (NORMED) {
      float g[8];
      load8<float>(p.gain + c, g);
#pragma unroll
      for (int e = 0; e < 8; ++e) xv[i][e] = fmaf(scale * yv[i][e], g[e], xv[i][e]);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) xv[i][e] = fmaf(scale, yv[i][e], xv[i][e]);
    }
    store8<float>(p.x + r * p.Dp + c, xv[i]);
    if (p.out_mode == OUT_CAST) {
      store8<T>(static_cast<T*>(p.out) + r * p.Dp + c, xv[i]);
    } else if (p.out_mode == OUT_TANH) {
      float w[8], b[8];
      load8<float>(p.w + c, w);
      load8<float>(p.b + c, b);
#pragma unroll
      for (int e = 0; e < 8; ++e) w[e] = fmaf(w[e], tanh_for<T>(alpha * xv[i][e]), b[e]);
      store8<T>(static_cast<T*>(p.out) + r * p.Dp + c, w);
    } else if (p.out_mode == OUT_RMS) {
#pragma unroll
      for (int e = 0; e < 8; ++e) so[0] = fmaf(xv[i][e], xv[i][e], so[0]);
    }
  }
  if (p.out_mode != OUT_RMS) return;
  block_sum<1>(so, sh);
  const float scale_out = rms_scale(so[0], p.D, p.out_eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (i * blockDim.x + threadIdx.x) * 8;
    if (c >= p.Dp) continue;
    scale_gain8(xv[i], scale_out, p.w, 1, c);
    store8<T>(static_cast<T*>(p.out) + r * p.Dp + c, xv[i]);
  }
}

// out[t, i] = mag (cos, sin) of pos[t] * freq[i]
__global__ void __launch_bounds__(256)
rotary_rows_kernel(const long* __restrict__ pos, const double* __restrict__ freq, float mag, float2* __restrict__ out, int T,
                   int half) {
  const long n = (long)T * half;
  for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (long)gridDim.x * blockDim.x) {
    const double two_pi = 6.283185307179586476925;
    const double a = (double)pos[i / half] * freq[i % half];
    float s, c;
    sincosf((float)(a - two_pi * rint(a / two_pi)), &s, &c);
    out[i] = make_float2(mag * c, mag * s);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
gelu_lookup_kernel(T* __restrict__ z, long ldz, const T* __restrict__ table, long ldt, const long* __restrict__ ids, int vocab,
                   int col, int n, int rows) {
  const long total = (long)rows * n;
  for (long i = (long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x) {
    const long r = i / n;
    const int c = (int)(i - r * n);
    long id = ids[r];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    const float v = (float)z[r * ldz + c], e = (float)table[id * ldt + col + c];
    const float u = 0.7978845608028654f * fmaf(0.044715f * v * v, v, v);
    z[r * ldz + c] = (T)(0.5f * v * (1.0f + tanh_for<T>(u)) * e);
  }
}

template <typename T, int SRC>
static int launch_step(const StreamStep& p, int threads, int nv, cudaStream_t st) {
  if (nv == 1) stream_step_kernel<T, SRC, 1><<<p.rows, threads, 0, st>>>(p);
  else if (nv == 2) stream_step_kernel<T, SRC, 2><<<p.rows, threads, 0, st>>>(p);
  else stream_step_kernel<T, SRC, 4><<<p.rows, threads, 0, st>>>(p);
  return (int)cudaGetLastError();
}

template <typename T>
static int launch_source(const StreamStep& p, int threads, int nv, cudaStream_t st) {
  switch (p.source) {
    case SRC_EMBED: return launch_step<T, SRC_EMBED>(p, threads, nv, st);
    case SRC_ROW: return launch_step<T, SRC_ROW>(p, threads, nv, st);
    case SRC_NORMED: return launch_step<T, SRC_NORMED>(p, threads, nv, st);
    case SRC_EXPERTS: return launch_step<T, SRC_EXPERTS>(p, threads, nv, st);
    case SRC_EXPERTS_NORMED: return launch_step<T, SRC_EXPERTS_NORMED>(p, threads, nv, st);
    default: return RC_BAD_ARG;
  }
}

}  // namespace omni

using namespace omni;

extern "C" int omni_stream_step(const StreamStep* args, int is_bf16, void* stream) {
  const StreamStep& p = *args;
  if (p.rows <= 0) return RC_OK;
  int threads, nv;
  if ((p.Dp & 7) || (p.ldy & 7) || (p.lds & 7) || p.D > p.Dp || !row_shape(p.Dp, threads, nv)) return RC_BAD_ARG;
  if (p.source == SRC_EMBED ? (!p.ids || !p.embed || p.vocab <= 0) : !p.y) return RC_BAD_ARG;
  const bool experts = p.source == SRC_EXPERTS || p.source == SRC_EXPERTS_NORMED;
  if (((p.source == SRC_NORMED || p.source == SRC_EXPERTS_NORMED) && !p.gain) || (experts && (!p.weights || p.k <= 0))) return RC_BAD_ARG;
  if ((p.out_mode != OUT_NONE && !p.out) || (p.out_mode == OUT_TANH && (!p.alpha || !p.w || !p.b)) || (p.out_mode == OUT_RMS && !p.w))
    return RC_BAD_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  return is_bf16 ? launch_source<__nv_bfloat16>(p, threads, nv, st) : launch_source<float>(p, threads, nv, st);
}

extern "C" int omni_rotary_rows(const long* pos, const double* freq, float mag, float* out, int T, int half, void* stream) {
  if (T <= 0 || half <= 0) return RC_OK;
  long blocks = ((long)T * half + 255) / 256;
  if (blocks > 148 * 8) blocks = 148 * 8;
  rotary_rows_kernel<<<(unsigned)blocks, 256, 0, (cudaStream_t)stream>>>(pos, freq, mag, reinterpret_cast<float2*>(out), T, half);
  return (int)cudaGetLastError();
}

extern "C" int omni_gelu_lookup(void* z, long ldz, const void* table, long ldt, const long* ids, int vocab, int col, int n,
                                int rows, int is_bf16, void* stream) {
  if (rows <= 0 || n <= 0) return RC_OK;
  if (vocab <= 0 || col < 0 || col + n > ldt || n > ldz) return RC_BAD_ARG;
  long blocks = ((long)rows * n + 255) / 256;
  if (blocks > 148 * 8) blocks = 148 * 8;
  cudaStream_t st = (cudaStream_t)stream;
  if (is_bf16)
    gelu_lookup_kernel<__nv_bfloat16><<<(unsigned)blocks, 256, 0, st>>>((__nv_bfloat16*)z, ldz, (const __nv_bfloat16*)table, ldt,
                                                                        ids, vocab, col, n, rows);
  else
    gelu_lookup_kernel<float><<<(unsigned)blocks, 256, 0, st>>>((float*)z, ldz, (const float*)table, ldt, ids, vocab, col, n, rows);
  return (int)cudaGetLastError();
}
