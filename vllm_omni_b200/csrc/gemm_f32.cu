// C[M, N] = A[M, K] W[N, K]^T (+ bias) in true fp32 on the CUDA cores: the matrix product of the exact
// mode, in which a decoder runs without any reduced-precision step.  64 x 64 tiles, 16-deep K slices,
// 4 x 4 results per thread; each result is one fixed-order chain over K, so a row's value does not
// depend on the other rows of the launch.
#include "host_util.h"

namespace omni {

constexpr int FB = 64, FK = 16;

// element strides between the problems of a batch (one per grid layer)
struct GemmF32Batch {
  long a, w, c, bias;
};

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ A, long lda, const float* __restrict__ W, long ldw, float* __restrict__ C,
                long ldc, int M, int N, int K, const float* __restrict__ bias, int act,
                float c0, float c1, GemmF32Batch b) {
  A += blockIdx.z * b.a;
  W += blockIdx.z * b.w;
  C += blockIdx.z * b.c;
  if (bias) bias += blockIdx.z * b.bias;
  __shared__ float sA[FK][FB + 4], sW[FK][FB + 4];
  const int m0 = blockIdx.y * FB, n0 = blockIdx.x * FB;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += FK) {
#pragma unroll
    for (int i = threadIdx.x; i < FB * FK; i += 256) {
      const int r = i / FK, k = i % FK;
      sA[k][r] = (m0 + r < M && k0 + k < K) ? A[(long)(m0 + r) * lda + k0 + k] : 0.f;
      sW[k][r] = (n0 + r < N && k0 + k < K) ? W[(long)(n0 + r) * ldw + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < FK; ++k) {
      float a[4], w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        a[i] = sA[k][ty * 4 + i];
        w[i] = sW[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], w[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N) {
        float v = acc[i][j] + (bias ? bias[n] : 0.f);
        if (act == 3) {                                    // squared ReLU
          v = fmaxf(v, 0.f);
          v *= v;
        } else if (act == 4) {                             // xIELU
          v = fmaf(0.5f, v, v > 0.f ? c0 * v * v : c1 * (expm1f(v) - v));
        }
        C[(long)m * ldc + n] = v;
      }
    }
}

}  // namespace omni

// `batch` problems of one shape whose operands lie the given strides apart; act: 0 none, 3 squared ReLU, 4 xIELU with
// two numbers (c0 z^2 + z / 2 above zero, c1 (e^z - 1 - z) + z / 2 below).
extern "C" int omni_gemm_f32_batched(const float* A, long lda, const float* W, long ldw, float* C, long ldc, int M, int N, int K,
                                     const float* bias, int act, int batch, long a_stride, long w_stride, long c_stride,
                                     long bias_stride, float c0, float c1, void* stream) {
  if (M <= 0 || N <= 0 || batch <= 0) return omni::RC_OK;
  if (K <= 0 || (M + omni::FB - 1) / omni::FB > 65535 || batch > 65535 || act < 0 || act == 1 || act == 2 || act > 4) return omni::RC_BAD_ARG;
  dim3 grid((N + omni::FB - 1) / omni::FB, (M + omni::FB - 1) / omni::FB, batch);
  const omni::GemmF32Batch b = {a_stride, w_stride, c_stride, bias_stride};
  omni::gemm_f32_kernel<<<grid, 256, 0, (cudaStream_t)stream>>>(A, lda, W, ldw, C, ldc, M, N, K, bias, act, c0, c1, b);
  return (int)cudaGetLastError();
}

extern "C" int omni_gemm_f32(const float* A, long lda, const float* W, long ldw, float* C, long ldc, int M, int N, int K,
                             const float* bias, void* stream) {
  return omni_gemm_f32_batched(A, lda, W, ldw, C, ldc, M, N, K, bias, 0, 1, 0, 0, 0, 0, 0.f, 0.f, stream);
}
