// Helpers of kernels that walk rows of channels: eight channels per 16-byte (bf16) or 32-byte (fp32) access, block sums,
// the launch shape of a row.
#pragma once
#include "ptx_sm100.cuh"

namespace omni {

// eight consecutive elements as fp32
template <typename T> __device__ __forceinline__ void load8(const T* p, float (&v)[8]);
template <> __device__ __forceinline__ void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <> __device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&v)[8]) {
  const uint4 u = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 f = unpack_bf16(w[j]);
    v[2 * j] = f.x;
    v[2 * j + 1] = f.y;
  }
}
template <typename T> __device__ __forceinline__ void store8(T* p, const float (&v)[8]);
template <> __device__ __forceinline__ void store8<float>(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
template <> __device__ __forceinline__ void store8<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]),
                                            pack_bf16(v[6], v[7]));
}

// Sum of NV values over the block; every thread gets the totals.  `sh` holds 32 * NV floats.
template <int NV>
__device__ __forceinline__ void block_sum(float (&s)[NV], float* sh) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1)
#pragma unroll
    for (int i = 0; i < NV; ++i) s[i] += __shfl_xor_sync(0xffffffffu, s[i], o);
  __syncthreads();          // the previous use of `sh` is over
  if (lane == 0)
#pragma unroll
    for (int i = 0; i < NV; ++i) sh[warp * NV + i] = s[i];
  __syncthreads();
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    float t = 0.f;
    for (int w = 0; w < nw; ++w) t += sh[w * NV + i];
    s[i] = t;
  }
}

__device__ __forceinline__ float rms_scale(float sumsq, int n, float eps) {
  return 1.0f / sqrtf(sumsq / (float)n + eps);
}

// multiply eight values by `s` and the gains of their channels
__device__ __forceinline__ void scale_gain8(float (&v)[8], float s, const float* g, int gs, int c) {
  if (gs == 0) {
    const float k = s * g[0];
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= k;
  } else {
    float w[8];
    load8<float>(g + c, w);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] *= s * w[e];
  }
}

// threads and vectors per thread for a row of n channels (n <= 32768)
inline bool row_shape(int n, int& threads, int& nv) {
  const int vec = n / 8;
  for (threads = 64; threads < 1024 && threads < vec; threads *= 2) {
    if (threads >= 256 && vec <= threads * 2) break;
  }
  nv = (vec + threads - 1) / threads;
  nv = nv <= 1 ? 1 : (nv <= 2 ? 2 : 4);
  return vec <= threads * nv;
}

}  // namespace omni
