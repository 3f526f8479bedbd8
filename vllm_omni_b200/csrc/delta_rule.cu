// Delta-rule recurrences token by token (delta_rule.cuh says what is computed).
//
//   omni_delta_steps    one block per (sequence, head): the head's state in registers, a thread owns four value columns of
//                       every n-th key row; per token convolution, unit lengths, decays, both reads of the state, the write,
//                       norm and gate.  Decoded tokens take exactly one turn (one launch does the whole mixer, and the state
//                       is read and written once); the exact mode walks whole portions.  States too large for one block are
//                       cut into column slices, whose results go to `raw`
//   omni_delta_finish   norm and gate of the results in `raw`
#include "delta_rule.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

constexpr int DS_THREADS = 256;

template <typename T, bool CHANNEL, int NR>
__global__ void __launch_bounds__(DS_THREADS)
delta_steps_kernel(const DeltaRule p, const int cw) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float sh[64];
  const int tid = threadIdx.x;
  const int seq = p.seq_list ? min(max(p.seq_list[blockIdx.x], 0), p.num_seqs - 1) : blockIdx.x;
  const int h = blockIdx.y, R = p.H / p.G, g = h / R;
  const int c0 = blockIdx.z * cw, w = min(cw, p.vp - c0);
  const int nc = w / 4, RG = DS_THREADS / nc;                // four-column groups, key rows side by side
  const int c4 = tid % nc, rg = tid / nc;
  const bool act = rg < RG;
  float* s_q = sm;                                           // [dp] r or q before its length
  float* s_k = s_q + p.dp;                                   // [dp] k before its length
  float* s_d = s_k + p.dp;                                   // [dp] channel: decay
  float* s_a = s_d + p.dp;                                   // [dp] channel: removal rate
  float* s_v = s_a + p.dp;                                   // [w]
  float* red = s_v + cw;                                     // [RG, w]
  float* red2 = red + 4 * DS_THREADS;
  const int q0 = p.q_start[seq], n = p.q_start[seq + 1] - q0, ctx = p.context[seq];
  if (n <= 0) return;
  int sin, sout;
  delta_rows(p, seq, sin, sout);
  const long head_state = (long)p.dp * p.vp;
  const float* S0 = p.state + ((long)sin * p.H + h) * head_state + c0 + c4 * 4;
  float4 S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = rg + i * RG;
    S[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (act && r < p.dp && ctx > 0) S[i] = *reinterpret_cast<const float4*>(S0 + (long)r * p.vp);
  }
  const T* proj = static_cast<const T*>(p.proj);
  T* hist = static_cast<T*>(p.hist);
  const int hl = p.taps - 1, C = 2 * p.G * p.dp + p.H * p.vp;
  // convolution input of channel c at row b of the portion (negative: history)
  auto conv_x = [&](int b, int c) -> float {
    if (b >= 0) return (float)proj[(long)(q0 + b) * p.ldp + p.q_col + c];
    if (ctx + b >= 0) return (float)hist[((long)sin * hl + hl + b) * C + c];
    return 0.f;
  };
  // channel of element i of this block: q, k of the head's group, v of the block's columns
  auto channel_of = [&](int i) {
    return i < p.dp ? g * p.dp + i : (i < 2 * p.dp ? p.G * p.dp + g * p.dp + i - p.dp : 2 * p.G * p.dp + h * p.vp + c0 + i - 2 * p.dp);
  };
  for (int t = 0; t < n; ++t) {
    const long row = q0 + t;
    const T* pr = proj + row * p.ldp;
    float ss[2] = {0.f, 0.f};                                // sums of squares of q and k
    if (CHANNEL) {
      const T* z = static_cast<const T*>(p.z) + row * p.ldz;
      for (int c = tid; c < p.dp; c += DS_THREADS) {
        const int hc = h * p.dp + c;
        const float k = (float)pr[p.k_col + hc];
        s_q[c] = (float)pr[p.q_col + hc];
        s_k[c] = k;
        s_d[c] = expf(p.decay_scale * dr_sigmoid((float)z[hc] + p.decay_bias[hc]));
        s_a[c] = dr_sigmoid((float)pr[p.a_col + hc] + p.removal_bias[hc]);
        ss[1] = fmaf(k, k, ss[1]);
      }
      for (int c = tid; c < w; c += DS_THREADS) s_v[c] = (float)pr[p.v_col + h * p.vp + c0 + c];
    } else {
      for (int i = tid; i < 2 * p.dp + w; i += DS_THREADS) {
        const int c = channel_of(i);
        float x = 0.f;
        for (int j = 0; j < p.taps; ++j) x = fmaf(p.conv[(long)j * C + c], conv_x(t - hl + j, c), x);
        x = x / (1.0f + expf(-x));
        if (i < p.dp) {
          s_q[i] = x;
          ss[0] = fmaf(x, x, ss[0]);
        } else if (i < 2 * p.dp) {
          s_k[i - p.dp] = x;
          ss[1] = fmaf(x, x, ss[1]);
        } else {
          s_v[i - 2 * p.dp] = x;
        }
      }
    }
    block_sum<2>(ss, sh);                                    // also: the vectors are in place
    const float ik = 1.0f / sqrtf(ss[1] + p.unit_eps);
    float decay = 1.f, beta = 1.f, o_mul = 1.f;
    if (!CHANNEL) {
      decay = expf(p.rate[h] * dr_softplus((float)pr[p.a_col + h] + p.dt_bias[h]));
      beta = dr_sigmoid((float)pr[p.b_col + h]);
      o_mul = p.q_mul / sqrtf(ss[0] + p.unit_eps);
    }
    // what the old state answers to the unit key
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    if (act) {
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int r = rg + i * RG;
        if (r < p.dp) {
          const float k = s_k[r];
          y.x = fmaf(k, S[i].x, y.x);
          y.y = fmaf(k, S[i].y, y.y);
          y.z = fmaf(k, S[i].z, y.z);
          y.w = fmaf(k, S[i].w, y.w);
        }
      }
      *reinterpret_cast<float4*>(red + rg * w + c4 * 4) = y;
    }
    __syncthreads();
    y = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 o = y;
    if (act) {
      for (int i = 0; i < RG; ++i) {
        const float4 a = *reinterpret_cast<const float4*>(red + i * w + c4 * 4);
        y.x += a.x; y.y += a.y; y.z += a.z; y.w += a.w;
      }
      y.x *= ik; y.y *= ik; y.z *= ik; y.w *= ik;
      const float4 v = *reinterpret_cast<const float4*>(s_v + c4 * 4);
      if (!CHANNEL) {                                        // what is written along the unit key
        y.x = beta * (v.x - decay * y.x) * ik;
        y.y = beta * (v.y - decay * y.y) * ik;
        y.z = beta * (v.z - decay * y.z) * ik;
        y.w = beta * (v.w - decay * y.w) * ik;
      }
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int r = rg + i * RG;
        if (r < p.dp) {
          const float k = s_k[r], q = s_q[r];
          if (CHANNEL) {
            const float d = s_d[r], a = -s_a[r] * (k * ik);
            S[i].x = fmaf(k, v.x, fmaf(a, y.x, d * S[i].x));
            S[i].y = fmaf(k, v.y, fmaf(a, y.y, d * S[i].y));
            S[i].z = fmaf(k, v.z, fmaf(a, y.z, d * S[i].z));
            S[i].w = fmaf(k, v.w, fmaf(a, y.w, d * S[i].w));
          } else {
            S[i].x = fmaf(k, y.x, decay * S[i].x);
            S[i].y = fmaf(k, y.y, decay * S[i].y);
            S[i].z = fmaf(k, y.z, decay * S[i].z);
            S[i].w = fmaf(k, y.w, decay * S[i].w);
          }
          o.x = fmaf(q, S[i].x, o.x);
          o.y = fmaf(q, S[i].y, o.y);
          o.z = fmaf(q, S[i].z, o.z);
          o.w = fmaf(q, S[i].w, o.w);
        }
      }
      *reinterpret_cast<float4*>(red2 + rg * w + c4 * 4) = o;
    }
    __syncthreads();                                         // every use of this token's vectors is over
    float res[4] = {0.f, 0.f, 0.f, 0.f}, so[1] = {0.f};
    if (tid < nc) {
      for (int i = 0; i < RG; ++i) {
        const float4 a = *reinterpret_cast<const float4*>(red2 + i * w + tid * 4);
        res[0] += a.x; res[1] += a.y; res[2] += a.z; res[3] += a.w;
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        res[e] *= o_mul;
        so[0] = fmaf(res[e], res[e], so[0]);
      }
    }
    const int col = h * p.vp + c0 + tid * 4;
    if (gridDim.z > 1) {
      if (tid < nc)
#pragma unroll
        for (int e = 0; e < 4; ++e) static_cast<T*>(p.raw)[row * p.H * p.vp + col + e] = (T)res[e];
    } else {
      block_sum<1>(so, sh);
      if (tid < nc) {
        const float s = rms_scale(so[0], p.dv, p.eps);
        const float* gain = p.gain + (long)h * p.gain_hs + tid * 4;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float gz = (float)pr[p.g_col + col + e], open = dr_sigmoid(gz);
          static_cast<T*>(p.out)[row * p.ldo + col + e] = (T)(res[e] * s * gain[e] * (CHANNEL ? open : gz * open));
        }
      }
    }
  }
  if (sout < 0) return;
  float* S1 = p.state + ((long)sout * p.H + h) * head_state + c0 + c4 * 4;
#pragma unroll
  for (int i = 0; i < NR; ++i) {
    const int r = rg + i * RG;
    if (act && r < p.dp) *reinterpret_cast<float4*>(S1 + (long)r * p.vp) = S[i];
  }
  if (!CHANNEL && hl > 0) {
    // new history: the group's first head writes q and k, every block its values
    const bool first = h == g * R && blockIdx.z == 0;
    for (int i = first ? tid : 2 * p.dp + tid; i < 2 * p.dp + w; i += DS_THREADS) {
      const int c = channel_of(i);
      for (int m = 0; m < hl; ++m) hist[((long)sout * hl + m) * C + c] = (T)conv_x(n - hl + m, c);
    }
  }
}

// One group of lanes per (row, head), eight channels per lane and turn.  ONE: a turn covers the head, and a group takes two
// rows with all loads in flight.
template <typename T, bool CHANNEL, bool ONE>
__global__ void __launch_bounds__(256)
delta_finish_kernel(const DeltaRule p, const int lph) {
  constexpr int ROWS = ONE ? 2 : 1;
  const int lane = threadIdx.x & (lph - 1), h = blockIdx.y;
  const int t0 = (blockIdx.x * (256 / lph) + threadIdx.x / lph) * ROWS;
  const float* gain = p.gain + (long)h * p.gain_hs;
  const float inv = 1.0f / (float)p.dv;
  auto opened = [&](float (&v)[8], const float (&z)[8], const float (&gn)[8], float s) {
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float open = sizeof(T) == 4 ? dr_sigmoid(z[e]) : dr_rcp(1.0f + dr_ex2(-1.4426950408889634f * z[e]));
      v[e] *= (s * gn[e]) * (CHANNEL ? open : z[e] * open);
    }
  };
  float gn[8];
  if (ONE && lane * 8 < p.vp) load8<float>(gain + lane * 8, gn);
  float v[ROWS][8], z[ROWS][8], ss[ROWS];
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const long row = min(t0 + i, p.T - 1);                   // idle groups keep the shuffles company
    const T* raw = static_cast<const T*>(p.raw) + row * p.H * p.vp + (long)h * p.vp;
    const T* gate = static_cast<const T*>(p.proj) + row * p.ldp + p.g_col + (long)h * p.vp;
#pragma unroll
    for (int e = 0; e < 8; ++e) v[i][e] = z[i][e] = 0.f;
    ss[i] = 0.f;
    for (int c = lane * 8; c < p.vp; c += lph * 8) {
      load8<T>(raw + c, v[i]);
      if (ONE) load8<T>(gate + c, z[i]);
      else
#pragma unroll
        for (int e = 0; e < 8; ++e) ss[i] = fmaf(v[i][e], v[i][e], ss[i]);
      if (ONE) break;
    }
  }
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    if (ONE)
#pragma unroll
      for (int e = 0; e < 8; ++e) ss[i] = fmaf(v[i][e], v[i][e], ss[i]);
    for (int o = lph >> 1; o > 0; o >>= 1) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], o);
  }
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    const long row = t0 + i;
    if (row >= p.T) return;
    const float s = sizeof(T) == 4 ? rms_scale(ss[i], p.dv, p.eps) : rsqrtf(fmaf(ss[i], inv, p.eps));
    T* out = static_cast<T*>(p.out) + row * p.ldo + (long)h * p.vp;
    for (int c = lane * 8; c < p.vp; c += lph * 8) {
      if (!ONE) {
        load8<T>(static_cast<const T*>(p.raw) + row * p.H * p.vp + (long)h * p.vp + c, v[i]);
        load8<T>(static_cast<const T*>(p.proj) + row * p.ldp + p.g_col + (long)h * p.vp + c, z[i]);
      }
      if (!ONE) load8<float>(gain + c, gn);
      opened(v[i], z[i], gn, s);
      store8<T>(out + c, v[i]);
      if (ONE) break;
    }
  }
}

template <typename T, bool CHANNEL>
static int launch_steps(const DeltaRule& p, int cw, cudaStream_t st) {
  const int nc = cw / 4, RG = DS_THREADS / nc, rows = (p.dp + RG - 1) / RG;
  const dim3 grid(p.seq_list ? p.n_list : p.num_seqs, p.H, (p.vp + cw - 1) / cw);
  const int smem = (4 * p.dp + cw + 8 * DS_THREADS) * 4;
  if (smem > 47 * 1024) return RC_TOO_LARGE;
  if (rows <= 4) delta_steps_kernel<T, CHANNEL, 4><<<grid, DS_THREADS, smem, st>>>(p, cw);
  else if (rows <= 8) delta_steps_kernel<T, CHANNEL, 8><<<grid, DS_THREADS, smem, st>>>(p, cw);
  else if (rows <= 16) delta_steps_kernel<T, CHANNEL, 16><<<grid, DS_THREADS, smem, st>>>(p, cw);
  else if (rows <= 24) delta_steps_kernel<T, CHANNEL, 24><<<grid, DS_THREADS, smem, st>>>(p, cw);
  else return RC_TOO_LARGE;
  return (int)cudaGetLastError();
}

template <typename T, bool CHANNEL>
static int launch_finish(const DeltaRule& p, cudaStream_t st) {
  int lph = 1;
  while (lph < 32 && lph * 8 < p.vp) lph *= 2;
  const bool one = lph * 8 >= p.vp;
  const int rows = 256 / lph * (one ? 2 : 1);
  const dim3 grid((p.T + rows - 1) / rows, p.H);
  if (one) delta_finish_kernel<T, CHANNEL, true><<<grid, 256, 0, st>>>(p, lph);
  else delta_finish_kernel<T, CHANNEL, false><<<grid, 256, 0, st>>>(p, lph);
  return (int)cudaGetLastError();
}

}  // namespace omni

using namespace omni;

// wide: results before the norm go to `raw`, column slices of a head's state to blocks of their own.
extern "C" int omni_delta_steps(const DeltaRule* args, int channel, int is_bf16, int wide, void* stream) {
  const DeltaRule& p = *args;
  if (p.T <= 0 || (p.seq_list && p.n_list <= 0)) return RC_OK;
  if (!delta_args_ok(p, channel) || (wide && !p.raw)) return RC_BAD_ARG;
  int cw = p.vp;
  if (wide) {                                                // at least two slices of at most 64 columns and 16384 numbers
    cw = 16;
    while (cw < 64 && 2 * cw < p.vp && 2 * cw * p.dp <= 16384) cw *= 2;
    if (cw >= p.vp) cw = p.vp > 16 ? 16 : 0;
    if (cw == 0) return RC_TOO_LARGE;
  } else if (p.dp * p.vp > 16384) {
    return RC_BAD_ARG;
  }
  if (cw > 4 * DS_THREADS) return RC_TOO_LARGE;
  cudaStream_t st = (cudaStream_t)stream;
  if (is_bf16) return channel ? launch_steps<bf16, true>(p, cw, st) : launch_steps<bf16, false>(p, cw, st);
  return channel ? launch_steps<float, true>(p, cw, st) : launch_steps<float, false>(p, cw, st);
}

extern "C" int omni_delta_finish(const DeltaRule* args, int channel, int is_bf16, void* stream) {
  const DeltaRule& p = *args;
  if (p.T <= 0) return RC_OK;
  if (!delta_args_ok(p, channel) || !p.raw) return RC_BAD_ARG;
  cudaStream_t st = (cudaStream_t)stream;
  if (is_bf16) return channel ? launch_finish<bf16, true>(p, st) : launch_finish<bf16, false>(p, st);
  return channel ? launch_finish<float, true>(p, st) : launch_finish<float, false>(p, st);
}
