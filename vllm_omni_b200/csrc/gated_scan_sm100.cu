// Gated linear recurrence of prompt portions on tcgen05 tensor cores (gated_scan.cuh says what is computed).
//
// A portion is cut into runs of consecutive tokens.  One block owns 128 channels of one part and two runs (streams),
// and keeps the gate weights of its channels in shared memory; a run is walked in tiles of 32 tokens.  The gates are
// computed transposed, D[channel, token] = W[channel, k] u[token, k]^T, so that a thread of the epilogue owns one
// channel (a TMEM lane) and meets its tokens in order: the scan is a register recurrence.
//   warps 0-3, 4-7   epilogue of stream 0 / 1: both gates from tensor memory, decay, input term, scan; output
//   warps 8-9, 10-11 producers of stream 0 / 1: causal convolution of all channels of the part, bf16, to shared memory
//   warp 12          gate weights (TMA), MMA issue
// A run starts from what its sequence's earlier runs leave.  When a portion has several runs the kernel runs twice:
// first for every run but the last the product of its decays and its state from zero go to `sums`, then every run
// folds the sums before it and writes its results.  (Computing the gates twice moves less memory than storing decays
// and input terms in fp32.)
// TMEM columns: 32 per (stream, buffer, gate), 256 in all.  Every wait is bounded.
#include "gated_scan.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

constexpr int SR_TOK = 32;
constexpr int SR_THREADS = 13 * 32;
constexpr int SR_WBOX = 128 * 128;               // 64 channels (128 bytes) of 128 gate rows
constexpr int SR_UBOX = SR_TOK * 128;            // 64 channels of a tile's tokens

template <int TAPS, bool SUMS>
__global__ void __launch_bounds__(SR_THREADS, 1)
scan_runs_kernel(const __grid_constant__ CUtensorMap tmW, const __grid_constant__ GatedScan p) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t w_full, u_full[2][2], t_full[2][2], done[2][2];
  __shared__ uint32_t tmem_base_s;
  __shared__ int s_abort;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kb = (p.part + 63) / 64;
  const int ctiles = (p.part + 127) / 128;
  const int blk = blockIdx.y / ctiles, ct = blockIdx.y % ctiles;
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t sW = base, sU = base + 2 * kb * SR_WBOX;                  // u: [stream][buffer][box]
  const uint32_t u_bytes = kb * SR_UBOX;
  int* status = p.status;

  // the two runs: sequence, first row, tokens, first run of the sequence
  auto load_run = [&](int s, int& seq, int& off, int& n, int& first) {
    const int i = 2 * blockIdx.x + s;
    n = 0;
    seq = off = first = 0;
    if (i >= p.n_runs) return;
    const int4 r = *reinterpret_cast<const int4*>(p.runs + 4 * i);
    seq = min(max(r.x, 0), p.num_seqs - 1);
    off = r.y;
    first = r.w;
    // no run follows the last one of a portion: its sums are not needed
    n = SUMS && off + r.z >= p.q_start[seq + 1] - p.q_start[seq] ? 0 : r.z;
  };

  if (threadIdx.x == 0) {
    s_abort = 0;
    mbar_init(smem_u32(&w_full), 1);
    for (int s = 0; s < 2; ++s)
      for (int b = 0; b < 2; ++b) {
        mbar_init(smem_u32(&u_full[s][b]), 2);               // producer warps
        mbar_init(smem_u32(&t_full[s][b]), 1);
        mbar_init(smem_u32(&done[s][b]), 4);                 // epilogue warps
      }
    fence_mbar_init();
    tma_prefetch_desc(&tmW);
  }
  if (warp == 12) {
    tmem_alloc(smem_u32(&tmem_base_s), 256);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = tmem_base_s;

  if (warp == 12) {
    if (elect_one()) {
      const uint32_t wb = smem_u32(&w_full);
      mbar_expect_tx(wb, (uint32_t)(2 * kb * SR_WBOX));
      for (int g = 0; g < 2; ++g)
        for (int x = 0; x < kb; ++x)
          tma_load_3d(sW + (g * kb + x) * SR_WBOX, &tmW, wb, 64 * x, ct * 128, g * p.blocks + blk);
      int tiles[2], most = 0;
      for (int s = 0; s < 2; ++s) {
        int seq, off, n, first;
        load_run(s, seq, off, n, first);
        tiles[s] = (n + SR_TOK - 1) / SR_TOK;
        most = max(most, tiles[s]);
      }
      const uint32_t idesc = umma_idesc(128, SR_TOK, 1, 1, 0, 0);
      const uint64_t dW = umma_desc_kmajor_sw128(sW), dU = umma_desc_kmajor_sw128(sU);
      const uint64_t wbox = SR_WBOX >> 4, ubox = SR_UBOX >> 4;
      const int steps = p.part >> 4;
      mbar_wait(wb, 0, &s_abort, status, ERR_WAIT_FULL);
      for (int it = 0; it < most; ++it)
        for (int s = 0; s < 2; ++s) {
          if (it >= tiles[s]) continue;
          const int b = it & 1;
          mbar_wait(smem_u32(&u_full[s][b]), (it >> 1) & 1, &s_abort, status, ERR_WAIT_FULL);
          tc_fence_after_sync();
          const uint64_t u0 = dU + (uint64_t)((s * 2 + b) * kb) * ubox;
          for (int g = 0; g < 2; ++g) {
            const uint64_t w0 = dW + (uint64_t)(g * kb) * wbox;
            const uint32_t d = tmem + ((s * 2 + b) * 2 + g) * SR_TOK;
            for (int k = 0; k < steps; ++k) {
              const uint64_t in = (uint64_t)((k & 3) * 2);               // 16 channels = 32 bytes of a row
              mma_f16_ss(d, w0 + (uint64_t)(k >> 2) * wbox + in, u0 + (uint64_t)(k >> 2) * ubox + in, idesc, k == 0 ? 0u : 1u);
            }
          }
          tc_commit(smem_u32(&t_full[s][b]));
        }
    }
  } else if (warp >= 8) {
    // ------------------------------------------------------------------ convolution
    const int s = (warp - 8) >> 1, tid = threadIdx.x - 256 - s * 64;
    int seq, off, n, first;
    load_run(s, seq, off, n, first);
    const int tiles = (n + SR_TOK - 1) / SR_TOK;
    const int vecs = p.part / 8, groups = 64 / vecs;         // vecs <= 32: at least two groups
    const int v = tid % vecs, grp = tid / vecs;
    const int per = (SR_TOK + groups - 1) / groups;
    const int tk0 = grp * per, tk1 = grp < groups ? min(SR_TOK, tk0 + per) : tk0;
    const int c = blk * p.part + v * 8;
    const int taps = TAPS > 0 ? TAPS : p.taps, h = taps - 1;
    int sin = 0, sout = -1, q0 = 0, ctx = 0;
    if (n > 0) {
      scan_rows(p, seq, sin, sout);
      q0 = p.q_start[seq];
      ctx = p.context[seq];
    }
    const bf16* x = static_cast<const bf16*>(p.proj) + (long)q0 * p.ldp + p.C + c;
    const bf16* hist = static_cast<const bf16*>(p.hist) + ((long)sin * h + h) * p.C + c;
    auto raw_x = [&](int b) {                                // row b of the portion; negative: history
      if (b >= 0) return *reinterpret_cast<const uint4*>(x + (long)b * p.ldp);
      if (ctx + b >= 0) return *reinterpret_cast<const uint4*>(hist + (long)b * p.C);
      return make_uint4(0u, 0u, 0u, 0u);
    };
    float w[TAPS > 0 ? TAPS : 1][8], bias[8];
    load8<float>(p.conv_b + c, bias);
    if (TAPS > 0) {
#pragma unroll
      for (int j = 0; j < TAPS; ++j) load8<float>(p.conv + (long)j * p.C + c, w[j]);
    }
    for (int it = 0; it < tiles; ++it) {
      const int b = it & 1, t0 = it * SR_TOK, nt = min(SR_TOK, n - t0);
      mbar_wait(smem_u32(&done[s][b]), ((it >> 1) & 1) ^ 1, &s_abort, status, ERR_WAIT_EMPTY);
      const uint32_t dst = sU + (s * 2 + b) * u_bytes + (v >> 3) * SR_UBOX;
      auto put = [&](int tk, const float (&o)[8]) {
        st_shared_v4(dst + tk * 128 + (((v & 7) ^ (tk & 7)) << 4),
                     make_uint4(pack_bf16(o[0], o[1]), pack_bf16(o[2], o[3]), pack_bf16(o[4], o[5]), pack_bf16(o[6], o[7])));
      };
      if (TAPS > 0) {
        constexpr int H = TAPS > 1 ? TAPS - 1 : 1, RUN = 8;
        uint4 win[H];
#pragma unroll
        for (int m = 0; m < TAPS - 1; ++m)
          win[m] = tk0 < min(tk1, nt) ? raw_x(off + t0 + tk0 - (TAPS - 1) + m) : make_uint4(0u, 0u, 0u, 0u);
        for (int r0 = tk0; r0 < tk1; r0 += RUN) {
          uint4 raw[RUN];                                    // loads of the run in flight together
#pragma unroll
          for (int i = 0; i < RUN; ++i)
            raw[i] = r0 + i < min(tk1, nt) ? *reinterpret_cast<const uint4*>(x + (long)(off + t0 + r0 + i) * p.ldp)
                                           : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
          for (int i = 0; i < RUN; ++i) {
            float o[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) o[e] = bias[e];
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {
              float f[8];
              load8<bf16>(reinterpret_cast<const bf16*>(j < TAPS - 1 ? &win[j < H ? j : 0] : &raw[i]), f);
#pragma unroll
              for (int e = 0; e < 8; ++e) o[e] = fmaf(w[j][e], f[e], o[e]);
            }
#pragma unroll
            for (int m = 0; m + 1 < TAPS - 1; ++m) win[m] = win[m + 1];
            if (TAPS > 1) win[H - 1] = raw[i];
            if (r0 + i < tk1) put(r0 + i, o);                // past the run's end: finite values nobody uses
          }
        }
      } else {
        for (int tk = tk0; tk < tk1; ++tk) {
          float o[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) o[e] = bias[e];
          for (int j = 0; j < taps && tk < nt; ++j) {
            float f[8], wj[8];
            const uint4 q = raw_x(off + t0 + tk - h + j);
            load8<bf16>(reinterpret_cast<const bf16*>(&q), f);
            load8<float>(p.conv + (long)j * p.C + c, wj);
#pragma unroll
            for (int e = 0; e < 8; ++e) o[e] = fmaf(wj[e], f[e], o[e]);
          }
          put(tk, o);
        }
      }
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&u_full[s][b]));
    }
  } else {
    // ------------------------------------------------------------------ gates, scan, output
    const int s = warp >> 2, q = warp & 3;
    int seq, off, n, first;
    load_run(s, seq, off, n, first);
    const int tiles = (n + SR_TOK - 1) / SR_TOK;
    const int cl = ct * 128 + q * 32 + lane;                 // channel within the part
    const bool ok = cl < p.part;
    const int cs = ok ? cl : p.part - 1, c = blk * p.part + cs;
    int sin = 0, sout = -1, q0 = 0, ctx = 0, q1 = 0;
    float S = 0.f, la_sum = 0.f;
    const int run = 2 * blockIdx.x + s;
    if (n > 0) {
      scan_rows(p, seq, sin, sout);
      q0 = p.q_start[seq];
      q1 = p.q_start[seq + 1];
      ctx = p.context[seq];
      if (!SUMS) {
        if (ctx > 0) S = p.state[(long)sin * p.C + c];
        for (int i = first; i < run; ++i) S = fmaf(p.sums[(long)i * 2 * p.C + c], S, p.sums[((long)i * 2 + 1) * p.C + c]);
      }
    }
    const float br = p.gates_b[c], bi = p.gates_b[p.C + c], decay2 = p.decay[c] * GS_LOG2E;
    const bf16* y = static_cast<const bf16*>(p.proj) + (long)(q0 + off) * p.ldp + c;
    bf16* out = static_cast<bf16*>(p.out) + (long)(q0 + off) * p.C + c;
    const uint32_t u_col = (uint32_t)(cs >> 6) * SR_UBOX + (cs & 7) * 2;
    const int u_vec = (cs & 63) >> 3;
    for (int it = 0; it < tiles; ++it) {
      const int b = it & 1, t0 = it * SR_TOK, nt = min(SR_TOK, n - t0);
      mbar_wait(smem_u32(&t_full[s][b]), (it >> 1) & 1, &s_abort, status, ERR_WAIT_TMEM_FULL);
      tc_fence_after_sync();
      const uint32_t ta = tmem + ((uint32_t)(q * 32) << 16) + (s * 2 + b) * 2 * SR_TOK;
      const uint32_t ua = sU + (s * 2 + b) * u_bytes + u_col;
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        uint32_t zr[16], zi[16];
        tmem_ld_32x16(ta + half * 16, zr);
        tmem_ld_32x16(ta + SR_TOK + half * 16, zi);
        bf16 yv[16];
        if (!SUMS) {
#pragma unroll
          for (int e = 0; e < 16; ++e) {
            const int tk = half * 16 + e;
            yv[e] = tk < nt ? y[(long)(t0 + tk) * p.ldp] : __float2bfloat16(0.f);
          }
        }
        tmem_wait_ld();
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          const int tk = half * 16 + e;
          unsigned short ur;
          asm volatile("ld.shared.u16 %0, [%1];" : "=h"(ur) : "r"(ua + tk * 128 + ((u_vec ^ (tk & 7)) << 4)));
          const float u = __bfloat162float(__ushort_as_bfloat16(ur));
          float la2, a, add;
          gate_step(__uint_as_float(zr[e]) + br, __uint_as_float(zi[e]) + bi, u, decay2, la2, a, add);
          if (tk < nt) {
            S = fmaf(a, S, add);
            if (SUMS) la_sum += la2;
            else if (ok) out[(long)(t0 + tk) * p.C] = __float2bfloat16(S * gelu_short(__bfloat162float(yv[e])));
          }
        }
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&done[s][b]));
    }
    if (n > 0 && ok) {
      if (SUMS) {
        p.sums[(long)run * 2 * p.C + c] = gs_ex2(la_sum);
        p.sums[((long)run * 2 + 1) * p.C + c] = S;
      } else if (sout >= 0 && q0 + off + n == q1) {
        p.state[(long)sout * p.C + c] = S;
        const int h = p.taps - 1;
        const bf16* x = static_cast<const bf16*>(p.proj) + (long)q0 * p.ldp + p.C + c;
        bf16* hist = static_cast<bf16*>(p.hist);
        for (int m = 0; m < h; ++m) {
          const int b = off + n - h + m;                     // row of the portion; negative: history
          bf16 v = __float2bfloat16(0.f);
          if (b >= 0) v = x[(long)b * p.ldp];
          else if (ctx + b >= 0) v = hist[((long)sin * h + h + b) * p.C + c];
          hist[((long)sout * h + m) * p.C + c] = v;
        }
      }
    }
  }

  tc_fence_before_sync();
  __syncthreads();
  if (s_abort) {
    // a wait ran out: give copies and products in flight time to finish before their memory goes
    const unsigned long long t0 = globaltimer_ns();
    while (globaltimer_ns() - t0 < 200000ull) {
    }
  }
  if (warp == 12) tmem_dealloc(tmem, 256);
}

template <int TAPS>
static int launch_runs(const CUtensorMap& tw, const GatedScan& p, int smem, cudaStream_t st) {
  static unsigned long long prep[2] = {0, 0};
  dim3 grid((p.n_runs + 1) / 2, p.blocks * ((p.part + 127) / 128));
  if (p.sums) {
    if (int e = ensure_dynamic_smem((const void*)scan_runs_kernel<TAPS, true>, 226 * 1024, prep[0])) return e;
    scan_runs_kernel<TAPS, true><<<grid, SR_THREADS, smem, st>>>(tw, p);
    if (int e = (int)cudaGetLastError()) return e;
  }
  if (int e = ensure_dynamic_smem((const void*)scan_runs_kernel<TAPS, false>, 226 * 1024, prep[1])) return e;
  scan_runs_kernel<TAPS, false><<<grid, SR_THREADS, smem, st>>>(tw, p);
  return (int)cudaGetLastError();
}

}  // namespace omni

using namespace omni;

// sums == nullptr: every portion is one run.
extern "C" int omni_scan_runs(const GatedScan* args, void* stream) {
  const GatedScan& p = *args;
  if (p.n_runs <= 0) return RC_OK;
  if (!scan_args_ok(p) || !p.runs || p.part > 256 || p.blocks * 2 > 65535) return RC_BAD_ARG;
  CUtensorMap tw;
  const int rc = make_tmap_3d(&tw, p.gates, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, p.part, p.part, 2 * p.blocks, (uint64_t)p.part * 2,
                              (uint64_t)p.part * p.part * 2, 64, 128);
  if (rc) return rc;
  const int kb = (p.part + 63) / 64;
  const int smem = 2 * kb * SR_WBOX + 4 * kb * SR_UBOX + 1024;
  cudaStream_t st = (cudaStream_t)stream;
  switch (p.taps) {
    case 1: return launch_runs<1>(tw, p, smem, st);
    case 2: return launch_runs<2>(tw, p, smem, st);
    case 3: return launch_runs<3>(tw, p, smem, st);
    case 4: return launch_runs<4>(tw, p, smem, st);
    default: return launch_runs<0>(tw, p, smem, st);
  }
}
