// Gated linear recurrence of prompt portions on tcgen05 tensor cores (gated_scan.cuh says what is computed; the
// convolution's rows come from gated_scan.cu).
//
// A portion is cut into runs of consecutive tokens.  One block owns 128 channels of one part and four runs (streams),
// and keeps the gate weights of its channels in shared memory; a run is walked in tiles of 64 tokens.  The gates are
// computed transposed, D[channel, token] = W[channel, k] u[token, k]^T, so that a thread of the epilogue owns one
// channel (a TMEM lane) and meets its tokens in order: the scan is a register recurrence.
//   warps 0-15   epilogue, four warps per stream: both gates from tensor memory, decay, input term, scan; output
//   warp 16      TMA: gate weights, then tiles of u in turn for every stream
//   warp 17      MMA issue in the same order
// The epilogue is bound by its exponentials, reciprocals and roots; four streams hide each other's waits.
// A run starts from what its sequence's earlier runs leave.  When a portion has several runs the kernel runs twice:
// first for every run but the last the product of its decays and its state from zero go to `sums`, then every run
// folds the sums before it and writes its results.  (Computing the gates twice moves less memory than storing decays
// and input terms in fp32.)
// TMEM columns: 64 per (stream, gate), 512 in all.  Every wait is bounded.
#include "gated_scan.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

constexpr int SR_STREAMS = 4, SR_TOK = 64, SR_MAX_BUF = 8;
constexpr int SR_THREADS = (4 * SR_STREAMS + 2) * 32;
constexpr int SR_WBOX = 128 * 128;               // 64 channels (128 bytes) of 128 gate rows
constexpr int SR_UBOX = SR_TOK * 128;            // 64 channels of a tile's tokens

template <bool SUMS>
__global__ void __launch_bounds__(SR_THREADS, 1)
scan_runs_kernel(const __grid_constant__ CUtensorMap tmW, const __grid_constant__ CUtensorMap tmU,
                 const __grid_constant__ GatedScan p, const int n_buf) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t w_full, u_full[SR_MAX_BUF], u_empty[SR_MAX_BUF], t_full[SR_STREAMS], t_empty[SR_STREAMS];
  __shared__ uint32_t tmem_base_s;
  __shared__ int s_abort;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kb = (p.part + 63) / 64;
  const int ctiles = (p.part + 127) / 128;
  const int blk = blockIdx.x / ctiles, ct = blockIdx.x % ctiles;
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t sW = base, sU = base + 2 * kb * SR_WBOX;                  // u: [buffer][box]
  int* status = p.status;

  // the runs of the block: sequence, first row, tokens, first run of the sequence
  auto load_run = [&](int s, int& seq, int& off, int& n, int& first) {
    const int i = SR_STREAMS * blockIdx.y + s;
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
    for (int i = 0; i < n_buf; ++i) {
      mbar_init(smem_u32(&u_full[i]), 1);
      mbar_init(smem_u32(&u_empty[i]), 1);
    }
    for (int s = 0; s < SR_STREAMS; ++s) {
      mbar_init(smem_u32(&t_full[s]), 1);
      mbar_init(smem_u32(&t_empty[s]), 4);                   // epilogue warps
    }
    fence_mbar_init();
    tma_prefetch_desc(&tmW);
    tma_prefetch_desc(&tmU);
  }
  if (warp == 17) {
    tmem_alloc(smem_u32(&tmem_base_s), 512);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = tmem_base_s;

  if (warp >= 16) {
    if (elect_one()) {
      int tiles[SR_STREAMS], row0[SR_STREAMS], most = 0;
      for (int s = 0; s < SR_STREAMS; ++s) {
        int seq, off, n, first;
        load_run(s, seq, off, n, first);
        tiles[s] = (n + SR_TOK - 1) / SR_TOK;
        row0[s] = n > 0 ? p.q_start[seq] + off : 0;
        most = max(most, tiles[s]);
      }
      const uint32_t wb = smem_u32(&w_full);
      int i = 0;                                             // tile count: buffer i % n_buf
      if (warp == 16) {
        mbar_expect_tx(wb, (uint32_t)(2 * kb * SR_WBOX));
        for (int g = 0; g < 2; ++g)
          for (int x = 0; x < kb; ++x)
            tma_load_3d(sW + (g * kb + x) * SR_WBOX, &tmW, wb, 64 * x, ct * 128, g * p.blocks + blk);
        for (int it = 0; it < most; ++it)
          for (int s = 0; s < SR_STREAMS; ++s) {
            if (it >= tiles[s]) continue;
            const int b = i % n_buf;
            mbar_wait(smem_u32(&u_empty[b]), ((i / n_buf) & 1) ^ 1, &s_abort, status, ERR_WAIT_EMPTY);
            mbar_expect_tx(smem_u32(&u_full[b]), (uint32_t)(kb * SR_UBOX));
            for (int x = 0; x < kb; ++x)
              tma_load_3d(sU + (b * kb + x) * SR_UBOX, &tmU, smem_u32(&u_full[b]), 64 * x, row0[s] + it * SR_TOK, blk);
            ++i;
          }
      } else {
        const uint32_t idesc = umma_idesc(128, SR_TOK, 1, 1, 0, 0);
        const uint64_t dW = umma_desc_kmajor_sw128(sW), dU = umma_desc_kmajor_sw128(sU);
        const uint64_t wbox = SR_WBOX >> 4, ubox = SR_UBOX >> 4;
        const int steps = p.part >> 4;
        mbar_wait(wb, 0, &s_abort, status, ERR_WAIT_FULL);
        for (int it = 0; it < most; ++it)
          for (int s = 0; s < SR_STREAMS; ++s) {
            if (it >= tiles[s]) continue;
            const int b = i % n_buf;
            mbar_wait(smem_u32(&t_empty[s]), (it & 1) ^ 1, &s_abort, status, ERR_WAIT_TMEM_EMPTY);
            mbar_wait(smem_u32(&u_full[b]), (i / n_buf) & 1, &s_abort, status, ERR_WAIT_FULL);
            tc_fence_after_sync();
            const uint64_t u0 = dU + (uint64_t)(b * kb) * ubox;
            for (int g = 0; g < 2; ++g) {
              const uint64_t w0 = dW + (uint64_t)(g * kb) * wbox;
              const uint32_t d = tmem + (s * 2 + g) * SR_TOK;
              for (int k = 0; k < steps; ++k) {
                const uint64_t in = (uint64_t)((k & 3) * 2);             // 16 channels = 32 bytes of a row
                mma_f16_ss(d, w0 + (uint64_t)(k >> 2) * wbox + in, u0 + (uint64_t)(k >> 2) * ubox + in, idesc, k == 0 ? 0u : 1u);
              }
            }
            tc_commit(smem_u32(&u_empty[b]));
            tc_commit(smem_u32(&t_full[s]));
            ++i;
          }
      }
    }
  } else {
    // ------------------------------------------------------------------ gates, scan, output
    const int s = warp >> 2, q = warp & 3;
    int seq, off, n, first;
    load_run(s, seq, off, n, first);
    const int tiles = (n + SR_TOK - 1) / SR_TOK;
    const int cl = ct * 128 + q * 32 + lane;                 // channel within the part
    const bool ok = cl < p.part;
    const int c = blk * p.part + (ok ? cl : p.part - 1);
    int sout = -1, q0 = 0, q1 = 0;
    float S = 0.f, la_sum = 0.f;
    const int run = SR_STREAMS * blockIdx.y + s;
    if (n > 0) {
      int sin;
      scan_rows(p, seq, sin, sout);
      q0 = p.q_start[seq];
      q1 = p.q_start[seq + 1];
      if (!SUMS) {
        if (p.context[seq] > 0) S = p.state[(long)sin * p.C + c];
#pragma unroll 8
        for (int i = first; i < run; ++i) S = fmaf(p.sums[(long)i * 2 * p.C + c], S, p.sums[((long)i * 2 + 1) * p.C + c]);
      }
    }
    const float br = p.gates_b[c], bi = p.gates_b[p.C + c], decay2 = p.decay[c] * GS_LOG2E;
    const bf16* y = static_cast<const bf16*>(p.proj) + (long)(q0 + off) * p.ldp + c;
    const bf16* u = static_cast<const bf16*>(p.u) + (long)(q0 + off) * p.C + c;
    bf16* out = static_cast<bf16*>(p.out) + (long)(q0 + off) * p.C + c;
    for (int it = 0; it < tiles; ++it) {
      const uint32_t ta = tmem + ((uint32_t)(q * 32) << 16) + s * 2 * SR_TOK;
#pragma unroll 1
      for (int k = 0; k < SR_TOK; k += 16) {
        const int t0 = it * SR_TOK + k, left = n - t0;       // tokens of this chunk that exist
        if (left <= 0 && k > 0) break;
        bf16 uv[16], yv[16];
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          uv[e] = e < left ? u[(long)(t0 + e) * p.C] : __float2bfloat16(0.f);
          if (!SUMS) yv[e] = e < left ? y[(long)(t0 + e) * p.ldp] : __float2bfloat16(0.f);
        }
        if (k == 0) {
          mbar_wait(smem_u32(&t_full[s]), it & 1, &s_abort, status, ERR_WAIT_TMEM_FULL);
          tc_fence_after_sync();
        }
        uint32_t zr[16], zi[16];
        tmem_ld_32x16(ta + k, zr);
        tmem_ld_32x16(ta + SR_TOK + k, zi);
        tmem_wait_ld();
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          float la2, a, add;
          gate_step(__uint_as_float(zr[e]) + br, __uint_as_float(zi[e]) + bi, __bfloat162float(uv[e]), decay2, la2, a, add);
          if (e < left) {
            S = fmaf(a, S, add);
            if (SUMS) la_sum += la2;
            else if (ok) out[(long)(t0 + e) * p.C] = __float2bfloat16(S * gelu_short(__bfloat162float(yv[e])));
          }
        }
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&t_empty[s]));
    }
    if (n > 0 && ok) {
      if (SUMS) {
        p.sums[(long)run * 2 * p.C + c] = gs_ex2(la_sum);
        p.sums[((long)run * 2 + 1) * p.C + c] = S;
      } else if (sout >= 0 && q0 + off + n == q1) {
        p.state[(long)sout * p.C + c] = S;
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
  if (warp == 17) tmem_dealloc(tmem, 512);
}

}  // namespace omni

using namespace omni;

// sums == nullptr: every portion is one run.
extern "C" int omni_scan_runs(const GatedScan* args, void* stream) {
  const GatedScan& p = *args;
  if (p.n_runs <= 0) return RC_OK;
  if (!scan_args_ok(p) || !p.runs || !p.u || p.part > 256 || (p.n_runs + SR_STREAMS - 1) / SR_STREAMS > 65535) return RC_BAD_ARG;
  CUtensorMap tw, tu;
  int rc = make_tmap_3d(&tw, p.gates, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, p.part, p.part, 2 * p.blocks, (uint64_t)p.part * 2,
                        (uint64_t)p.part * p.part * 2, 64, 128);
  // u as (channel of a part, row, part)
  if (!rc) rc = make_tmap_3d(&tu, p.u, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, p.part, p.T, p.blocks, (uint64_t)p.C * 2,
                             (uint64_t)p.part * 2, 64, SR_TOK);
  if (rc) return rc;
  const int kb = (p.part + 63) / 64, limit = 226 * 1024;
  int n_buf = (limit - 1024 - 2 * kb * SR_WBOX) / (kb * SR_UBOX);
  if (n_buf > SR_MAX_BUF) n_buf = SR_MAX_BUF;
  const int smem = 2 * kb * SR_WBOX + n_buf * kb * SR_UBOX + 1024;
  cudaStream_t st = (cudaStream_t)stream;
  dim3 grid(p.blocks * ((p.part + 127) / 128), (p.n_runs + SR_STREAMS - 1) / SR_STREAMS);
  static unsigned long long prep[2] = {0, 0};
  if (p.sums) {
    if (int e = ensure_dynamic_smem((const void*)scan_runs_kernel<true>, limit, prep[0])) return e;
    scan_runs_kernel<true><<<grid, SR_THREADS, smem, st>>>(tw, tu, p, n_buf);
    if (int e = (int)cudaGetLastError()) return e;
  }
  if (int e = ensure_dynamic_smem((const void*)scan_runs_kernel<false>, limit, prep[1])) return e;
  scan_runs_kernel<false><<<grid, SR_THREADS, smem, st>>>(tw, tu, p, n_buf);
  return (int)cudaGetLastError();
}
