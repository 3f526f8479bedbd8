// Gated linear recurrence of prompt portions on tcgen05 tensor cores (gated_scan.cuh says what is computed; the
// convolution's rows come from short_conv.cu).
//
// A portion is cut into runs of consecutive tokens.  One block owns 128 channels of one part and four runs (streams),
// and keeps the gate weights of its channels in shared memory; a run is walked in tiles of 32 tokens.  The gates are
// computed transposed, D[channel, token] = W[channel, k] u[token, k]^T, so that a thread of the epilogue owns one
// channel (a TMEM lane) and meets its tokens in order: the scan is a register recurrence.
//   warps 0-15   epilogue, four warps per stream: both gates from tensor memory, decay, input term, scan; the output
//                takes the place of the gelu branch's tile in shared memory and leaves in 16-byte stores
//   warp 16      TMA: gate weights, then tiles of u and of the gelu branch in turn for every stream
//   warp 17      MMA issue in the same order
// The epilogue is bound by instruction issue and its exponentials, reciprocals and roots: it reads its operands from
// shared memory at constant offsets (no address arithmetic), and four streams hide each other's waits.
// A run starts from what its sequence's earlier runs leave.  When a portion has several runs the kernel runs twice:
// first for every run but the last the product of its decays and its state from zero go to `sums`, then every run
// folds the sums before it and writes its results.  (Computing the gates twice moves less memory than storing decays
// and input terms in fp32.)
// TMEM columns: 32 per (stream, slot, gate), 512 in all.  Every wait is bounded.
#include <type_traits>

#include "gated_scan.cuh"

namespace omni {

typedef __nv_bfloat16 bf16;

constexpr int SR_STREAMS = 4, SR_TOK = 32, SR_SLOTS = 2;
constexpr int SR_THREADS = (4 * SR_STREAMS + 2) * 32;
constexpr int SR_WBOX = 128 * 128;               // 64 channels (128 bytes) of 128 gate rows
constexpr int SR_UBOX = SR_TOK * 128;            // 64 channels of a tile's tokens

__device__ __forceinline__ float sr_ld(uint32_t addr) {
  unsigned short v;
  asm volatile("ld.shared.u16 %0, [%1];" : "=h"(v) : "r"(addr));
  return __bfloat162float(__ushort_as_bfloat16(v));
}
__device__ __forceinline__ void sr_st(uint32_t addr, float x) {
  asm volatile("st.shared.u16 [%0], %1;" ::"r"(addr), "h"(__bfloat16_as_ushort(__float2bfloat16(x))) : "memory");
}

// n_slots: tiles of a stream in flight (1 where shared memory allows no more)
template <bool SUMS>
__global__ void __launch_bounds__(SR_THREADS, 1)
scan_runs_kernel(const __grid_constant__ CUtensorMap tmW, const __grid_constant__ CUtensorMap tmU,
                 const __grid_constant__ CUtensorMap tmY, const __grid_constant__ GatedScan p, const int n_slots) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ __align__(8) uint64_t w_full, full[SR_STREAMS][SR_SLOTS], t_full[SR_STREAMS][SR_SLOTS], done[SR_STREAMS][SR_SLOTS];
  __shared__ uint32_t tmem_base_s;
  __shared__ int s_abort;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int kb = (p.part + 63) / 64;
  const int ctiles = (p.part + 127) / 128;
  const int blk = blockIdx.x / ctiles, ct = blockIdx.x % ctiles;
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t sW = base, sT = base + 2 * kb * SR_WBOX;                  // tiles: [stream][slot]{u boxes, two y boxes}
  const uint32_t t_bytes = (kb + 2) * SR_UBOX;
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
    for (int s = 0; s < SR_STREAMS; ++s)
      for (int d = 0; d < SR_SLOTS; ++d) {
        mbar_init(smem_u32(&full[s][d]), 1);
        mbar_init(smem_u32(&t_full[s][d]), 1);
        mbar_init(smem_u32(&done[s][d]), 4);                 // epilogue warps
      }
    fence_mbar_init();
    tma_prefetch_desc(&tmW);
    tma_prefetch_desc(&tmU);
    tma_prefetch_desc(&tmY);
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
      if (warp == 16) {
        mbar_expect_tx(wb, (uint32_t)(2 * kb * SR_WBOX));
        for (int g = 0; g < 2; ++g)
          for (int x = 0; x < kb; ++x)
            tma_load_3d(sW + (g * kb + x) * SR_WBOX, &tmW, wb, 64 * x, ct * 128, g * p.blocks + blk);
        for (int it = 0; it < most; ++it)
          for (int s = 0; s < SR_STREAMS; ++s) {
            if (it >= tiles[s]) continue;
            const int d = it % n_slots;
            const uint32_t fb = smem_u32(&full[s][d]), dst = sT + (s * n_slots + d) * t_bytes;
            const int row = row0[s] + it * SR_TOK;
            mbar_wait(smem_u32(&done[s][d]), ((it / n_slots) & 1) ^ 1, &s_abort, status, ERR_WAIT_EMPTY);
            mbar_expect_tx(fb, SUMS ? (uint32_t)(kb * SR_UBOX) : t_bytes);
            for (int x = 0; x < kb; ++x) tma_load_3d(dst + x * SR_UBOX, &tmU, fb, 64 * x, row, blk);
            if (!SUMS)
              for (int x = 0; x < 2; ++x) tma_load_3d(dst + (kb + x) * SR_UBOX, &tmY, fb, ct * 128 + 64 * x, row, blk);
          }
      } else {
        const uint32_t idesc = umma_idesc(128, SR_TOK, 1, 1, 0, 0);
        const uint64_t dW = umma_desc_kmajor_sw128(sW), dT = umma_desc_kmajor_sw128(sT);
        const uint64_t wbox = SR_WBOX >> 4, ubox = SR_UBOX >> 4;
        const int steps = p.part >> 4;
        mbar_wait(wb, 0, &s_abort, status, ERR_WAIT_FULL);
        for (int it = 0; it < most; ++it)
          for (int s = 0; s < SR_STREAMS; ++s) {
            if (it >= tiles[s]) continue;
            const int d = it % n_slots;
            mbar_wait(smem_u32(&full[s][d]), (it / n_slots) & 1, &s_abort, status, ERR_WAIT_FULL);
            tc_fence_after_sync();
            const uint64_t u0 = dT + (uint64_t)((s * n_slots + d) * (t_bytes >> 4));
            for (int g = 0; g < 2; ++g) {
              const uint64_t w0 = dW + (uint64_t)(g * kb) * wbox;
              const uint32_t acc = tmem + ((s * SR_SLOTS + d) * 2 + g) * SR_TOK;
              for (int k = 0; k < steps; ++k) {
                const uint64_t in = (uint64_t)((k & 3) * 2);             // 16 channels = 32 bytes of a row
                mma_f16_ss(acc, w0 + (uint64_t)(k >> 2) * wbox + in, u0 + (uint64_t)(k >> 2) * ubox + in, idesc, k == 0 ? 0u : 1u);
              }
            }
            tc_commit(smem_u32(&t_full[s][d]));
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
    const float nbr = -GS_LOG2E * p.gates_b[c], nbi = -GS_LOG2E * p.gates_b[p.C + c], decay2 = p.decay[c] * GS_LOG2E;
    // a thread's channel in a row of a swizzled box: 16-byte piece `vec` ^ (row & 7)
    const int vec = (q & 1) * 4 + (lane >> 3);
    const uint32_t lane_off = (uint32_t)(vec << 4) + (lane & 7) * 2;
    const uint32_t u_box = min((uint32_t)(2 * ct + (q >> 1)), (uint32_t)kb - 1) * SR_UBOX, y_box = (uint32_t)(kb + (q >> 1)) * SR_UBOX;
    // 16-byte pieces of the warp's 32 channels that a lane stores: piece of the row, rows lane / 4 + 8 i
    const int sv = (q & 1) * 4 + (lane & 3), sc = ct * 128 + q * 32 + (lane & 3) * 8;
    bf16* out = static_cast<bf16*>(p.out) + (long)(q0 + off) * p.C + blk * p.part + sc;

    auto walk = [&](auto whole, uint32_t ua, uint32_t ya, uint32_t ta, int nt) {
      constexpr bool WHOLE = decltype(whole)::value;         // all 32 tokens exist
#pragma unroll 1
      for (int k = 0; k < SR_TOK; k += 16) {
        if (!WHOLE && k >= nt) break;
        uint32_t zr[16], zi[16];
        tmem_ld_32x16(ta + k, zr);
        tmem_ld_32x16(ta + SR_TOK + k, zi);
        tmem_wait_ld();
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          const uint32_t at = (uint32_t)((e & 7) << 4), to = (uint32_t)(e * 128);
          float la2, a, add;
          gate_step(__uint_as_float(zr[e]), __uint_as_float(zi[e]), nbr, nbi, sr_ld((ua ^ at) + to), decay2, la2, a, add);
          if (WHOLE || k + e < nt) {
            S = fmaf(a, S, add);
            if (SUMS) la_sum += la2;
          }
          if (!SUMS) sr_st((ya ^ at) + to, S * gelu_short(sr_ld((ya ^ at) + to)));
        }
        ua += 16 * 128;
        ya += 16 * 128;
      }
    };
    for (int it = 0; it < tiles; ++it) {
      const int d = it % n_slots, t0 = it * SR_TOK, nt = min(SR_TOK, n - t0);
      const uint32_t tile = sT + (s * n_slots + d) * t_bytes;
      const uint32_t ph = (it / n_slots) & 1;
      mbar_wait(smem_u32(&full[s][d]), ph, &s_abort, status, ERR_WAIT_FULL);
      mbar_wait(smem_u32(&t_full[s][d]), ph, &s_abort, status, ERR_WAIT_TMEM_FULL);
      tc_fence_after_sync();
      const uint32_t ta = tmem + ((uint32_t)(q * 32) << 16) + (s * SR_SLOTS + d) * 2 * SR_TOK;
      if (nt == SR_TOK) walk(std::true_type{}, tile + u_box + lane_off, tile + y_box + lane_off, ta, nt);
      else walk(std::false_type{}, tile + u_box + lane_off, tile + y_box + lane_off, ta, nt);
      if (!SUMS) {
        __syncwarp();
#pragma unroll
        for (int i = 0; i < SR_TOK / 8; ++i) {
          const int tk = i * 8 + (lane >> 2);
          const uint4 v = ld_shared_v4(tile + y_box + tk * 128 + ((sv ^ (tk & 7)) << 4));
          if (tk < nt && sc < p.part) *reinterpret_cast<uint4*>(out + (long)(t0 + tk) * p.C) = v;
        }
        fence_proxy_async_smem();
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(smem_u32(&done[s][d]));
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
  CUtensorMap tw, tu, ty;
  int rc = make_tmap_3d(&tw, p.gates, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, p.part, p.part, 2 * p.blocks, (uint64_t)p.part * 2,
                        (uint64_t)p.part * p.part * 2, 64, 128);
  // u and the gelu branch as (channel of a part, row, part)
  if (!rc) rc = make_tmap_3d(&tu, p.u, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, p.part, p.T, p.blocks, (uint64_t)p.C * 2,
                             (uint64_t)p.part * 2, 64, SR_TOK);
  if (!rc) rc = make_tmap_3d(&ty, p.proj, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, p.part, p.T, p.blocks, (uint64_t)p.ldp * 2,
                             (uint64_t)p.part * 2, 64, SR_TOK);
  if (rc) return rc;
  const int kb = (p.part + 63) / 64, limit = 226 * 1024;
  const int tiles = SR_STREAMS * (kb + 2) * SR_UBOX;                        // one slot of every stream
  const int n_slots = 2 * kb * SR_WBOX + 2 * tiles + 1024 <= limit ? 2 : 1;
  const int smem = 2 * kb * SR_WBOX + n_slots * tiles + 1024;
  cudaStream_t st = (cudaStream_t)stream;
  dim3 grid(p.blocks * ((p.part + 127) / 128), (p.n_runs + SR_STREAMS - 1) / SR_STREAMS);
  static unsigned long long prep[2] = {0, 0};
  if (p.sums) {
    if (int e = ensure_dynamic_smem((const void*)scan_runs_kernel<true>, limit, prep[0])) return e;
    scan_runs_kernel<true><<<grid, SR_THREADS, smem, st>>>(tw, tu, ty, p, n_slots);
    if (int e = (int)cudaGetLastError()) return e;
  }
  if (int e = ensure_dynamic_smem((const void*)scan_runs_kernel<false>, limit, prep[1])) return e;
  scan_runs_kernel<false><<<grid, SR_THREADS, smem, st>>>(tw, tu, ty, p, n_slots);
  return (int)cudaGetLastError();
}
