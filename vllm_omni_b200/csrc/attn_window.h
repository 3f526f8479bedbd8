// Operands of the windowed paged attention family (attn_window.cu, attn_window_sm100.cu).
//
// Position i of a sequence attends to j <= i with i - j < window or j < keep_first.  The score is
// (q . k) * scale, optionally bounded to cap * tanh(score / cap), minus r1[h] * ln(1 + r2[h] * (i - j)).
// `sink[h]` joins the softmax denominator as exp(sink[h]).  `gate` multiplies head h's result by
// sigmoid(gate[row, h]), or channel c of it by sigmoid(gate[row, h, c]).
//
// With maps = 2 (differential attention) every query and key head has two maps that share the head's values; with a1, a2
// the maps' results, head h's result is u / sqrt(<u^2> + out_eps) * out_mul for u = a1 - lam a2, then the gate.  Query
// heads are ordered (KV head, map, head of the group), a cached key holds its two maps side by side.  Heads are padded to dp (query / key) and vp (value) channels, multiples of 16
// with zero padding.
#pragma once
#include <cuda_runtime.h>

namespace omni {

struct WinAttn {
  const void* q; long q_rs;            // [T, maps * H, dp], row pitch in elements
  const void* k_cache; const void* v_cache;     // [num_blocks, block_size, G, maps * dp | vp]
  const int* block_tables; int bt_stride;       // [S, bt_stride]
  const int* q_start; const int* context;       // [S + 1], [S]
  const int* row_seq;                  // [T] (row-per-block kernel)
  const int* seq_list; int n_list;     // decode kernel: sequences with exactly one row
  const int* items; int n_items;       // prefill kernel: (sequence, first token of the block) pairs
  int block_tokens;                    // prefill kernel: tokens per block, one or two tiles' worth
  void* out; long o_rs;                // [T, H, vp]
  const void* gate; long g_rs;         // logits at row * g_rs + h * g_hs + c * g_cs (g_cs 0: one per head), or nullptr
  const float* r1; const float* r2;    // [H] or nullptr
  const float* sink;                   // [H] or nullptr
  float scale, cap;                    // cap <= 0: no bound
  int bounded;                         // the cap may serve as softmax reference (see attn_window_sm100.cu)
  int window, keep_first;              // window <= 0: unbounded
  int T, H, G, dp, vp, num_seqs, num_blocks, block_size;
  int splits; float* part_o; float* part_ml;    // decode: shares of the visible keys, merged by a second kernel
  int* status;
  long k_ts, v_ts;                     // elements from one cached token to the next in k_cache / v_cache
  // Keys in two parts (prefill kernel): the first dp_u channels of a key are the head's own (k_cache), the other
  // dp - dp_u are one vector per token shared by all heads (k_shared, pitch ks_ts).  dp_u = dp: one part.
  const void* k_shared; long ks_ts; int dp_u;
  // Keys back to back instead of in pages (prefill kernel): key j of sequence s is row key_start[s] + j of key_rows
  // (key_start is negative where the first keys, which a window leaves out, are not there).
  const int* key_start; long key_rows;
  long g_hs; int g_cs;
  int maps;                            // 1 or 2
  float lam, out_mul, out_eps;         // maps = 2
  int vdim;                            // maps = 2: real channels of a value head
};

}  // namespace omni
