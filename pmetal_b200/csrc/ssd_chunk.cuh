// Blockwise recurrence (csrc/ssd_chunk.cu), shared by the state-space layers, the linear attention layers and the gated ones
// (gated_linear.cu). The kinds differ in their decays:
//   kSsdPlain   one rate per head and a step size per token (the default: steps of 1); with lo > 0 B and C are sums of two terms
//   kSsdMemory  a log decay and a weight per token and head, and a normaliser: the sum of the decayed, weighted B
//   kSsdChannel a decay per token and state row. B and C (two terms) already hold the decays to the block's end and from its
//               start, the scores within blocks come from the caller
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

namespace pm {

enum : int { kSsdPlain = 0, kSsdMemory = 1, kSsdChannel = 2 };

struct SsdParams {
  const __nv_bfloat16* act;   // [tokens, ld]: B of group g at column b0 + g NB, C at c0 + g NB
  const __nv_bfloat16* x;     // [tokens, ldx]: x of head h at column h P; null: act
  const float* dt;            // [tokens, H] step sizes (kSsdMemory: weights), null: 1 for every token
  const float* a_log;         // [H] decay exp(-exp(a_log) dt), or
  const float* log2_decay;    // [H] decay 2^(log2_decay dt) (a_log is null)
  const float* dskip;         // [H] weight of x in y, null: 0
  const float* ldec;          // kSsdMemory: [tokens, H] log2 decays of the tokens
  const float* mrun;          // kSsdMemory: [tokens, H] running maximum m of the logarithms
  float* nstate;              // kSsdMemory: [slots][H][N] normalisers
  float* seg_n;               // kSsdMemory: work buffer [seq][max_seg][H][N]
  float* den;                 // kSsdMemory: [tokens, H] max(|n . c|, exp(-m)) + den_eps
  const __nv_bfloat16* score; // kSsdChannel: [tokens, H, 128] scores against the block's 64 tokens, second terms behind the first
  const float* block_decay;   // kSsdChannel: [c_start / 64 + sequence + block][H][NB]
  const int* c_start;         // kSsdChannel: first token of every sequence, counted over these sequences alone
  float yscale, den_eps;      // kSsdMemory: factor of C
  float* state;               // [slots][H][N][P4]
  const int* slots;
  const int* q_start;
  const int* q_lens;
  const int* seq_lens;
  __nv_bfloat16* y;           // [tokens, H P]
  // work buffers: seg_state [seq][max_seg][H][N][P4] (0: the state a sequence starts from, k > 0: what segment k - 1 adds to
  // it), seg_decay [seq][max_seg][H] (decay of the state over segment k; kSsdChannel: [..][H][N])
  float* seg_state;
  float* seg_decay;
  int H, P, N, G, P4;
  int ld, b0, c0;
  int ldx;
  int kind;
  int NB;                     // columns of a group, 0: N
  int lo;                     // > 0: B and C are sums of two bf16 terms, the second ones lo columns further on
  // filled by the launcher
  int n_seg, seg_chunks;      // segments of the longest portion, blocks per segment
  int n16;                    // N rounded up to 16
  int aligned, aligned_x;     // rows of B and C, rows of x can be copied 16 bytes at a time
};

constexpr int kSsdMaxState = 256;      // largest N

// max_q: the longest of q_lens; max_seg: segments that the work buffers have room for. Returns a CUDA error code or -1.
int ssd_chunk_launch(SsdParams p, int n_seq, int max_q, int max_seg, cudaStream_t st);

}  // namespace pm
