// Blockwise recurrence with one decay per head (csrc/ssd_chunk.cu), shared by the state-space layers and the linear
// attention layers.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>

namespace pm {

struct SsdParams {
  const __nv_bfloat16* act;   // [tokens, ld]: x of head h at column h P, B of group g at b0 + g N, C at c0 + g N
  const float* dt;            // [tokens, H] step sizes, null: 1 for every token
  const float* a_log;         // [H] decay exp(-exp(a_log) dt), or
  const float* log2_decay;    // [H] decay 2^(log2_decay dt) (a_log is null)
  const float* dskip;         // [H] weight of x in y, null: 0
  float* state;               // [slots][H][N][P4]
  const int* slots;
  const int* q_start;
  const int* q_lens;
  const int* seq_lens;
  __nv_bfloat16* y;           // [tokens, H P]
  // work buffers: seg_state [seq][max_seg][H][N][P4] (0: the state a sequence starts from, k > 0: what segment k - 1 adds to
  // it), seg_decay [seq][max_seg][H] (decay of the state over segment k)
  float* seg_state;
  float* seg_decay;
  int H, P, N, G, P4;
  int ld, b0, c0;
  int lo;                     // > 0: B and C are sums of two bf16 terms, the second ones lo columns further on
  // filled by the launcher
  int n_seg, seg_chunks;      // segments of the longest portion, blocks per segment
  int n16;                    // N rounded up to 16
  int aligned;                // rows can be copied 16 bytes at a time
};

constexpr int kSsdMaxState = 256;      // largest N

// max_q: the longest of q_lens; max_seg: segments that the work buffers have room for. Returns a CUDA error code or -1.
int ssd_chunk_launch(SsdParams p, int n_seq, int max_q, int max_seg, cudaStream_t st);

}  // namespace pm
