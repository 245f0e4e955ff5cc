// C interface of libpmetal_b200.so: every launcher of the sm_100a kernel library.
//
// All functions take raw device pointers and a CUDA stream, allocate nothing unless their comment says so, and return
// 0 on success, a negative value for an argument or descriptor error, or the CUDA error code of the launch. `status`
// arguments point at a device int that a kernel sets when one of its bounded waits runs out (codes 101-109); the
// caller reads it after synchronising the stream. Pointers and the stream must belong to the current device.
// The no-allocation paged-attention entry point is declared in paged_attn_static.h.
//
// This file is written by pmetal_b200/build.py from the definitions in csrc/*.cu; every source includes it, so a
// declaration that drifts from its definition fails to compile.
#pragma once
#include <cuda_runtime.h>

#ifdef __cplusplus
extern "C" {
#endif

// ---------------------------------------------------------------- attention.cu
// q:[T,hq,128] k:[T,hkv,128] v:[T,hkv,128] with per-token strides; out:[T,hq,128]; lse:[hq,T]
int pm_attn_fwd(const void* q, long long q_stride, const void* k, long long k_stride, const void* v, long long
    v_stride, void* out, long long o_stride, float* lse, const int* seq_start, int T, int hq, int hkv, float scale,
    int window, cudaStream_t st);
// dq:[T,hq,128] dk,dv:[T,hkv,128] (strided). delta:[hq,T] = rowsum(dO*O) computed beforehand.
int pm_attn_bwd(const void* dout, const void* q, long long q_stride, const void* k, long long k_stride, const void*
    v, long long v_stride, long long o_stride, const float* lse, const float* delta, void* dq, long long dq_stride,
    void* dk, long long dk_stride, void* dv, long long dv_stride, const int* seq_start, int T, int hq, int hkv,
    float scale, int window, cudaStream_t st);
int pm_paged_attn_ex(const void* q, const void* k_cache, const void* v_cache, void* out, const int* block_table,
    const int* seq_lens, const int* q_start, const int* q_lens, float* part_o, float* part_ml, int num_seqs, int
    max_blocks, int total_q, int max_q, int hq, int hkv, int n_split, float scale, int window, int sink, const
    float* k_scale, const float* v_scale, cudaStream_t st);
// 4-bit code-book cache: k_cache / v_cache hold two codes per byte [num_blocks, 64, hkv, 64]; a cached value is
// lut16[code] * scale (scales as for the int8 cache). lut16: 16 floats on the host. The query and the output live in
// whatever basis the cached vectors were quantised in (the caller rotates the query and un-rotates the output).
int pm_paged_attn_q4(const void* q, const void* k_cache, const void* v_cache, void* out, const int* block_table,
    const int* seq_lens, const int* q_start, const int* q_lens, float* part_o, float* part_ml, int num_seqs, int
    max_blocks, int total_q, int max_q, int hq, int hkv, int n_split, float scale, int window, int sink, const
    float* k_scale, const float* v_scale, const float* lut16, cudaStream_t st);
int pm_paged_attn(const void* q, const void* k_cache, const void* v_cache, void* out, const int* block_table, const
    int* seq_lens, const int* q_start, const int* q_lens, float* part_o, float* part_ml, int num_seqs, int
    max_blocks, int total_q, int max_q, int hq, int hkv, int n_split, float scale, int window, cudaStream_t st);
int pm_kv_append_q8(const void* k, long long k_stride, const void* v, long long v_stride, void* k_cache, void*
    v_cache, float* k_scale, float* v_scale, const long long* slots, int n_tokens, int hkv, cudaStream_t st);
// sign: 128 floats (+-1) on the device; thr: 15 ascending thresholds on the device.
int pm_kv_append_tq4(const void* k, long long k_stride, const void* v, long long v_stride, void* k_cache, void*
    v_cache, float* k_scale, float* v_scale, const long long* slots, const float* sign, const float* thr, int
    n_tokens, int hkv, cudaStream_t st);
// x, y: [rows / heads, heads, 128] bf16 with token strides x_stride / y_stride (elements); inverse 0: y = H (x sign) / sqrt(d),
// inverse 1: y = (H x) / sqrt(d) * sign.
int pm_tq_rotate(const void* x, long long x_stride, const float* sign, void* y, long long y_stride, long long
    tokens, int heads, int inverse, cudaStream_t st);
int pm_kv_append(const void* k, long long k_stride, const void* v, long long v_stride, void* k_cache, void*
    v_cache, const long long* slots, int n_tokens, int hkv, cudaStream_t st);
int pm_paged_attn_static_max_rows(void);
const char* pm_paged_attn_static_strerror(int code);

// ---------------------------------------------------------------- attention_tc.cu
int pm_attn_fwd_tc_rect(const void* q, long long q_stride, const void* k, long long k_stride, const void* v, long
    long v_stride, void* out, long long o_stride, float* lse, const int* seq_start, int T, int Tk, int shift, int
    hq, int hkv, float scale, int* status, cudaStream_t st);
// pm_attn_fwd_tc_rect with capped scores (softcap > 0: softcap tanh(score / softcap)), a sink per head (fp32 [hq], nullable:
// exp(sink) joins the softmax sum) and an output gate (bf16 [T, ldg], nullable: head h times the sigmoid of column h).
int pm_attn_fwd_tc_ex(const void* q, long long q_stride, const void* k, long long k_stride, const void* v, long
    long v_stride, void* out, long long o_stride, float* lse, const int* seq_start, int T, int Tk, int shift, int
    hq, int hkv, float scale, float softcap, const float* sink, const void* gate, long long ldg, int* status,
    cudaStream_t st);
// The same with sigmoid weights: key j counts for head h with the sigmoid of its score + wbias[h] (fp32 [hq]), the sum is not divided
// by anything and multiplied with out_scale.
int pm_attn_fwd_tc_sigmoid(const void* q, long long q_stride, const void* k, long long k_stride, const void* v,
    long long v_stride, void* out, long long o_stride, const int* seq_start, int T, int Tk, int shift, int hq, int
    hkv, float scale, const float* wbias, float out_scale, int* status, cudaStream_t st);
// Single-softmax-group variant of the same kernel (kept selectable for comparison measurements).
int pm_attn_fwd_tc_rect_v1(const void* q, long long q_stride, const void* k, long long k_stride, const void* v,
    long long v_stride, void* out, long long o_stride, float* lse, const int* seq_start, int T, int Tk, int shift,
    int hq, int hkv, float scale, int* status, cudaStream_t st);
int pm_attn_fwd_tc(const void* q, long long q_stride, const void* k, long long k_stride, const void* v, long long
    v_stride, void* out, long long o_stride, float* lse, const int* seq_start, int T, int hq, int hkv, float scale,
    int* status, cudaStream_t st);

// ---------------------------------------------------------------- attention_tc_bwd.cu
// dout, q: [T, hq*128] (token strides o_stride / q_stride); k, v: [T, hkv*128] (v may be a strided view).
// dq:[T,hq,128], dk:[T,hkv,128], dv:[T,hkv,128] (strided). lse, delta: [hq][T].
int pm_attn_bwd_tc(const void* dout, long long do_stride, const void* q, long long q_stride, const void* k, long
    long k_stride, const void* v, long long v_stride, const float* lse, const float* delta, void* dq, long long
    dq_stride, void* dk, long long dk_stride, void* dv, long long dv_stride, const int* seq_start, int T, int hq,
    int hkv, float scale, int* status, cudaStream_t st);

// ---------------------------------------------------------------- decode_mega.cu
// 1 when one launch can run the step: up to 16 rows, 1 / 2 / 4 query heads per kv head, reduction sizes that are
// multiples of 32, and the staged activations fit in shared memory.
int pm_decode_layers_supported(int M, int H, int hq, int hkv, int I);
// layers: device array of n_layers DmLayer records (10 pointers each). bar: 2 words, counters: M * hkv words, all zero
// at launch (a completed launch leaves the counters zero; the caller clears bar before every launch).
int pm_decode_layers(const void* layers, int n_layers, int M, int H, int hq, int hkv, int I, float eps, float
    scale, void* x, void* h, void* qkv, void* attn, void* act, float* part_o, float* part_ml, unsigned* counters,
    const float* cs, const float* sn, const int* block_table, const int* seq_lens, const long long* slots, int
    max_blocks, int n_split, unsigned* bar, int* status, unsigned long long* trace, cudaStream_t st);

// ---------------------------------------------------------------- dp_fused.cu
// ptr arrays hold `world` device addresses each (peer-mapped). shadows may be null.
int pm_dp_reduce_adamw(const unsigned long long* grads, const unsigned long long* params, const unsigned long long*
    shadows, const unsigned long long* pads, float* m, float* v, const float* lr_mult, const float* wd, const
    float* gnorm_sq, const float* hp, long long n, int rank, int world, float lr, float beta1, float beta2, float
    eps, int step, float grad_scale, float max_norm, double timeout_s, int ctas, int* status, cudaStream_t st);
int pm_dp_pad_words();

// ---------------------------------------------------------------- elementwise.cu
int pm_rmsnorm_fwd(const void* x, const void* res, const void* w, void* y, void* h_out, float* rstd, int T, int H,
    float eps, cudaStream_t st);
int pm_rmsnorm_bwd(const void* dy, const void* h, const void* w, const float* rstd, const void* dh_add, void* dx,
    float* dw, int T, int H, cudaStream_t st);
int pm_rope_table(const int* pos, float* cs, float* sn, int T, int half, float theta, float rope_scale,
    cudaStream_t st);
int pm_rope_table_freqs(const int* pos, const float* inv_freq, float* cs, float* sn, int T, int half, float mscale,
    cudaStream_t st);
int pm_qknorm_rope_fwd(const void* qkv, int ld, const void* qw, const void* kw, const float* cs, const float* sn,
    void* q_out, void* k_out, int T, int hq, int hkv, float eps, cudaStream_t st);
int pm_qknorm_rope_cache(const void* qkv, int ld, const void* qw, const void* kw, const float* cs, const float* sn,
    void* q_out, void* k_cache, void* v_cache, const long long* slots, int T, int hq, int hkv, float eps,
    cudaStream_t st);
int pm_qknorm_rope_bwd(const void* dq, const void* dk, const void* qkv, int ld, const void* qw, const void* kw,
    const float* cs, const float* sn, void* dqkv, int T, int hq, int hkv, float eps, cudaStream_t st);
int pm_swiglu_fwd(const void* gu, void* out, long long T, int I, cudaStream_t st);
int pm_swiglu_bwd(const void* dout, const void* gu, void* dgu, long long T, int I, cudaStream_t st);
// act(gate) * up for separate gate / up matrices (row strides in elements, multiples of 8); act: 0 SiLU, 1 GELU-tanh, 2 GELU.
int pm_glu_fwd(const void* gate, const void* up, long long ldg, long long ldu, void* out, long long T, int I, int
    act, cudaStream_t st);
int pm_glu_bwd(const void* dout, const void* gate, const void* up, long long ldg, long long ldu, void* dgate, void*
    dup, long long lddg, long long lddu, long long T, int I, int act, cudaStream_t st);
// row_loss (optional): per-row loss out. row_scale (optional): per-row gradient scale replacing *inv_n.
int pm_ce_fwd_bwd(void* logits, long long ldl, const long long* labels, float* loss_sum, const float* inv_n, float*
    row_loss, const float* row_scale, int n_rows, int V, long long ignore_index, int write_grad, cudaStream_t st);
// Cross entropy plus the z term z_coef * logsumexp(logits)^2 per valid row: z_sum receives the sum of the squared
// normalisers, and the gradient written over the logits is that of (cross entropy + z_coef * z) summed over rows.
int pm_ce_z_fwd_bwd(void* logits, long long ldl, const long long* labels, float* loss_sum, float* z_sum, const
    float* inv_n, int n_rows, int V, long long ignore_index, int write_grad, float z_coef, cudaStream_t st);
// The same with label smoothing (0 <= smooth < 1) and soft-capped logits (softcap > 0: cap * tanh(x / cap)).
int pm_ce_opt_fwd_bwd(void* logits, long long ldl, const long long* labels, float* loss_sum, float* z_sum, const
    float* inv_n, int n_rows, int V, long long ignore_index, int write_grad, float z_coef, float smooth, float
    softcap, cudaStream_t st);
int pm_sumsq(const float* x, long long n, float* out, cudaStream_t st);
int pm_adamw_flat(float* p, const float* g, float* m, float* v, void* shadow, const float* lr_mult, const float*
    wd, const float* gnorm_sq, const float* hp, long long n, float lr, float beta1, float beta2, float eps, int
    step, float grad_scale, float max_norm, cudaStream_t st);
int pm_attn_delta(const void* o, const void* dout, float* delta, int T, int H, cudaStream_t st);
int pm_f32_to_bf16(const float* in, void* out, long long n, cudaStream_t st);
int pm_dequant_4bit(const void* data, const float* absmax, const void* absmax_q, float am_scale, float am_offset,
    void* out, long long n, int block_size, int fp4, cudaStream_t st);

// ---------------------------------------------------------------- gated_linear.cu
// Channel gates token by token. q / v: head 0's first column in row 0 of rows ldu apart, z fp32 rows of H N logits ldz apart, bias
// and lower fp32 [H N]; state [slots][H][N][P4] fp32, read and written; y [tokens, H P]. Sequence i covers tokens q_start[i] ..
// + q_lens[i] - 1 and ends at position seq_lens[i] - 1.
int pm_channel_scan(const void* q, const void* v, int f32, long long ldu, const float* z, long long ldz, const
    float* bias, const float* lower, float* state, const int* slots, const int* q_start, const int* q_lens, const
    int* seq_lens, int n_seq, int H, int N, int P, void* y, cudaStream_t st);
// Matrix memory token by token. q / k / v as above, z fp32 rows of H input gates and H forget gates, bias fp32 [2 H]; nstate
// [slots][H][N] and mstate [slots][H][P4 / 4] fp32 beside the state; y [tokens, H P] without, den fp32 [tokens, H] with the
// normaliser: the result is y / den.
int pm_memory_scan(const void* q, const void* k, const void* v, int f32, long long ldu, const float* z, long long
    ldz, const float* bias, float cap, float qscale, float den_eps, float* state, float* nstate, float* mstate,
    const int* slots, const int* q_start, const int* q_lens, const int* seq_lens, int n_seq, int H, int N, int P,
    void* y, float* den, cudaStream_t st);
// pm_channel_scan for longer portions of bf16 models, N <= 256, n16 = N rounded up to 16. Work buffers over all rows of the step: act
// bf16 [tokens, 4 H n16], score bf16 [tokens, H, 128]; block_decay fp32 [n_tok / 64 + n_seq + 1][H][n16]; seg_state
// [n_seq][max_seg][H][N][P4] and seg_decay [n_seq][max_seg][H][N] fp32. c_start: first token of every sequence, counted over these
// sequences alone; max_q: the longest of q_lens.
int pm_channel_chunk(const void* q, const void* v, long long ldu, const float* z, long long ldz, const float* bias,
    const float* lower, float* state, const int* slots, const int* q_start, const int* q_lens, const int* seq_lens,
    const int* c_start, int n_seq, int max_q, int H, int N, int P, void* act, void* score, float* block_decay,
    float* seg_state, float* seg_decay, int max_seg, void* y, cudaStream_t st);
// pm_memory_scan for longer portions of bf16 models, N <= 256. u: rows ldu apart with the keys of head 0 at column k_at and the
// queries at q_at; work buffers gates fp32 [3][tokens, H], seg_state [n_seq][max_seg][H][N][P4], seg_decay [n_seq][max_seg][H] and
// seg_n [n_seq][max_seg][H][N] fp32.
int pm_memory_chunk(const void* u, int q_at, int k_at, const void* v, long long ldu, const float* z, long long ldz,
    const float* bias, float cap, float qscale, float den_eps, float* state, float* nstate, float* mstate, const
    int* slots, const int* q_start, const int* q_lens, const int* seq_lens, int n_seq, int n_tok, int max_q, int H,
    int N, int P, float* gates, float* seg_state, float* seg_decay, float* seg_n, int max_seg, void* y, float* den,
    cudaStream_t st);

// ---------------------------------------------------------------- gdn.cu
// Returns 0, -1 for an unsupported head shape (supported: dk x dv in {64, 128} x {64, 128}), or a CUDA error code.
int pm_gdn_scan(const float* q, const float* k, const float* v, const float* g, const float* beta, float* state,
    float* y, int B, int T, int H, int dk, int dv, cudaStream_t st);

// ---------------------------------------------------------------- gemm_2sm.cu
// Same contract as pm_gemm_bf16 with the tile fixed at 256 x 256 per CTA pair.
int pm_gemm_bf16_2sm(const void* A, int a_mn, int lda, int a_rows, const void* B, int b_mn, int ldb, int b_rows,
    const void* A2, int a2_mn, int lda2, int a2_k, const void* B2, int b2_mn, int ldb2, int b2_rows, void* D, int
    out_mode, int ldd, const void* R, int ldr, int M, int N, int K, int K2, int n_store, float alpha, int splits,
    int seg_mode, const int* seg_end, int seg_r, int max_ctas, float* tail, int tail_from, int ld_tail, int*
    status, cudaStream_t stream);

// ---------------------------------------------------------------- gemm_q4_2sm.cu
// A [M, K] bf16 (K-major). codes: packed weight [w_rows, w_cols / 2] bytes, first element of a pair in the high nibble;
// absmax (fp32) or absmax_q (+ am_scale / am_offset) hold one scale per 64 consecutive weights of a row.
//   trans 0: D[M, w_rows] (K = w_cols);  trans 1: D[M, w_cols] (K = w_rows).
// A2 / B2 (bf16, optional) add the low-rank product as in pm_gemm_bf16_2sm; seg_mode 0 or 1. D bf16 (+ R).
// w_cols % 128 == 0 and w_rows % 64 == 0. Returns 0, a negative argument error or a CUDA error code.
int pm_gemm_q4_2sm(const void* A, int lda, int a_rows, const void* codes, const float* absmax, const void*
    absmax_q, float am_scale, float am_offset, int fp4, int w_rows, int w_cols, int trans, const void* A2, int
    a2_mn, int lda2, int a2_k, const void* B2, int b2_mn, int ldb2, int b2_rows, void* D, int ldd, const void* R,
    int ldr, int M, int K2, int n_store, float alpha, int seg_mode, const int* seg_end, int seg_r, int max_ctas,
    int* status, cudaStream_t stream);

// ---------------------------------------------------------------- gemm_tcgen05.cu
// Returns 0 on success, negative on argument / descriptor errors, or the CUDA error code.
//   a_rows/b_rows: extent of the operand along M / N as seen by the tensor map (rows beyond it read as zero).
//   tail (nullable, bf16 output without R): columns from tail_from (a multiple of 8) on go there in fp32, rows ld_tail apart.
int pm_gemm_bf16(const void* A, int a_mn, int lda, int a_rows, const void* B, int b_mn, int ldb, int b_rows, const
    void* A2, int a2_mn, int lda2, int a2_k, const void* B2, int b2_mn, int ldb2, int b2_rows, void* D, int
    out_mode, int ldd, const void* R, int ldr, int M, int N, int K, int K2, int n_store, float alpha, int bn, int
    splits, int seg_mode, const int* seg_end, int seg_r, int max_ctas, float* ws, long long ws_floats, unsigned*
    ws_cnt, long long ws_cnt_len, float* tail, int tail_from, int ld_tail, int* status, cudaStream_t stream);

// ---------------------------------------------------------------- gemv.cu
// As pm_gemv with the epilogue of models that have biases and clamped gated units: bias [N_w] fp32 (nullable) is added to
// the scaled products; with swiglu and clamped != 0 the pair becomes min(g, limit) * sigmoid(beta min(g, limit)) *
// (clamp(u, -limit, limit) + shift); without swiglu, clamped = 2 applies the exact gelu; out_f32 != 0: y is fp32. tail (nullable):
// output columns from tail_from on are stored there in fp32, rows ld_tail apart, and not in y.
int pm_gemv_ex(const void* x, int ldx, const void* w, int ldw, const void* norm_w, float eps, const void* residual,
    int ldr, void* y, int ldy, int M, int N, int K, int swiglu, float alpha, const void* t, int ldt, const float*
    lora_b, int r, const int* seg_end, const float* bias, int clamped, float limit, float beta, float shift, int
    out_f32, float* tail, int tail_from, int ld_tail, cudaStream_t st);
// Returns 0, a negative argument error, or a CUDA error code. K % 8 == 0, row strides % 8 == 0, M <= 16,
// M * cols-per-warp <= 32.
int pm_gemv(const void* x, int ldx, const void* w, int ldw, const void* norm_w, float eps, const void* residual,
    int ldr, void* y, int ldy, int M, int N, int K, int swiglu, float alpha, const void* t, int ldt, const float*
    lora_b, int r, const int* seg_end, cudaStream_t st);
// 4-bit weights: qdata holds N_w * K / 2 bytes (two codes per byte, first element in the high nibble), absmax one fp32
// per qblock elements or absmax_q one byte per block with scale / offset (double quantisation). K % 32 == 0,
// qblock % 32 == 0. Other arguments as pm_gemv.
int pm_gemv_q4(const void* x, int ldx, const void* qdata, const float* absmax, const void* absmax_q, float
    am_scale, float am_offset, int qblock, int fp4, const void* norm_w, float eps, const void* residual, int ldr,
    void* y, int ldy, int M, int N, int K, int swiglu, float alpha, const void* t, int ldt, const float* lora_b,
    int r, const int* seg_end, cudaStream_t st);

// ---------------------------------------------------------------- grouped_gemm.cu
// a, b: the two operands of the mode (see the table at the top); both bf16, row strides lda / ldb in elements.
// off: int32 [E + 1] on the device, multiples of 128, off[E] <= rows_cap. D: bf16 [rows_cap, ldd] (modes 0, 1) or fp32
// [E, N, ldd] (mode 2; experts without rows are left untouched, so clear D first unless accumulating). gelu (mode 0): exact gelu of
// the products.
int pm_grouped_gemm(int mode, const void* a, int lda, const void* b, int ldb, void* D, int ldd, const int* off, int
    E, int rows_cap, int N, int K, float alpha, int accumulate, int gelu, int* status, cudaStream_t stream);
// Few rows per expert (see the kernel): x [rows, K] expert-sorted with offsets off [E + 1] (any alignment), w stacked
// [E * N, K] (act 0; act 2: exact gelu of the products) or [E * 2N, K] with gate rows above up rows per expert (act 1); y [rows, N] bf16.
// bn (32, 64, 128) is the token tile: experts with more rows take several passes over their weights.
int pm_grouped_gemm_skinny(const void* x, int ldx, int rows, const void* w, int ldw, void* y, int ldy, const int*
    off, int E, int N, int K, int bn, int act, float alpha, int* status, cudaStream_t stream);

// ---------------------------------------------------------------- latent_attn.cu
// qd [n, ld]: the queries' rotated parts are turned in place; with cache != null the down-projection behind the queries is
// normed / rotated and written to row slots[t] of cache [.., W + 8]. cs / sn [n, dr / 2]. lead > 0 (with H = 0): qd begins with
// a query latent of that many channels, which is normed in place with the weight lead_w (fp32).
int pm_latent_prep(void* qd, int f32, long long ld, const float* norm_w, float eps, const float* cs, const float*
    sn, int n, int H, int dn, int dr, int rank, void* cache, int W, const long long* slots, int lead, const float*
    lead_w, cudaStream_t st);
// Whether the tensor-core kernel covers H heads over rows of W columns with `rank` value columns.
int pm_latent_mma_supported(int H, int W, int rank);
// Attention of short portions in the latent space. qd as pm_latent_prep leaves it, wuk [H * dn, rank], wuv [H * dv, rank],
// cache [pages, 64, W + 8]. The n_tok tokens of the listed sequences are counted through: sequence i covers compact tokens
// c_start[i] .. of the work buffers q_lat [n_tok, H, W], part_o [n_split, n_tok * H, rank] fp32 and part_ml [n_split,
// n_tok * H, 2] fp32, and compact token j is row tok_rows[j] of qd and out. out [.., ldo]: H * dv columns. max_q: longest of
// q_lens. cs / sn (nullable) [.., dr / 2]: the queries' rotated parts are still to be turned. n_split <= 64 (1 for fp32 and for sizes that the tensor-core kernel does not cover).
int pm_latent_attn(const void* qd, int f32, long long ld, const void* wuk, const void* wuv, const void* cache,
    const int* block_table, const int* seq_lens, const int* c_start, const int* q_lens, const int* tok_rows, int
    n_seq, int max_blocks, int n_tok, int max_q, int H, int dn, int dr, int dv, int rank, int W, int n_split, float
    scale, void* q_lat, float* part_o, float* part_ml, void* out, long long ldo, const float* cs, const float* sn,
    int* status, cudaStream_t st);
// lat [n, r8] bf16 = latents of the n cache rows in `slots` (page * 64 + offset; zero padded).
int pm_latent_gather(const void* cache, const long long* slots, int n, int W, int rank, int r8, void* lat,
    cudaStream_t st);
// Operands [.., H, 128] bf16 of the flash-attention kernels for n_q queries and the n keys in `slots`; dn + dr <= 128,
// dv <= 128. qd: the first query row; kv [n, ldkv] = [keys: H * dn | values: H * dv].
int pm_latent_assemble(const void* qd, long long ldq, int n_q, const void* kv, long long ldkv, int n, const void*
    cache, const long long* slots, int W, int rank, int H, int dn, int dr, int dv, void* q128, void* k128, void*
    v128, cudaStream_t st);
// out [n, ldo] (H * dv columns) = the first dv channels of every head of o128 [n, H, 128].
int pm_latent_take(const void* o128, int n, int H, int dv, void* out, long long ldo, cudaStream_t st);

// ---------------------------------------------------------------- linear_attn.cu
// Token-by-token recurrence. u [tokens, ldu]; cs / sn fp32 [tokens, R / 2] (unused when R is 0); rot: 1 pairs (i, i + R / 2),
// 2 pairs (2 i, 2 i + 1); act: 1 silu on q, k, v; decay fp32 [H]; state [slots][H][N][P4] fp32, read and written;
// y [tokens, H P]. Sequence i covers tokens q_start[i] .. + q_lens[i] - 1 and ends at position seq_lens[i] - 1.
int pm_linear_scan(const void* u, int f32, long long ldu, const float* cs, const float* sn, const float* decay,
    float kscale, float* state, const int* slots, const int* q_start, const int* q_lens, const int* seq_lens, int
    n_seq, int H, int N, int P, int R, int rot, int act, void* y, cudaStream_t st);
// Whether pm_linear_chunk covers keys of N channels.
int pm_linear_chunk_supported(int N);
// The same for longer portions of bf16 models (act bf16 [n_tok, H P + 2 H N], twice the key and query columns when R > 0:
// work buffer over all n_tok rows of the step; log2_decay fp32 [H]; seg_state [n_seq][max_seg][H][N][P4] and seg_decay
// [n_seq][max_seg][H] fp32 work buffers; max_q: the longest of q_lens).
int pm_linear_chunk(const void* u, long long ldu, const float* cs, const float* sn, const float* log2_decay, float
    kscale, float* state, const int* slots, const int* q_start, const int* q_lens, const int* seq_lens, int n_seq,
    int n_tok, int max_q, int H, int N, int P, int R, int rot, int act, void* act_buf, float* seg_state, float*
    seg_decay, int max_seg, void* y, cudaStream_t st);
// out [tokens, ldo] = RMS norm over every part of y [tokens, parts * width], times w (fp32 [parts * width], shared 1: [width] for every
// part, or null), times sigmoid(gate) or, silu 1, silu(gate), times scale; gate rows are ldg apart (null: no gate). den (fp32
// [tokens, parts], nullable): y is divided by it first.
int pm_norm_gate(const void* y, const void* gate, int f32, long long ldg, const float* w, float eps, int parts, int
    width, int silu, void* out, int n_tok, const float* den, int shared, float scale, long long ldo, cudaStream_t
    st);

// ---------------------------------------------------------------- mhc.cu
// x [T, n, C] bf16; either phi [n C, n^2 + 2n] fp32 (dot products formed here) or raw [T, ld_raw] fp32 = x . phi computed by
// the caller; bias [n^2 + 2n], alpha [3]; n in {2, 4, 8}, C % 8 == 0, iters <= 32.
int pm_mhc_mappings(const void* x, const float* phi, const float* raw, int ld_raw, const float* bias, const float*
    alpha, int T, int n, int C, int iters, float* h_tilde, float* rms_inv, float* h_pre, float* h_post, float*
    h_res, cudaStream_t st);
int pm_mhc_pre(const void* x, const float* h_pre, int T, int n, int C, void* h_in, cudaStream_t st);
int pm_mhc_post_res(const void* x, const void* h_out, const float* h_res, const float* h_post, int T, int n, int C,
    void* x_out, cudaStream_t st);
int pm_mhc_mix_bwd(const void* x, const void* h_out, const void* dh_in, const void* dx_out, const float* h_pre,
    const float* h_post, const float* h_res, int T, int n, int C, void* dx, void* dh_out, float* d_pre, float*
    d_post, float* d_res, cudaStream_t st);
int pm_mhc_constraints_bwd(const float* h_tilde, const float* d_pre, const float* d_post, const float* d_res, int
    T, int n, int iters, float* d_tilde, cudaStream_t st);
// gains [2] fp32, cleared here: largest absolute row sum and column sum of H_res over all tokens
int pm_mhc_amax_gain(const float* h_res, int T, int n, float* gains, cudaStream_t st);
int pm_mhc_expand(const void* x, int T, int n, int C, void* xs, cudaStream_t st);
int pm_mhc_collapse(const void* xs, int T, int n, int C, void* x, cudaStream_t st);

// ---------------------------------------------------------------- moe_experts.cu
// out [T, n] fp32 = h [T, K] W^T (bf16, W [>= n, K]) for at most 64 outputs; K a multiple of 32, ldh of 8.
int pm_router_logits(const void* h, long long ldh, const void* W, int T, int n, int K, float* out, cudaStream_t
    st);
// xs [rows, width] = w[pair] * h[pair / k] (w null: h) for the pairs perm[0 .. n) sorted by expert (off [E + 1]). align 0: rows = n in
// sorted order. align > 0: every expert's slab starts at a multiple of align (off_pad [E + 1]), dest [n] is the row of each
// pair, rows between slabs are zero; rows must be at least n + (align - 1) per expert with pairs.
int pm_expert_gather(const void* h, int f32, long long ldh, const int* perm, const float* w, const int* off, int E,
    int k, int align, int rows, int width, void* xs, int* off_pad, int* dest, cudaStream_t st);
// Both bf16 products of a step with few rows per expert. act 1: out [n, N] = silu(w G_e h) * (w U_e h) for the n sorted pairs
// perm, h [.., ldx] token rows, w [n] weights by pair, W [E][2 N][K]. act 2: out = gelu(W_e h) for the same pairs, W [E][N][K].
// act 0: out = x W_e^T for sorted rows x. K, ldx and W in 16-byte pieces.
int pm_expert_gemv(const void* x, long long ldx, const void* W, const int* perm, const float* w, const int* off,
    int n, int E, int k, int N, int K, int act, void* out, cudaStream_t st);
// x [rows, K] sorted by expert (off [E + 1]; rows behind off[E] are skipped), W [E][N or, act 1, 2 N][K] -> out [rows, N] =
// x W_e^T, act 1: silu(x G_e^T) * (x U_e^T) (gate rows above up rows), act 2: gelu(x W_e^T).
int pm_expert_rows(const void* x, int f32, int rows, const void* W, const int* off, int E, int N, int K, int act,
    void* out, cudaStream_t st);

// ---------------------------------------------------------------- moe_gemm.cu
int pm_ep_prepare(const unsigned long long* offset_ptrs, const unsigned long long* pad_ptrs, int rank, int world,
    int e_loc, void* tiles, void* runs, int max_tiles, int max_runs, int* counts_out, double timeout_s, int*
    status, cudaStream_t st);
// a: local A buffer [a_rows, K] (row stride lda): the staging buffer of the gate/up launch or the hidden rows of the
// down launch; w: [e_loc * N, K]; out_ptrs[r]: output base of rank r (push = 0 uses out_ptrs[rank] only).
// copy_src_ptrs (gate/up launch): rank r's sorted token buffer [*, K] (row stride K) that tiles are staged in from;
// tile_ready: uint32 [max_tiles], zero-initialised once. Both null for the down projection.
int pm_moe_gemm(const void* a, int a_rows, int lda, const void* w, int ldw, int e_loc, const unsigned long long*
    out_ptrs, int ldd, const void* tiles, const void* runs, const int* n_tiles, int max_tiles, int N, int K, int
    swiglu, int rank, int world, int push, const unsigned long long* pad_ptrs, const unsigned long long*
    copy_src_ptrs, void* tile_ready, double timeout_s, int* status, cudaStream_t st);

// ---------------------------------------------------------------- moe_quant.cu
// Routing, counts, offsets and the expert-sorted order of T tokens. Logit rows (fp32 or bf16) are ldl apart; score 0 is the
// softmax over the experts, 1 the sigmoid of every logit; renorm divides the k weights by their sum. groups > 0 (at most 32,
// dividing E): the choice goes by score + correction (fp32 [E], nullable) among the experts of the `keep` groups of neighbours
// with the largest such sum, and the weights are multiplied by factor. offsets2: optional second destination for the [E + 1]
// offsets (may be null).
int pm_moe_route3(const void* logits, int is_f32, int ldl, int score, const float* correction, int groups, int
    keep, float factor, int T, int E, int k, int renorm, int* topk_idx, float* topk_w, int* counts, int* offsets,
    int* offsets2, int* perm, int* inv, cudaStream_t st);
int pm_moe_route2(const void* logits, int is_f32, int T, int E, int k, int renorm, int* topk_idx, float* topk_w,
    int* counts, int* offsets, int* offsets2, int* perm, int* inv, cudaStream_t st);
int pm_moe_route(const void* logits, int is_f32, int T, int E, int k, int renorm, int* topk_idx, float* topk_w,
    int* counts, int* offsets, int* perm, int* inv, cudaStream_t st);
// Routing plus the padded layout of the assignments that belong to experts [e0, e0 + e_loc) (see the kernel).
int pm_moe_route_local(const void* logits, int is_f32, int T, int E, int k, int renorm, int e0, int e_loc, int
    align, int* topk_idx, float* topk_w, int* off, int* dest, int* src, cudaStream_t st);
// off_end points at the device int holding the number of rows in use (off[e_loc]); cap bounds the launch.
int pm_moe_gather_padded(const void* x, const int* src, const int* off_end, int k, void* xs, int cap, int H,
    cudaStream_t st);
int pm_moe_combine_local(const void* z, const int* dest, const float* w, int k, const void* residual, void* y, long
    long T, int H, cudaStream_t st);
int pm_moe_gather(const void* x, const int* perm, int k, void* out, long long n, int H, cudaStream_t st);
int pm_moe_combine2(const void* z, const int* inv, const float* w, int k, const void* residual, void* y, long long
    T, int H, cudaStream_t st);
int pm_moe_combine(const void* z, const int* inv, const float* w, int k, void* y, long long T, int H, cudaStream_t
    st);
int pm_gguf_dequant_bf16(const void* src, void* dst, long long n, int type, cudaStream_t st);
int pm_fp8_quant(const void* x, void* q, float* scales, long long n, cudaStream_t st);
int pm_fp8_dequant(const void* q, const float* scales, void* y, long long n, cudaStream_t st);

// ---------------------------------------------------------------- postnorm.cu
// xf [n, width] fp32 = table[ids] * scale, xc the same in the table's type (nullable). f32: the table is fp32, else bf16.
int pm_embed_scale(const long long* ids, const void* table, int f32, float scale, int n, int width, float* xf,
    void* xc, cudaStream_t st);
// of / oc [n, width] (fp32 / compute type, each nullable) = LN(alpha * x + y + bias) * w + b for the n rows listed in
// `rows` (nullable: row i). y [.., ldy] and bias are nullable; without y the row is x itself. of may be x when rows is
// null.
int pm_post_layernorm(const float* x, const void* y, int f32, long long ldy, const float* bias, float alpha, const
    float* w, const float* b, float eps, int n, int width, const long long* rows, float* of, void* oc, cudaStream_t
    st);
// v = x + y + sum_j z[inv[t * k + j]] + x0 for the n rows listed in `rows` (nullable: row i); of [n, width] fp32 (nullable, may
// be x when rows is null) = v, oc [n, width] in the compute type = v / rms(v) * (w_base + w). y [.., ldy], z [.., width] (compute type,
// inv int32 per token and j < k) and x0 (fp32) are nullable.
int pm_add_rmsnorm(const float* x, const void* y, int f32, long long ldy, const void* z, const int* inv, int k,
    const float* x0, const float* w, float w_base, float eps, int n, int width, const long long* rows, float* of,
    void* oc, cudaStream_t st);
// v = x + r / rms(r) * (w_base + w) with r = y + sum over j < k of wt[t, j] * (ids[t, j] < n_experts ? z[row[t, j]] : x[t]); of
// [n, width] fp32 = v (may be x), oc the same in the compute type (nullable). y [.., ldy] is nullable, k may be 0.
int pm_add_normed(const float* x, const void* y, int f32, long long ldy, const void* z, const int* row, const int*
    ids, const float* wt, int k, int n_experts, const float* w, float w_base, float eps, int n, int width, float*
    of, void* oc, cudaStream_t st);
// out [n, ldo] = exact gelu of x [n, ldx] on the first `cols` columns; out may be x.
int pm_gelu(const void* x, int f32, long long ldx, int n, int cols, void* out, long long ldo, cudaStream_t st);
// gu [n, ld]: gate columns [0, ff), up columns [ff, 2 ff); bias fp32 [2 ff] or null -> out [n, ff].
int pm_clamped_glu(const void* gu, int f32, long long ld, const float* bias, int n, int ff, float limit, float
    beta, float shift, void* out, cudaStream_t st);
// cos / sin [n, half] fp32 of pos * freq (freq fp64 [half] on the device).
int pm_rope_table_f64(const int* pos, const double* freq, int n, int half, float* cs, float* sn, cudaStream_t st);

// ---------------------------------------------------------------- sampling.cu
int pm_sample(const void* logits, int is_bf16, long long ld, int rows, int vocab, const int* counts, const int*
    count_rows, const float* temperature, const int* top_k, const float* top_p, const float* min_p, const float*
    rep_pen, const float* freq_pen, const float* pres_pen, const unsigned long long* seeds, unsigned long long
    step, int* out_token, float* out_logprob, cudaStream_t st);
int pm_spec_verify(const float* target, const float* draft, const int* tokens, int n_seq, int K, int vocab, float
    temperature, const unsigned long long* seeds, unsigned long long step, int* n_accepted, int* next_token,
    cudaStream_t st);
int pm_count_tokens(int* counts, const int* count_rows, const int* tokens, int rows, int vocab, cudaStream_t st);

// ---------------------------------------------------------------- sandwich.cu
// xf [n, width] fp32 = table[id] + pairs[row] + pos_table[position], xc (nullable, rows ldc apart) the same in the tables' type; row =
// (previous id * mul_prev + id * mul_cur) mod buckets, `buckets` itself for a sequence's first token. Sequence i brings the tokens
// q_start[i] .. + q_lens[i] - 1; last[slots[i]] (int32) holds its latest token, read and written. Positions lie below max_pos.
int pm_pair_embed(const long long* ids, const void* table, const void* pairs, const void* pos_table, int f32, const
    int* pos, const int* seq_of, const int* q_start, const int* q_lens, const int* slots, int* last, long long
    buckets, long long mul_prev, long long mul_cur, int n, int width, int max_pos, float* xf, void* xc, long long
    ldc, cudaStream_t st);
// v = x + r / rms(r) (base + wb), r = y + bias (y nullable: v = x), for the n rows listed in `rows` (nullable: row i); of [n, width]
// fp32 (nullable, written when there is a y; may be x when rows is null) = v, oc (nullable, compute type, rows ldo apart) =
// v / rms(v) (base + wn), without wn v itself. conv (nullable, [taps][width] fp32, with wn and without rows): row i is the only new
// token of a sequence, at position pos[i] with the ring of slot slots[i]; oc = h + sum_j conv[j] h_(taps - 1 - j tokens earlier).
int pm_branch_norm(const float* x, const void* y, int f32, long long ldy, const float* bias, const float* wb, const
    float* wn, float base, float eps, const long long* rows, float* of, void* oc, long long ldo, const float* conv,
    int taps, void* ring, const int* slots, const int* pos, int n, int width, cudaStream_t st);
// out [tokens, width] = h + causal convolution of h with w [taps][width] fp32 along every sequence; h and out in the compute type,
// two buffers. ring [slot][taps - 1][width] (compute type) holds the sequences' earlier inputs, read and written. taps <= 17.
int pm_canon(const void* h, int f32, const float* w, int taps, void* ring, const int* slots, const int* q_start,
    const int* q_lens, const int* seq_lens, int n_seq, int max_q, int width, void* out, cudaStream_t st);

// ---------------------------------------------------------------- ssm.cu
// Token-by-token recurrence with the convolution inside. u [tokens, ldu]; conv_w [taps][conv], conv_b, dt_bias, a_log,
// dskip fp32; ring [slots][taps][conv] in u's type; state [slots][H][N][P4] fp32, read and written; y [tokens, H P].
// Sequence i covers tokens q_start[i] .. + q_lens[i] - 1 and ends at position seq_lens[i] - 1.
int pm_ssm_scan(const void* u, int f32, long long ldu, const float* conv_w, const float* conv_b, const float*
    dt_bias, const float* a_log, const float* dskip, const void* ring, float* state, const int* slots, const int*
    q_start, const int* q_lens, const int* seq_lens, int n_seq, int H, int P, int N, int G, int taps, void* y,
    cudaStream_t st);
// Whether pm_ssm_chunk covers a state of N rows.
int pm_ssm_chunk_supported(int N);
// The same for longer portions of bf16 models: act [tokens, conv] bf16, dt [tokens, H], seg_state [n_seq][max_seg][H][N][P4]
// and seg_decay [n_seq][max_seg][H] fp32 are work buffers, max_q is the longest of q_lens. A portion is cut into at most
// max_seg segments that run in parallel (fewer when sequences and heads fill the machine by themselves).
int pm_ssm_chunk(const void* u, long long ldu, const float* conv_w, const float* conv_b, const float* dt_bias,
    const float* a_log, const float* dskip, const void* ring, float* state, const int* slots, const int* q_start,
    const int* q_lens, const int* seq_lens, int n_seq, int max_q, int H, int P, int N, int G, int taps, void* act,
    float* dt, float* seg_state, float* seg_decay, int max_seg, void* y, cudaStream_t st);
// out [tokens, H P] = RMS norm over `parts` equal parts of y * silu(z) (z: the first H P columns of u), times w; the last
// taps - 1 convolution inputs of every sequence go to the ring. seq_of / pos [tokens]: sequence index and position.
int pm_ssm_gate_norm(const void* y, const void* u, int f32, long long ldu, const float* w, float eps, int parts,
    void* out, void* ring, const int* slots, const int* seq_of, const int* pos, const int* seq_lens, int n_tok, int
    H, int P, int N, int G, int taps, cudaStream_t st);

// ---------------------------------------------------------------- tp_fused.cu
// mode 0: x_ptrs[r] = rank r's X shard [rows_per_rank, K] (ldx), w = W_loc [N, K] (ldw), out = Y [M, ldd].
// mode 1: x_ptrs[rank] = local X [M, K] (ldx), w = W_loc [N, K], stage_ptrs[r] = rank r's staging buffer,
//         out = Y_r [rows_per_rank, ldd]. K and N are the local extents. mode 0 also takes `gathered` (local bf16
//         [M, K] scratch) and `blk_ready` (uint32 [M / 128], zero-initialised once). Returns 0, a negative argument
//         error, or a CUDA error code.
int pm_tp_gemm(int mode, const unsigned long long* x_ptrs, int ldx, const void* w, int ldw, void* out, int ldd,
    const unsigned long long* stage_ptrs, const unsigned long long* pad_ptrs, int rank, int world, int M, int N,
    int K, void* gathered, void* blk_ready, double timeout_s, int max_ctas, int* status, cudaStream_t stream);
// x: bf16 [n] (n a multiple of 8, at most slot_elems), summed in place over the ranks. bufs[r] / pads[r]: rank r's
// exchange buffer (2 * world * slot_elems bf16) and signal pad (64 uint32, zero-initialised once), peer-mapped.
int pm_peer_allreduce(void* x, long long n, const unsigned long long* bufs, const unsigned long long* pads, long
    long slot_elems, int rank, int world, double timeout_s, int* status, cudaStream_t st);

// ---------------------------------------------------------------- train_aux.cu
int pm_kd_fwd_bwd(void* student, long long ld, const void* teacher, long long ldt, int rows, int V, float
    temperature, int kind, float beta, const float* row_scale, float* row_loss, float* loss_sum, int write_grad,
    cudaStream_t st);
int pm_merge_fused(const void* const* models, const void* base, const float* weights, const float* thresholds,
    const float* densities, int n_models, int in_bf16, int out_bf16, int consensus, int rescale, float lam,
    unsigned long long seed, void* out, long long n, cudaStream_t st);
int pm_dot_norms(const void* a, const void* b, int bf16, long long n, float* out3, cudaStream_t st);

// ---------------------------------------------------------------- window_attn.cu
// u [n_tok, ldu]: queries [H][M][D] from column 0 and, with pages, keys [G][M][D] from column k_at and values [G][DV] from
// column v_at (k_at again: the values are the keys before rotation and norm). q_out [n_tok, H M, D8] (wide > 0: rows of that many
// channels, those of map i from i D8 on, zeros elsewhere) and the cache rows
// pages[slot] get rotated (first R channels; pairs 1: (2 i, 2 i + 1), else (i, i + R / 2); cs / sn fp32 [n_tok, R / 2]) and,
// normed 1, normalised vectors times qw / kw (fp32 [D], nullable). temp_every > 0: queries at position p = pos[t] are multiplied
// by 1 + temp_coef ln(floor((p + 1) / temp_every) + 1).
int pm_window_prep(const void* u, int f32, long long ldu, const float* cs, const float* sn, int n_tok, int H, int
    G, int M, int D, int DV, int wide, int k_at, int v_at, int R, int pairs, int normed, float eps, const float*
    qw, const float* kw, const int* pos, float temp_coef, int temp_every, void* q_out, void* pages, const long
    long* slots, cudaStream_t st);
// Attention of the new tokens q_start[i] .. + q_lens[i] - 1 of n_seq sequences (rows of q as pm_window_prep leaves them and out [.., ldo])
// over their cached keys; sequence i has seq_lens[i] keys behind row i of block_table. Scores times scale, capped when
// softcap > 0; sink (fp32 [H], M = 1) adds exp(sink) to a head's softmax sum; gate [.., ldg] multiplies head h by the sigmoid of
// column h. M = 2: the result of a head is a_1 - lambda[0] a_2 over its root mean square (eps inside), times keep; it takes o
// [n_tok, H M, DV] in the compute type unless parts are given. few 1: decode tiles (a few rows per sequence), which take work
// buffers po [n_split][n_tok][H M][DV8] and pml [n_split][n_tok][H M][2] (both or none; needed for n_split > 1). chunked 1: a position
// sees the keys of its own chunk of `window` positions. wbias (fp32 [H], nullable, M = 1, without sink): the weight of a key is the
// sigmoid of its score + wbias, not divided by their sum. out_scale multiplies the result.
int pm_window_attn(const void* q, int f32, const void* pages, const int* block_table, const int* seq_lens, const
    int* q_start, const int* q_lens, int n_seq, int max_blocks, int n_tok, int max_q, int H, int G, int M, int D,
    int DV, int wide, int window, float scale, float softcap, const float* sink, const void* gate, long long ldg,
    const float* lambda, float keep, float eps, int few, int n_split, float* po, float* pml, void* o, void* out,
    long long ldo, int chunked, const float* wbias, float out_scale, cudaStream_t st);
// k128 / v128 [n, G, 128] bf16 = the cached keys (M maps of D8 channels side by side) and values (DV8) of the n cache rows in `slots`
// (page * 64 + offset), zero padded. M D8 <= 128 and DV8 <= 128.
int pm_window_expand(const void* pages, const long long* slots, int n, int G, int M, int D, int DV, void* k128,
    void* v128, cudaStream_t st);
// The last step of pm_window_attn by itself, for the tokens of n_seq sequences: o [n_tok, H M, OP] (bf16, DV channels per row) -> out
// [.., ldo]: the difference of two maps with its norm (M = 2: lambda, keep, eps) and the heads' gates (nullable).
int pm_window_finish(const void* o, int n_tok, int H, int M, int DV, int OP, const int* q_start, const int* q_lens,
    int n_seq, int max_q, const float* lambda, float keep, float eps, const void* gate, long long ldg, void* out,
    long long ldo, cudaStream_t st);

#ifdef __cplusplus
}
#endif
