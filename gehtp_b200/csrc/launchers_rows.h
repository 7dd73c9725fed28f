// Launchers behind the row-count opcodes (OP_EMBED_ROWS .. OP_WINDOW_ATTEND, wtop_format.h). Pointers are device
// pointers, sizes in elements; `bf16` = activations in bf16 (else fp32); `exact` = the simple kernels with fp32
// arithmetic throughout, which fp32 runlists always take and bf16 ones in the one-kernel-per-op plan.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>
#include "launchers.h"

namespace gehtp {

// ---- rows, norms, sampling (ops_rows.cu)
void k_embed_rows(cudaStream_t st, const uint16_t* table, const int32_t* ids, float* x, void* act, uint32_t act_ld, uint32_t rows, uint32_t width,
                  uint32_t vocab, float scale, bool bf16);
struct NormResidArgs {
    const void* y; const float* w; const float* x; float* x_out; void* act;
    uint32_t width, rows_arg; float eps, base; bool act_bf16, y_bf16;
};
void k_norm_resid(cudaStream_t st, const NormResidArgs& a, uint32_t rows);
// x_out = x + t(y, p), act = t(x_out, next), t(z, p) = tanh(alpha z) w + b (p = 0: z); rows of y, or those idx picks
struct TanhResidArgs {
    const void* y; const int32_t* idx; uint32_t y_rows;
    const float *p, *x, *next; float* x_out; void* act;
    uint32_t width, act_ld, rows_arg; bool act_bf16, y_bf16;
};
void k_tanh_resid(cudaStream_t st, const TanhResidArgs& a, uint32_t rows);
void k_pick_rows(cudaStream_t st, const float* x, const int32_t* idx, float* out, uint32_t rows, uint32_t width, uint32_t x_rows);
void k_argmax_rows_f32(cudaStream_t st, const float* x, int32_t* out, uint32_t rows, uint32_t n);
void k_state_advance(cudaStream_t st, uint32_t* counters, uint32_t n, uint32_t rows);

// ---- projections (linear_rows.cu, f16_gemm_sm100.cu): y[M, N] = act(x[M, K] . w^T + bias), w bf16 [N, K], fp32 accumulation
struct LinearArgs {
    const void* x; const uint16_t* w; void* y;
    uint32_t K, N, xs, ys;          // row strides of x and y
    uint32_t rows_arg;
    bool x_bf16, y_bf16, relu2;
    bool gelu_gate;                 // rows of w are (gate, up) pairs, y[M, N / 2] = gelu(gate) * up
    const float* bias;
    // the projection goes straight into the residual sum: x_out = res + t(x . w^T, p), act = t(x_out, next); y is not
    // written (tanh_norm in linear_epi.cuh)
    bool tanh;
    const float *p, *res, *next; float* x_out; void* act; uint32_t act_ld;
};
void k_linear(cudaStream_t st, const LinearArgs& a, uint32_t M, bool exact, unsigned int* status);
// tcgen05 form (bf16 x): false = shape or alignment not taken, nothing launched
bool k_linear_sm100(cudaStream_t st, const LinearArgs& a, uint32_t M, unsigned int* status);

// ---- latent attention (latent_attn.cu, latent_prefill.cu)
struct LatentArgs {
    const void* y; const float* norm_w; const float* rope; void* q; float* gate;      // append
    void* state; const uint32_t* counter; uint32_t nslots; uint32_t state_idx;
    const uint16_t* w_kv; void* out; float* work;                                     // attend
    uint32_t heads, dim, rot, vdim, rank, rows_arg, rope_rows;
    float eps, scale; bool bf16;
    unsigned int* status;
    // columns of a y row: q at 0, latent | rotated key part, gate, and the row length
    __host__ __device__ uint32_t col_lat() const { return (heads * (dim + rot) + 7u) & ~7u; }
    __host__ __device__ uint32_t col_gate() const { return col_lat() + ((rank + rot + 7u) & ~7u); }
    __host__ __device__ uint32_t y_cols() const { return col_gate() + ((heads + 7u) & ~7u); }
    __host__ __device__ uint32_t ls() const { return latent_row(rank, rot); }
    __host__ __device__ static uint32_t latent_row(uint32_t rank, uint32_t rot) { return (rank + rot + 15u) & ~15u; }   // elements of a state row, zero-padded
};
size_t latent_work_floats(const LatentArgs& a, uint32_t max_rows);
void k_latent_append(cudaStream_t st, const LatentArgs& a, uint32_t rows);
// n_past: the host's count of positions before this run; exact = true launches nothing that depends on it
void k_latent_attend(cudaStream_t st, const LatentArgs& a, uint32_t rows, uint32_t n_past, bool exact);
// append + attend for few rows in one chain (rotary, latent, query absorption in one launch); false: not taken
bool k_latent_step(cudaStream_t st, const LatentArgs& a, uint32_t rows);

// ---- grouped-query attention over a window of positions, keys and values in a ring (window_attn.cu, window_prefill.cu)
struct WindowArgs {
    const void* y; uint32_t y_cols; const float* norms; const float* rope; void* q;         // append
    void* state; const uint32_t* counter; uint32_t ring, state_idx, positions;
    void* out; uint32_t window, gate_col;                                                   // attend; gate_col ~0: no gate
    uint32_t heads, kv_heads, dim, vdim, rot, rows_arg;
    float eps, scale; bool bf16;
    unsigned int* status;
    // columns of a y row: q at 0, k, v; elements of a state row: k of every key head, then v
    __host__ __device__ uint32_t col_k() const { return (heads * dim + 7u) & ~7u; }
    __host__ __device__ uint32_t col_v() const { return col_k() + ((kv_heads * dim + 7u) & ~7u); }
    __host__ __device__ uint32_t min_cols() const { return col_v() + kv_heads * vdim; }
    __host__ __device__ uint32_t row() const { return kv_row(kv_heads, dim, vdim); }
    __host__ __device__ static uint32_t kv_row(uint32_t kvh, uint32_t dim, uint32_t vdim) { return (kvh * (dim + vdim) + 7u) & ~7u; }
};
void k_heads_append(cudaStream_t st, const WindowArgs& a, uint32_t rows);
void k_window_attend(cudaStream_t st, const WindowArgs& a, uint32_t rows, bool exact);
// append + attention of one row in one launch; false: not taken
bool k_window_step(cudaStream_t st, const WindowArgs& a, uint32_t rows);

// ---- gated delta rule with a decay per key channel (channel_delta.cu)
struct DeltaArgs {
    const void* y; uint32_t ys, b_col;                      // joined projection rows, column of the step-size logits
    const float* conv_w; float* conv_state; const uint32_t* conv_count; uint32_t taps;
    float* qkv;                                             // convolved q | k | v, fp32
    const float* a; const float* a_log; const float* dt_bias;
    float* S; float* o; float* work;
    uint32_t heads, kv_heads, dim, vdim, rows_arg;
    const float* norm_w; const float* gate; void* out; float eps; bool bf16;
    // one-kernel step: second halves of the low-rank decay and gate projections, columns of their first halves in y
    const uint16_t *a2, *g2; uint32_t rank_a, rank_g, a_col, g_col;
    __host__ __device__ uint32_t channels() const { return 2 * kv_heads * dim + heads * vdim; }
};
void k_short_conv(cudaStream_t st, const DeltaArgs& a, uint32_t rows);
size_t delta_work_floats(const DeltaArgs& a, uint32_t max_rows);
void k_channel_delta(cudaStream_t st, const DeltaArgs& a, uint32_t rows);
// all of the above for up to 4 rows in one launch, the low-rank projections included; false: sizes not taken
bool k_delta_step(cudaStream_t st, const DeltaArgs& a, uint32_t rows);
void k_gated_norm(cudaStream_t st, const DeltaArgs& a, uint32_t rows);

// what a planned row-count op was resolved to
struct RowsArgs {
    LinearArgs lin;
    NormResidArgs norm;
    TanhResidArgs tanh;
    WindowArgs win;
    LatentArgs lat;
    DeltaArgs del;
};

}  // namespace gehtp
