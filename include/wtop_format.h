/* WTOP runlist blob: wire format and in-memory form.
 *
 * This is the ABI shared with the GEHTP toolchain (kernels/include/oplist_parse.h:1-312
 * in the reference): a blob produced by its `wtop_emit` parses with wt_parse()
 * below into the same struct layout, and the numeric values of every constant
 * here are the reference's. Names are kept so that callers written against the
 * reference header compile unchanged.
 *
 * Wire layout, little endian:
 *   0   "WTOP"
 *   4   u16 version (1 or 2)        6   u16 0x1234 byte-order probe
 *   8   u32 n_slots                 12  u32 n_ops
 *   16  slot records: v1 = 16 B {len, count, offset32, addr}
 *                     v2 = 24 B {len, count, offset_lo, offset_hi, addr, reserved}
 *   ..  op records: {u16 opcode, u16 n_args, u32 args[n_args]}
 *   ..  weight area, starting at the next multiple of 128 after the op table;
 *       slot offsets are relative to it and 128-byte aligned.
 *
 * An op argument that names a tensor is a "ref":
 *   bare value          temp id
 *   0x8000 | slot       constant / input slot
 *   0x4000 | temp       temp resident in on-chip scratch (VTCM on Hexagon; an
 *                       ordinary arena temp on a GPU)
 *   0x6000 | state      persistent state buffer (KV ring, conv window, delta S)
 *   0xC000 | face       engine face, OP_DMA only
 */
#ifndef GEHTP_B200_WTOP_FORMAT_H
#define GEHTP_B200_WTOP_FORMAT_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define WT_BLOB_VER        1u
#define WT_BLOB_VER_2      2u
#define WT_ENDIAN_CHK      0x1234u
#define WT_SLOT_SIZE       16u
#define WT_SLOT_SIZE_V2    24u
#define WT_WEIGHT_ALIGN    128u
#define WT_MAX_SLOTS       4096u
#define WT_MAX_OPS         65536u
#define WT_MAX_ARGS        16u
#define WT_MAX_STATES      64u
#define WT_EXEC_MAX_TEMPS  4096

/* slot.addr markers (oplist_parse.h:62-88) */
#define WT_SLOT_EXT_IN     0xFFFFFFFFu  /* data comes from run_io's in_ptr        */
#define WT_SLOT_EXT_OUT    0xFFFFFFFEu
#define WT_SLOT_TEMPOFF    0xFFFFFFFDu  /* static temp offset table               */
#define WT_SLOT_EXT_WGT    0xFFFFFFFCu  /* data in the external weight file       */
#define WT_SLOT_STATE      0xFFFFFFFBu  /* persistent state size table            */
#define WT_KV_POS_AUTO     0xFFFFFFFAu  /* KV pos / n_kv taken from state counter */

/* Row-count runlists (no counterpart in the reference). A blob with a WT_SLOT_ROWS slot - u32 {max_rows, max_sel} -
 * may be run with any number of token rows up to max_rows, of which up to max_sel are picked for the head
 * (gehtp_cuda_set_rows). Row arguments of the ops below take these markers instead of a number. */
#define WT_SLOT_ROWS       0xFFFFFFF7u
#define WT_ROWS_AUTO       0xFFFFFFF9u  /* token rows of the run                     */
#define WT_SEL_AUTO        0xFFFFFFF8u  /* rows picked for the head in this run      */

#define WT_REF_SLOT_FLAG   0x8000u
#define WT_REF_VTCM_FLAG   0x4000u
#define WT_REF_STATE_FLAG  0x6000u
#define WT_REF_ENG_FLAG    0xC000u
#define WT_ENG_ACT  0u
#define WT_ENG_OUT  1u
#define WT_ENG_WT   2u
#define WT_ENG_BIAS 3u
#define WT_DMA_FENCE_NONE  0xFFu

/* Opcodes (oplist_parse.h:103-215). Argument lists are given beside the
 * executor entry that implements each one, in gehtp_b200/csrc/. */
enum {
    OP_NOP = 0, OP_MATMUL_W4A16 = 1, OP_RMSNORM_F16 = 2, OP_PIN = 3, OP_SILU_F16 = 4,
    OP_IM2COL = 5, OP_CONV2D_F16 = 6, OP_ADD_F16 = 7, OP_SPILL = 8, OP_FILL = 9,
    OP_TRANSPOSE_F16 = 10, OP_UNARY_F16 = 11, OP_BINARY_F16 = 12, OP_SOFTMAX_F16 = 13,
    OP_CONCAT_F16 = 14, OP_STRIDED_SLICE_F16 = 15, OP_SPLIT_F16 = 16, OP_REDUCE_F16 = 17,
    OP_CUMSUM_F32 = 18, OP_CONV1D_SSM_F16 = 19, OP_GATHER_F16 = 20, OP_ARGMAX_F16 = 21,
    OP_KV_APPEND_F16 = 22, OP_KV_GATHER_F16 = 23, OP_MATMUL_F16 = 24, OP_RMSNORM2_F16 = 25,
    OP_BROADCAST_F16 = 26, OP_TRANSPOSE_GEN_F16 = 27, OP_SCATTER_ND_F16 = 28,
    OP_CONV1D_SSM_STEP_F16 = 29, OP_DELTA_CHUNK_F16 = 30,
    OP_DMA = 33, OP_PAD_F16 = 34, OP_MATMUL_F16_SPLIT = 35
};

/* Opcodes of this executor alone, far from the reference's numbers. Activations are bf16 or fp32 (WT_DT_*), weights
 * bf16 as stored in checkpoints, the residual stream, norms, gates, scores and recurrent state fp32.
 * "rows" arguments: a number, WT_ROWS_AUTO or WT_SEL_AUTO. Sizes are in elements, *_bits are fp32 bit patterns.
 *
 * OP_EMBED_ROWS     [table, ids, x_out, act_out, rows, width, vocab, dt, scale_bits, act_stride, act_col]
 *                   x = table[id] * scale (fp32), act[:, act_col: act_col + width] = x in dt; act_stride 0 = width
 * OP_LINEAR         [x, w, y, rows, K, N, flags, x_col, x_stride, bias]       y = act(x[:, x_col: x_col + K] . w^T + bias), w bf16
 *                   [N, K], bias fp32 [N] (0: none); flags: WT_LIN_*; x_stride 0 = K. With WT_LIN_GELU_GATE the rows of w are
 *                   (gate, up) pairs and y [rows, N / 2] = gelu(gate) * up, the tanh form of gelu
 * OP_NORM_RESID     [y, w, x, x_out, act_out, rows, width, flags, eps_bits]   x_out = x + y / rms(y) * (b + w), w fp32;
 *                   flags: bit 0 b = 1 (weights are deviations from one) else b = 0, bit 1 act_out is bf16, bit 2 y is bf16.
 *                   x = 0: no residual; x_out / act_out = 0: not written
 * OP_PICK_ROWS      [x, idx, idx_off, out, rows, width]                       out[r] = x[idx[idx_off + r]] (fp32 rows, int32 idx)
 * OP_LATENT_APPEND  [y, norm_w, rope, q_out, gate_out, state, rows, heads, dim, rot, rank, eps_bits, flags]
 *                   y rows = [q: heads x (dim | rot) | latent: rank | key part: rot | gate: heads], each group starting at a
 *                   multiple of 8; rope: fp32 [positions][rot / 2][cos, sin], neighbouring components paired. Appends
 *                   [norm(latent) * norm_w | rotated key part] to the state at the state's position counter; flags: WT_DT_*
 * OP_LATENT_ATTEND  [q, gate, state, w_kv, out, work, rows, heads, dim, rot, vdim, rank, scale_bits, flags]
 *                   w_kv bf16 = [up-projection of keys: heads x dim | of values: heads x vdim][rank]; causal over the state;
 *                   out = softmax(q . k * scale) v * sigmoid(gate) per head; work: scratch temp
 * OP_SHORT_CONV     [y, w, state, out, rows, channels, taps, y_stride, flags] out = silu(causal depthwise conv of y[:, :channels]),
 *                   w fp32 [channels][taps], last tap = current token; fp32 out, the last taps - 1 inputs live in the state
 * OP_CHANNEL_DELTA  [qkv, a, y, a_log, dt_bias, state, out, work, rows, heads, kv_heads, dim, vdim, b_col, y_stride, flags]
 *                   delta rule with a decay per key channel: S <- exp(-exp(a_log) softplus(a + dt_bias)) S,
 *                   u = sigmoid(b)(v - S^T k), S <- S + k u^T, out = S^T q; q, k unit vectors, q * dim^-1/2
 * OP_GATED_NORM     [o, w, gate, out, rows, heads, vdim, eps_bits, flags]     out = o / rms(o) * w * sigmoid(gate) per head
 * OP_ARGMAX_ROWS    [x, out, rows, n]                                         int32 per row of fp32 x
 * OP_STATE_ADVANCE  [first, n, rows]                                          adds rows to the position counters of n states
 * OP_TANH_RESID     [y, p, x, x_out, next, act_out, rows, width, flags, act_stride, act_col]
 *                   element by element: x_out = x + t(y, p), act_out[:, act_col: act_col + width] = t(x_out, next) with
 *                   t(z, p) = tanh(alpha z) w + b, p fp32 [alpha, 0, 0, 0 | w: width | b: width]; p, next = 0: t(z) = z;
 *                   x = 0: no residual; x_out / act_out = 0: not written; flags: bit 1 act_out is bf16, bit 2 y is bf16
 * OP_HEADS_APPEND   [y, norms, rope, q_out, state, rows, heads, kv_heads, dim, vdim, rot, eps_bits, y_stride, positions, dt]
 *                   y rows = [q: heads x dim | k: kv_heads x dim | v: kv_heads x vdim | ...], each group starting at a multiple of
 *                   8; q and k per head: / rms * norms (fp32 [q: dim | k: dim]; 0: left as they are), then the first rot components
 *                   turned, i with i + rot / 2 (rope: fp32 [positions][rot / 2][cos, sin]). Appends [k | v] to the state, a ring:
 *                   position p lies in row p mod (rows of the state); positions: the most the counter may reach
 * OP_WINDOW_ATTEND  [q, y, state, out, rows, heads, kv_heads, dim, vdim, window, scale_bits, gate_col, y_stride, dt]
 *                   softmax(q . k * scale) v over the last `window` positions up to the row's own, query head h with key head
 *                   h / (heads / kv_heads); times sigmoid(y[:, gate_col: gate_col + heads * vdim]) unless gate_col is all ones */
enum {
    OP_EMBED_ROWS = 0x140, OP_LINEAR, OP_NORM_RESID, OP_PICK_ROWS, OP_LATENT_APPEND, OP_LATENT_ATTEND, OP_SHORT_CONV,
    OP_CHANNEL_DELTA, OP_GATED_NORM, OP_ARGMAX_ROWS, OP_STATE_ADVANCE, OP_TANH_RESID, OP_HEADS_APPEND, OP_WINDOW_ATTEND, OP_ROWS_END
};
#define WT_DT_F32   0u
#define WT_DT_BF16  1u
#define WT_LIN_X_BF16  1u
#define WT_LIN_Y_BF16  2u
#define WT_LIN_RELU2   16u   /* y = max(x . w, 0)^2 */
#define WT_LIN_GELU_GATE 32u
#define WT_COL_ALIGN   8u    /* column groups of a joined projection start at multiples of this many elements */

/* Fixed argument count per opcode (oplist_parse.h:218-251). */
#define WT_ARITY_NOP 0
#define WT_ARITY_MATMUL 6
#define WT_ARITY_RMSNORM 4
#define WT_ARITY_PIN 1
#define WT_ARITY_SILU 3
#define WT_ARITY_IM2COL 15
#define WT_ARITY_CONV2D_F16 13
#define WT_ARITY_ADD_F16 4
#define WT_ARITY_SPILL 4
#define WT_ARITY_FILL 4
#define WT_ARITY_TRANSPOSE_F16 6
#define WT_ARITY_UNARY_F16 4
#define WT_ARITY_BINARY_F16 5
#define WT_ARITY_SOFTMAX_F16 4
#define WT_ARITY_CONCAT_F16 16
#define WT_ARITY_STRIDED_SLICE_F16 16
#define WT_ARITY_SPLIT_F16 16
#define WT_ARITY_REDUCE_F16 9
#define WT_ARITY_CUMSUM_F32 7
#define WT_ARITY_CONV1D_SSM_F16 6
#define WT_ARITY_GATHER_F16 15
#define WT_ARITY_ARGMAX_F16 3
#define WT_ARITY_KV_APPEND_F16 4
#define WT_ARITY_KV_GATHER_F16 7
#define WT_ARITY_MATMUL_F16 7
#define WT_ARITY_RMSNORM2_F16 5
#define WT_ARITY_BROADCAST_F16 12
#define WT_ARITY_TRANSPOSE_GEN_F16 8
#define WT_ARITY_SCATTER_ND_F16 14
#define WT_ARITY_DMA 8
#define WT_ARITY_PAD_F16 7
#define WT_ARITY_MATMUL_F16_SPLIT 9
#define WT_ARITY_CONV1D_SSM_STEP_F16 6
#define WT_ARITY_DELTA_CHUNK_F16 12

struct wt_slot {
    uint32_t len;     /* bytes */
    uint32_t count;   /* elements (f16 unless the consuming op says otherwise) */
    uint64_t offset;  /* bytes from weight_base (or from the external weight base) */
    uint32_t addr;    /* 0 or one of WT_SLOT_* */
};

struct wt_op {
    uint16_t opcode;
    uint16_t n_args;
    uint32_t args[WT_MAX_ARGS];
};

/* About 4.5 MB: callers allocate it on the heap. */
struct wt_blob {
    uint16_t ver;
    uint32_t n_slots;
    uint32_t n_ops;
    uint32_t weight_off;         /* absolute offset of the weight area in the blob */
    struct wt_slot slots[WT_MAX_SLOTS];
    struct wt_op ops[WT_MAX_OPS];
    const uint8_t* weight_base;  /* points into the caller's blob buffer */
    size_t weight_bytes;
};

/* wt_parse() results (oplist_parse.h:277-292). */
enum {
    WT_OK = 0,
    WT_ERR_SHORT = -1, WT_ERR_MAGIC = -2, WT_ERR_VER = -3, WT_ERR_ENDIAN = -4,
    WT_ERR_NSLOTS = -5, WT_ERR_NOPS = -6, WT_ERR_SLOTS_OVERRUN = -7,
    WT_ERR_WEIGHT_OVERRUN = -8, WT_ERR_OP_TRUNC = -9, WT_ERR_OPCODE = -10,
    WT_ERR_ARITY = -11, WT_ERR_BAD_REF = -12, WT_ERR_ALIGN = -13
};

/* Parses and bounds-checks a blob. `out` is valid only when WT_OK is returned;
 * it keeps pointers into `buf`, which must outlive it.
 * Replaces wt_parse (kernels/src/runtime/oplist_parse.c:86-169). */
int wt_parse(const uint8_t* buf, size_t size, struct wt_blob* out);

/* Short English text for a wt_parse() result (oplist_parse.c:171-189). */
const char* wt_err_str(int rc);

static inline uint32_t wt_rd_u32(const uint8_t* p) {
    return (uint32_t)p[0] | ((uint32_t)p[1] << 8) | ((uint32_t)p[2] << 16) | ((uint32_t)p[3] << 24);
}
static inline uint16_t wt_rd_u16(const uint8_t* p) {
    return (uint16_t)(p[0] | (p[1] << 8));
}

#ifdef __cplusplus
}
#endif
#endif
