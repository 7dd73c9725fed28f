// Planning of the row-count opcodes (wtop_format.h): validation, temp sizes for the blob's largest counts, launches
// that take their row count from the run (rows_of).
#include <cstdio>
#include <cstring>
#include "launchers_rows.h"
#include "planner.h"

namespace gehtp {

namespace {

float from_bits(uint32_t u) { float f; std::memcpy(&f, &u, 4); return f; }

uint32_t max_of(uint32_t arg) { return arg == WT_ROWS_AUTO ? g.max_rows : arg == WT_SEL_AUTO ? g.max_sel : arg; }

// temp sized for the largest count of `rows_arg`, reported at the size of the run
uint8_t* temp_rows(Planner& P, uint32_t id, uint32_t rows_arg, uint64_t row_bytes, PlanOp& p) {
    if (row_bytes * max_of(rows_arg) > 0xFFFFFFFFull) return nullptr;
    uint8_t* t = P.temp_get(id, row_bytes * max_of(rows_arg), p);
    for (int k = 0; k < 2; k++)
        if (p.out_id[k] == id) { p.out_row_bytes[k] = (uint32_t)row_bytes; p.out_rows_arg[k] = rows_arg; }
    return t;
}

// Bytes of a slot that holds data; 0 when `arg` is no such slot.
uint64_t slot_bytes(const wt_blob* b, uint32_t arg) {
    if (!(arg & 0x8000u) || (arg & 0x7FFFu) >= b->n_slots) return 0;
    return b->slots[arg & 0x7FFFu].len;
}

int state_index(uint32_t arg) {
    if ((arg & 0xE000u) != WT_REF_STATE_FLAG || (arg & 0x1FFFu) >= g.n_states) return -1;
    return (int)(arg & 0x1FFFu);
}

// bytes a temp operand was last planned with
bool temp_holds(const Planner& P, uint32_t arg, uint64_t bytes) {
    if (arg & 0xC000u) return true;
    return arg < kMaxTemps && P.last[arg] >= bytes;
}

}  // namespace

void plan_rows_op(Planner& P, const wt_op& op, PlanOp& p) {
    const wt_blob* b = P.b;
    const uint32_t* a = op.args;
    p.engine = WT_ENG_HVX;
    auto bad_rows = [&](uint32_t r) { return max_of(r) == 0; };
    p.rows_args = std::make_shared<RowsArgs>();
    switch (op.opcode) {
    case OP_EMBED_ROWS: {
        const uint32_t rows = a[4], width = a[5], vocab = a[6];
        const bool bf = a[7] == WT_DT_BF16;
        const float scale = from_bits(a[8]);
        const uint32_t es = bf ? 2u : 4u, ld = a[9] ? a[9] : width, col = a[10];
        if (bad_rows(rows) || !width || !vocab || (uint64_t)col + width > ld) FAIL("embed shape");
        if (slot_bytes(b, a[0]) != (uint64_t)vocab * width * 2u) FAIL("embed table size");
        const uint16_t* tab = (const uint16_t*)P.ref(a[0]);
        const int32_t* ids = (const int32_t*)P.ref(a[1]);
        if ((a[1] & 0x8000u) && slot_bytes(b, a[1]) < (uint64_t)max_of(rows) * 4u) FAIL("embed ids too short");
        float* x = (float*)temp_rows(P, a[2], rows, (uint64_t)width * 4u, p);
        uint8_t* act = a[3] ? temp_rows(P, a[3], rows, (uint64_t)ld * es, p) : nullptr;
        if (!tab || !ids || !x || (a[3] && !act)) FAIL("embed ref fail");
        if (act) act += (size_t)col * es;
        if (P.build) p.launch = [=](cudaStream_t st) { k_embed_rows(st, tab, ids, x, act, ld, rows_of(rows), width, vocab, scale, bf); };
        return;
    }
    case OP_LINEAR: {
        const uint32_t rows = a[3], K = a[4], N = a[5], fl = a[6], xc = a[7];
        LinearArgs l{};
        l.K = K; l.N = N; l.xs = a[8] ? a[8] : K; l.ys = N; l.rows_arg = rows;
        l.x_bf16 = fl & WT_LIN_X_BF16; l.y_bf16 = fl & WT_LIN_Y_BF16; l.relu2 = fl & WT_LIN_RELU2; l.gelu_gate = fl & WT_LIN_GELU_GATE;
        if (l.y_bf16 && !l.x_bf16) FAIL("linear: bf16 output of fp32 input");
        if (l.gelu_gate) {
            if ((N & 1u) || l.relu2 || a[9] || l.y_bf16 != l.x_bf16) FAIL("linear: gated form n%u flags %u", N, fl);
            l.ys = N / 2;
        }
        const uint32_t xe = l.x_bf16 ? 2u : 4u;
        if (bad_rows(rows) || !K || !N || (uint64_t)xc + K > l.xs) FAIL("linear shape k%u n%u col%u stride%u", K, N, xc, l.xs);
        if (slot_bytes(b, a[1]) != (uint64_t)K * N * 2u) FAIL("linear weight size");
        const uint8_t* x = P.ref(a[0]);
        if (!temp_holds(P, a[0], (uint64_t)max_of(rows) * l.xs * xe)) FAIL("linear input too small");
        l.w = (const uint16_t*)P.ref(a[1]);
        l.bias = a[9] ? (const float*)P.ref(a[9]) : nullptr;
        if (a[9] && slot_bytes(b, a[9]) != (uint64_t)N * 4u) FAIL("linear bias size");
        l.y = temp_rows(P, a[2], rows, (uint64_t)l.ys * (l.y_bf16 ? 2u : 4u), p);
        if (!x || !l.w || !l.y || (a[9] && !l.bias)) FAIL("linear ref fail");
        l.x = x + (size_t)xc * xe;
        p.engine = WT_ENG_HMX;
        p.rows_args->lin = l;
        if (P.build) p.launch = [=](cudaStream_t st) { k_linear(st, l, rows_of(rows), !g.opt_fuse || g.exact_ops, g.d_status); };
        return;
    }
    case OP_NORM_RESID: {
        NormResidArgs n{};
        const uint32_t rows = a[5], fl = a[7];
        n.width = a[6]; n.rows_arg = rows; n.eps = from_bits(a[8]); n.base = (fl & 1u) ? 1.0f : 0.0f;
        n.act_bf16 = fl & 2u; n.y_bf16 = fl & 4u;
        if (bad_rows(rows) || !n.width) FAIL("norm shape");
        if (slot_bytes(b, a[1]) != (uint64_t)n.width * 4u) FAIL("norm weight size");
        n.y = P.ref(a[0]);
        n.w = (const float*)P.ref(a[1]);
        if (!temp_holds(P, a[0], (uint64_t)max_of(rows) * n.width * (n.y_bf16 ? 2u : 4u))) FAIL("norm input too small");
        if (a[2]) { n.x = (const float*)P.ref(a[2]); if (!n.x || !temp_holds(P, a[2], (uint64_t)max_of(rows) * n.width * 4u)) FAIL("norm residual ref fail"); }
        if (a[3]) { n.x_out = (float*)temp_rows(P, a[3], rows, (uint64_t)n.width * 4u, p); if (!n.x_out) FAIL("norm out fail"); }
        if (a[4]) { n.act = temp_rows(P, a[4], rows, (uint64_t)n.width * (n.act_bf16 ? 2u : 4u), p); if (!n.act) FAIL("norm out fail"); }
        if (!n.y || !n.w) FAIL("norm ref fail");
        p.rows_args->norm = n;
        if (P.build) p.launch = [=](cudaStream_t st) { k_norm_resid(st, n, rows_of(rows)); };
        return;
    }
    case OP_TANH_RESID: {
        TanhResidArgs n{};
        const uint32_t rows = a[6], fl = a[8], col = a[10];
        n.width = a[7]; n.rows_arg = rows; n.act_bf16 = fl & 2u; n.y_bf16 = fl & 4u; n.act_ld = a[9] ? a[9] : n.width;
        const uint32_t es = n.act_bf16 ? 2u : 4u;
        const uint64_t pb = (4u + 2u * (uint64_t)n.width) * 4u;
        if (bad_rows(rows) || !n.width || (uint64_t)col + n.width > n.act_ld) FAIL("tanh norm shape");
        if ((a[1] && slot_bytes(b, a[1]) != pb) || (a[4] && slot_bytes(b, a[4]) != pb)) FAIL("tanh norm parameter size");
        n.y = P.ref(a[0]);
        if (!n.y || !temp_holds(P, a[0], (uint64_t)max_of(rows) * n.width * (n.y_bf16 ? 2u : 4u))) FAIL("tanh norm input too small");
        if (a[1]) { n.p = (const float*)P.ref(a[1]); if (!n.p) FAIL("tanh norm ref fail"); }
        if (a[4]) { n.next = (const float*)P.ref(a[4]); if (!n.next) FAIL("tanh norm ref fail"); }
        if (a[2]) { n.x = (const float*)P.ref(a[2]); if (!n.x || !temp_holds(P, a[2], (uint64_t)max_of(rows) * n.width * 4u)) FAIL("tanh norm residual ref fail"); }
        if (a[3]) { n.x_out = (float*)temp_rows(P, a[3], rows, (uint64_t)n.width * 4u, p); if (!n.x_out) FAIL("tanh norm out fail"); }
        if (a[5]) {
            uint8_t* act = temp_rows(P, a[5], rows, (uint64_t)n.act_ld * es, p);
            if (!act) FAIL("tanh norm out fail");
            n.act = act + (size_t)col * es;
        }
        p.rows_args->tanh = n;
        if (P.build) p.launch = [=](cudaStream_t st) { k_tanh_resid(st, n, rows_of(rows)); };
        return;
    }
    case OP_PICK_ROWS: {
        const uint32_t rows = a[4], width = a[5];
        if (bad_rows(rows) || !width) FAIL("pick shape");
        const float* x = (const float*)P.ref(a[0]);
        const int32_t* idx = (const int32_t*)P.ref(a[1]);
        if ((a[1] & 0x8000u) && slot_bytes(b, a[1]) < ((uint64_t)a[2] + max_of(rows)) * 4u) FAIL("pick index too short");
        const uint32_t x_rows = (a[0] & 0xC000u) ? 0u : (uint32_t)(P.last[a[0] & 0x3FFFu] / ((uint64_t)width * 4u));
        float* out = (float*)temp_rows(P, a[3], rows, (uint64_t)width * 4u, p);
        if (!x || !idx || !out || !x_rows) FAIL("pick ref fail");
        const int32_t* id0 = idx + a[2];
        TanhResidArgs& t = p.rows_args->tanh;             // the picked rows, for a norm fused behind
        t.y = x; t.idx = id0; t.y_rows = x_rows;
        if (P.build) p.launch = [=](cudaStream_t st) { k_pick_rows(st, x, id0, out, rows_of(rows), width, x_rows); };
        return;
    }
    case OP_LATENT_APPEND: case OP_LATENT_ATTEND: {
        const bool app = op.opcode == OP_LATENT_APPEND;
        LatentArgs l{};
        l.rows_arg = a[6]; l.heads = a[7]; l.dim = a[8]; l.rot = a[9];
        l.vdim = app ? 0 : a[10]; l.rank = app ? a[10] : a[11];
        l.bf16 = (app ? a[12] : a[13]) == WT_DT_BF16;
        const uint32_t es = l.bf16 ? 2u : 4u, rows = l.rows_arg;
        const uint64_t mr = max_of(rows), qrow = (uint64_t)l.heads * (l.dim + l.rot);
        if (bad_rows(rows) || !l.heads || !l.dim || !l.rank || (l.rot & 1u) || (!app && !l.vdim)) FAIL("latent shape");
        const int si = state_index(app ? a[5] : a[2]);
        if (si < 0) FAIL("latent state ref bad");
        const uint32_t row_bytes = l.ls() * es;
        if (g.st_bytes[si] % row_bytes) FAIL("latent state %d has %u bytes, rows of %u", si, g.st_bytes[si], row_bytes);
        KvGeom& kv = g.kv[si];
        if (kv.ready && kv.posmap) FAIL("latent state %d is a KV ring", si);
        kv.ready = true; kv.slot_bytes = row_bytes; kv.nslots = g.st_bytes[si] / row_bytes;
        l.state = g.st_buf[si]; l.counter = g.d_st_count + si; l.nslots = kv.nslots; l.state_idx = (uint32_t)si;
        l.status = g.d_status;
        if (app) {
            l.eps = from_bits(a[11]);
            l.y = P.ref(a[0]); l.norm_w = (const float*)P.ref(a[1]);
            l.rope = l.rot ? (const float*)P.ref(a[2]) : nullptr;
            if (slot_bytes(b, a[1]) != (uint64_t)l.rank * 4u) FAIL("latent norm weight size");
            if (l.rot && slot_bytes(b, a[2]) < (uint64_t)kv.nslots * l.rot * 4u) FAIL("latent rotary table shorter than the state");
            if (!temp_holds(P, a[0], mr * l.y_cols() * es)) FAIL("latent input too small");
            l.q = temp_rows(P, a[3], rows, qrow * es, p);
            l.gate = (float*)temp_rows(P, a[4], rows, (uint64_t)l.heads * 4u, p);
            if (!l.y || !l.norm_w || (l.rot && !l.rope) || !l.q || !l.gate) FAIL("latent ref fail");
            p.pos_append_state = si;
            if (P.build) p.launch = [=](cudaStream_t st) { k_latent_append(st, l, rows_of(rows)); };
        } else {
            l.scale = from_bits(a[12]);
            l.q = (void*)P.ref(a[0]); l.gate = (float*)P.ref(a[1]);
            if (!temp_holds(P, a[0], mr * qrow * es) || !temp_holds(P, a[1], mr * l.heads * 4u)) FAIL("latent input too small");
            if (slot_bytes(b, a[3]) != (uint64_t)l.heads * (l.dim + l.vdim) * l.rank * 2u) FAIL("latent kv weight size");
            l.w_kv = (const uint16_t*)P.ref(a[3]);
            l.out = temp_rows(P, a[4], rows, (uint64_t)l.heads * l.vdim * es, p);
            l.work = (float*)P.temp_get(a[5], latent_work_floats(l, (uint32_t)mr) * 4u, p);
            if (!l.q || !l.gate || !l.w_kv || !l.out || !l.work) FAIL("latent ref fail");
            p.engine = WT_ENG_HMX;
            // runs that may be captured take the kernel that reads the position count on the device
            if (P.build) p.launch = [=](cudaStream_t st) {
                const uint32_t n = rows_of(rows);
                k_latent_attend(st, l, n, g.st_count[l.state_idx], !g.opt_fuse || g.exact_ops || n <= kGraphRows);
            };
        }
        p.rows_args->lat = l;
        return;
    }
    case OP_HEADS_APPEND: case OP_WINDOW_ATTEND: {
        const bool app = op.opcode == OP_HEADS_APPEND;
        WindowArgs w{};
        const uint32_t rows = w.rows_arg = a[app ? 5 : 4];
        w.heads = a[app ? 6 : 5]; w.kv_heads = a[app ? 7 : 6]; w.dim = a[app ? 8 : 7]; w.vdim = a[app ? 9 : 8];
        w.y_cols = a[12]; w.bf16 = a[app ? 14 : 13] == WT_DT_BF16;
        const uint32_t es = w.bf16 ? 2u : 4u;
        const uint64_t mr = max_of(rows), qrow = (uint64_t)w.heads * w.dim, orow = (uint64_t)w.heads * w.vdim;
        if (bad_rows(rows) || !w.heads || !w.kv_heads || w.heads % w.kv_heads || !w.dim || !w.vdim) FAIL("window heads shape");
        const int si = state_index(app ? a[4] : a[2]);
        if (si < 0) FAIL("window state ref bad");
        const uint32_t row_bytes = w.row() * es;
        if (g.st_bytes[si] % row_bytes || g.st_bytes[si] / row_bytes < mr) FAIL("window state %d has %u bytes, rows of %u", si, g.st_bytes[si], row_bytes);
        KvGeom& kv = g.kv[si];
        if (kv.ready && kv.posmap) FAIL("window state %d is a KV ring of another kind", si);
        w.state = g.st_buf[si]; w.counter = g.d_st_count + si; w.ring = g.st_bytes[si] / row_bytes; w.state_idx = (uint32_t)si; w.status = g.d_status;
        if (app) {
            w.rot = a[10]; w.eps = from_bits(a[11]); w.positions = a[13];
            if ((w.rot & 1u) || w.rot > w.dim || !w.positions) FAIL("window rotation %u of %u", w.rot, w.dim);
            if (w.y_cols < w.min_cols() || !temp_holds(P, a[0], mr * w.y_cols * es)) FAIL("window input too small");
            if (a[1] && slot_bytes(b, a[1]) != (uint64_t)w.dim * 8u) FAIL("window norm weight size");
            if (w.rot && slot_bytes(b, a[2]) < (uint64_t)w.positions * w.rot * 4u) FAIL("window rotary table too short");
            w.y = P.ref(a[0]);
            w.norms = a[1] ? (const float*)P.ref(a[1]) : nullptr;
            w.rope = w.rot ? (const float*)P.ref(a[2]) : nullptr;
            w.q = temp_rows(P, a[3], rows, qrow * es, p);
            if (!w.y || (a[1] && !w.norms) || (w.rot && !w.rope) || !w.q) FAIL("window ref fail");
            kv.ready = true; kv.slot_bytes = row_bytes; kv.nslots = w.positions;      // room is a matter of positions, not of ring rows
            p.pos_append_state = si;
            if (P.build) p.launch = [=](cudaStream_t st) { k_heads_append(st, w, rows_of(rows)); };
        } else {
            w.window = a[9] < 0x40000000u ? a[9] : 0x40000000u; w.scale = from_bits(a[10]); w.gate_col = a[11];
            const bool gate = w.gate_col != 0xFFFFFFFFu;
            if (!w.window) FAIL("window of no positions");
            // a run's rows are appended before they attend: the ring holds them and the windows behind the first of them,
            // unless no position is ever overwritten
            if (kv.ready && kv.nslots > w.ring && (uint64_t)w.window - 1u + mr > w.ring) FAIL("window %u and %llu rows exceed a ring of %u", w.window, (unsigned long long)mr, w.ring);
            if (gate && (uint64_t)w.gate_col + orow > w.y_cols) FAIL("window gate columns");
            w.q = (void*)P.ref(a[0]);
            if (!w.q || !temp_holds(P, a[0], mr * qrow * es)) FAIL("window input too small");
            if (gate) { w.y = P.ref(a[1]); if (!w.y || !temp_holds(P, a[1], mr * w.y_cols * es)) FAIL("window gate too small"); }
            w.out = temp_rows(P, a[3], rows, orow * es, p);
            if (!w.out) FAIL("window ref fail");
            p.engine = WT_ENG_HMX;
            if (P.build) p.launch = [=](cudaStream_t st) { k_window_attend(st, w, rows_of(rows), !g.opt_fuse || g.exact_ops); };
        }
        p.rows_args->win = w;
        return;
    }
    case OP_SHORT_CONV: {
        DeltaArgs d{};
        const uint32_t rows = a[4], C = a[5];
        d.rows_arg = rows; d.taps = a[6]; d.ys = a[7]; d.bf16 = a[8] == WT_DT_BF16;
        // expressed through the channel count alone: heads of one value channel each
        d.kv_heads = 0; d.heads = C; d.vdim = 1; d.dim = 0;
        if (bad_rows(rows) || !C || !d.taps || d.ys < C) FAIL("short conv shape");
        const int si = state_index(a[2]);
        // two banks of the last taps - 1 inputs: a run reads one and writes the other
        if (si < 0 || g.st_bytes[si] < (d.taps > 1 ? (uint64_t)2 * (d.taps - 1) * C * 4u : 4u)) FAIL("short conv state bad");
        g.kv[si].ready = true; g.kv[si].slot_bytes = 4; g.kv[si].nslots = 0xFFFFFFFFu;
        if (slot_bytes(b, a[1]) != (uint64_t)C * d.taps * 4u) FAIL("short conv weight size");
        d.y = P.ref(a[0]); d.conv_w = (const float*)P.ref(a[1]);
        if (!temp_holds(P, a[0], (uint64_t)max_of(rows) * d.ys * (d.bf16 ? 2u : 4u))) FAIL("short conv input too small");
        d.conv_state = (float*)g.st_buf[si]; d.conv_count = g.d_st_count + si;
        d.qkv = (float*)temp_rows(P, a[3], rows, (uint64_t)C * 4u, p);
        if (!d.y || !d.conv_w || !d.qkv) FAIL("short conv ref fail");
        p.rows_args->del = d;
        if (P.build) p.launch = [=](cudaStream_t st) { k_short_conv(st, d, rows_of(rows)); };
        return;
    }
    case OP_CHANNEL_DELTA: {
        DeltaArgs d{};
        const uint32_t rows = a[8];
        d.rows_arg = rows; d.heads = a[9]; d.kv_heads = a[10]; d.dim = a[11]; d.vdim = a[12]; d.b_col = a[13]; d.ys = a[14];
        d.bf16 = a[15] == WT_DT_BF16;
        const uint64_t mr = max_of(rows);
        if (bad_rows(rows) || !d.heads || !d.kv_heads || d.heads % d.kv_heads || !d.dim || !d.vdim || d.b_col + d.heads > d.ys) FAIL("channel delta shape");
        if (d.dim > 512) FAIL("channel delta: key dim %u above 512", d.dim);
        const int si = state_index(a[5]);
        if (si < 0 || g.st_bytes[si] < (uint64_t)d.heads * d.dim * d.vdim * 4u) FAIL("channel delta state bad");
        if (slot_bytes(b, a[3]) != (uint64_t)d.heads * 4u || slot_bytes(b, a[4]) != (uint64_t)d.heads * d.dim * 4u) FAIL("channel delta constants size");
        d.qkv = (float*)P.ref(a[0]); d.a = (const float*)P.ref(a[1]); d.y = P.ref(a[2]);
        if (!temp_holds(P, a[0], mr * d.channels() * 4u) || !temp_holds(P, a[1], mr * d.heads * d.dim * 4u) ||
            !temp_holds(P, a[2], mr * d.ys * (d.bf16 ? 2u : 4u))) FAIL("channel delta input too small");
        d.a_log = (const float*)P.ref(a[3]); d.dt_bias = (const float*)P.ref(a[4]);
        d.S = (float*)g.st_buf[si];
        d.o = (float*)temp_rows(P, a[6], rows, (uint64_t)d.heads * d.vdim * 4u, p);
        d.work = (float*)P.temp_get(a[7], delta_work_floats(d, (uint32_t)mr) * 4u, p);
        if (!d.qkv || !d.a || !d.y || !d.a_log || !d.dt_bias || !d.o || !d.work) FAIL("channel delta ref fail");
        p.rows_args->del = d;
        if (P.build) p.launch = [=](cudaStream_t st) { k_channel_delta(st, d, rows_of(rows)); };
        return;
    }
    case OP_GATED_NORM: {
        DeltaArgs d{};
        const uint32_t rows = a[4];
        d.rows_arg = rows; d.heads = a[5]; d.vdim = a[6]; d.eps = from_bits(a[7]); d.bf16 = a[8] == WT_DT_BF16;
        const uint64_t mr = max_of(rows), n = (uint64_t)d.heads * d.vdim;
        if (bad_rows(rows) || !n) FAIL("gated norm shape");
        if (slot_bytes(b, a[1]) != (uint64_t)d.vdim * 4u) FAIL("gated norm weight size");
        d.o = (float*)P.ref(a[0]); d.norm_w = (const float*)P.ref(a[1]); d.gate = (const float*)P.ref(a[2]);
        if (!temp_holds(P, a[0], mr * n * 4u) || !temp_holds(P, a[2], mr * n * 4u)) FAIL("gated norm input too small");
        d.out = temp_rows(P, a[3], rows, n * (d.bf16 ? 2u : 4u), p);
        if (!d.o || !d.norm_w || !d.gate || !d.out) FAIL("gated norm ref fail");
        p.rows_args->del = d;
        if (P.build) p.launch = [=](cudaStream_t st) { k_gated_norm(st, d, rows_of(rows)); };
        return;
    }
    case OP_ARGMAX_ROWS: {
        const uint32_t rows = a[2], n = a[3];
        if (bad_rows(rows) || !n) FAIL("argmax shape");
        const float* x = (const float*)P.ref(a[0]);
        if (!temp_holds(P, a[0], (uint64_t)max_of(rows) * n * 4u)) FAIL("argmax input too small");
        int32_t* out = (int32_t*)temp_rows(P, a[1], rows, 4u, p);
        if (!x || !out) FAIL("argmax ref fail");
        if (P.build) p.launch = [=](cudaStream_t st) { k_argmax_rows_f32(st, x, out, rows_of(rows), n); };
        return;
    }
    case OP_STATE_ADVANCE: {
        const uint32_t first = a[0], n = a[1], rows = a[2];
        if (!n || first + n > g.n_states || bad_rows(rows)) FAIL("state advance range");
        p.adv_first = first; p.adv_n = n; p.adv_rows = rows;
        uint32_t* ctr = g.d_st_count + first;
        if (P.build) p.launch = [=](cudaStream_t st) { k_state_advance(st, ctr, n, rows_of(rows)); };
        return;
    }
    default:
        FAIL("opcode %u unhandled", (unsigned)op.opcode);
    }
}

}  // namespace gehtp
