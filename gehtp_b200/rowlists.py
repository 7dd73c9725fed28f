"""Row-count runlists: one op list that runs any number of token rows of a sequence from the states earlier runs left
(prompts whole or in portions, and single decoded tokens), written with the executor's own row ops.

`RowsEmitter` holds the mechanisms - projections, norms on the residual stream, latent attention, the delta rule with a
decay per key channel, dense feed-forwards, the picked-row head - each with its sizes and constants as arguments; a
model design (ripidra.py) strings them together. Activations are bf16 or fp32, weights bf16, the residual stream fp32.

Temps are named and reused from layer to layer: a layer's intermediate faces share the memory of the layer before.
"""
import struct

import numpy as np

from .checkpoint import bf16_to_f32
from .wtop import COL_ALIGN, DT_BF16, DT_F32, LIN_RELU2, LIN_X_BF16, LIN_Y_BF16, OP, ROWS_AUTO, S, SEL_AUTO, ST, BlobBuilder


def bits(x):
    """fp32 bit pattern of an op argument."""
    return struct.unpack("<I", struct.pack("<f", float(x)))[0]


def up(n, a=COL_ALIGN):
    return (n + a - 1) // a * a


def latent_row(rank, rot):
    """Elements of one cached position: latent, rotated key part, zeros up to a multiple of 16."""
    return up(rank + rot, 16)


def join_rows(parts):
    """Stacks projections [n_i, K] into one, each starting at a multiple of COL_ALIGN rows (zero rows between).
    Returns (weights, start of each part)."""
    out, at, pos = [], [], 0
    for w in parts:
        at.append(pos)
        out.append(w)
        pad = up(w.shape[0]) - w.shape[0]
        if pad:
            out.append(np.zeros((pad, w.shape[1]), w.dtype))
        pos += w.shape[0] + pad
    return np.concatenate(out), at


def rope_pairs(positions, dims, base):
    """fp32 [positions][dims / 2][cos, sin] for neighbouring components turned by p * base^(-2i / dims)."""
    ang = np.arange(positions, dtype=np.float64)[:, None] * np.float64(base) ** (-np.arange(0, dims, 2, dtype=np.float64) / dims)
    return np.stack([np.cos(ang), np.sin(ang)], axis=-1).astype(np.float32)


class RowsEmitter:
    def __init__(self, dtype, nslots, max_rows, max_sel):
        if dtype not in ("bfloat16", "float32"):
            raise ValueError("dtype %r: bfloat16 or float32" % (dtype,))
        self.b = BlobBuilder()
        self.bf16 = dtype == "bfloat16"
        self.dt = DT_BF16 if self.bf16 else DT_F32
        self.es = 2 if self.bf16 else 4
        self.nslots, self.max_rows, self.max_sel = nslots, max_rows, max_sel
        self.names, self.slots, self.tables = {}, {}, {}
        # states: position-counted caches first, then convolution windows (counted in runs), then plain states
        self.caches, self.windows, self.plain = [], [], []
        self._state_args = []        # (op index, arg index, kind, ordinal): state numbers are known at the end
        self.b.add_rows(max_rows, max_sel)
        self.face = self.b.add_ext_in(4 * (max_rows + max_sel))

    # ---- names, slots, states
    def temp(self, name):
        return self.names.setdefault(name, len(self.names) + 1)

    def slot(self, key, make):
        """Slot of a constant; layers that share weights share the slot by its key."""
        if key not in self.slots:
            self.slots[key] = self.b.add_slot(np.ascontiguousarray(make()))
        return S(self.slots[key])

    def rope_table(self, dims, base):
        if dims == 0:
            return 0
        return self.slot(("rope", dims, float(base)), lambda: rope_pairs(self.nslots, dims, base))

    def _state(self, kind, nbytes):
        lst = {"cache": self.caches, "window": self.windows, "plain": self.plain}[kind]
        if nbytes > 0xFFFFFFFF:
            raise ValueError("a state of %d bytes: above 4 GiB" % nbytes)
        lst.append(nbytes)
        return kind, len(lst) - 1

    def op(self, opcode, args):
        args = list(args)
        idx = len(self.b.ops)
        for i, a in enumerate(args):
            if isinstance(a, tuple):
                self._state_args.append((idx, i) + a)
                args[i] = 0
        return self.b.add_op(opcode, args)

    # ---- single ops
    def embed(self, table, vocab, width):
        self.op(OP.EMBED_ROWS, [table, S(self.face), self.temp("x"), self.temp("act") if self.bf16 else 0, ROWS_AUTO, width, vocab, self.dt])

    def act(self):
        """The residual stream as projections read it: its bf16 copy, or the stream itself in fp32."""
        return self.temp("act") if self.bf16 else self.temp("x")

    def linear(self, x, w, out, K, N, y_act=True, relu2=False, rows=ROWS_AUTO, col=0, stride=0):
        fl = (LIN_X_BF16 if self.bf16 else 0) | (LIN_Y_BF16 if self.bf16 and y_act else 0) | (LIN_RELU2 if relu2 else 0)
        t = self.temp(out)
        self.op(OP.LINEAR, [x, w, t, rows, K, N, fl, col, stride])
        return t

    def add_norm(self, y, w, width, eps, about_one):
        """x <- x + norm(y), and the activation copy of x."""
        x = self.temp("x")
        self.op(OP.NORM_RESID, [y, w, x, x, self.temp("act") if self.bf16 else 0, ROWS_AUTO, width,
                                (1 if about_one else 0) | (2 if self.bf16 else 0), bits(eps)])

    # ---- mixers: read the stream, leave the output projection's rows (fp32) in temp "mix"
    def latent_attention(self, key, width, heads, dim, rot, vdim, rank, base, scale, eps, w):
        """w: q, dkv, dkv_norm, uk, uv, g, o (arrays through zero-argument callables, called once per weight set)."""
        ycols = up(heads * (dim + rot)) + up(rank + rot) + up(heads)
        w_in = self.slot((key, "in"), lambda: join_rows([w["q"](), w["dkv"](), w["g"]()])[0])
        w_kv = self.slot((key, "kv"), lambda: np.concatenate([w["uk"](), w["uv"]()]))
        w_o = self.slot((key, "o"), w["o"])
        nw = self.slot((key, "norm"), lambda: bf16_to_f32(w["dkv_norm"]()))
        st = self._state("cache", self.nslots * latent_row(rank, rot) * self.es)
        y = self.linear(self.act(), w_in, "proj", width, ycols)
        q, gate, out = self.temp("q"), self.temp("gate"), self.temp("heads")
        self.op(OP.LATENT_APPEND, [y, nw, self.rope_table(rot, base), q, gate, st, ROWS_AUTO, heads, dim, rot, rank, bits(eps), self.dt])
        self.op(OP.LATENT_ATTEND, [q, gate, st, w_kv, out, self.temp("work"), ROWS_AUTO, heads, dim, rot, vdim, rank, bits(scale), self.dt])
        return self.linear(out, w_o, "mix", heads * vdim, width, y_act=False)

    def channel_delta(self, key, width, heads, kv_heads, dim, vdim, taps, rank_a, rank_g, eps, w):
        """w: q, k, v, q_conv, k_conv, v_conv, b, a_log, norm, a1, a2, dt_bias, g1, g2, o."""
        C = 2 * kv_heads * dim + heads * vdim
        b_col = up(C)
        a_col = b_col + up(heads)
        g_col = a_col + up(rank_a)
        ycols = g_col + up(rank_g)

        def joined():
            m, at = join_rows([np.concatenate([w["q"](), w["k"](), w["v"]()]), w["b"](), w["a1"](), w["g1"]()])
            assert at == [0, b_col, a_col, g_col] and m.shape[0] == ycols
            return m
        w_in = self.slot((key, "in"), joined)
        conv = self.slot((key, "conv"), lambda: bf16_to_f32(np.concatenate([w["q_conv"](), w["k_conv"](), w["v_conv"]()])))
        a2, g2, w_o = self.slot((key, "a2"), w["a2"]), self.slot((key, "g2"), w["g2"]), self.slot((key, "o"), w["o"])
        alog, dtb, nw = (self.slot((key, n), lambda n=n: bf16_to_f32(w[n]())) for n in ("a_log", "dt_bias", "norm"))
        win = self._state("window", max(2 * (taps - 1) * C * 4, 4))
        st = self._state("plain", heads * dim * vdim * 4)
        y = self.linear(self.act(), w_in, "proj", width, ycols)
        a = self.linear(y, a2, "decay", rank_a, heads * dim, y_act=False, col=a_col, stride=ycols)
        g = self.linear(y, g2, "gate_rows", rank_g, heads * vdim, y_act=False, col=g_col, stride=ycols)
        qkv, o, out = self.temp("qkv"), self.temp("read"), self.temp("heads")
        self.op(OP.SHORT_CONV, [y, conv, win, qkv, ROWS_AUTO, C, taps, ycols, self.dt])
        self.op(OP.CHANNEL_DELTA, [qkv, a, y, alog, dtb, st, o, self.temp("work"), ROWS_AUTO, heads, kv_heads, dim, vdim, b_col, ycols, self.dt])
        self.op(OP.GATED_NORM, [o, nw, g, out, ROWS_AUTO, heads, vdim, bits(eps), self.dt])
        return self.linear(out, w_o, "mix", heads * vdim, width, y_act=False)

    def dense_relu2(self, key, width, ff, w):
        h = self.linear(self.act(), self.slot((key, "up"), w["up"]), "ff", width, ff, relu2=True)
        return self.linear(h, self.slot((key, "down"), w["down"]), "mix", ff, width, y_act=False)

    def head(self, norm_w, table, vocab, width, eps, about_one):
        """Picked rows -> norm -> logits (fp32) and the greedy choice."""
        p, h = self.temp("picked"), self.temp("picked_act")
        self.op(OP.PICK_ROWS, [self.temp("x"), S(self.face), self.max_rows, p, SEL_AUTO, width])
        self.op(OP.NORM_RESID, [p, norm_w, 0, 0, h, SEL_AUTO, width, (1 if about_one else 0) | (2 if self.bf16 else 0), bits(eps)])
        logits = self.linear(h, table, "logits", width, vocab, y_act=False, rows=SEL_AUTO)
        tok = self.temp("token")
        self.op(OP.ARGMAX_ROWS, [logits, tok, SEL_AUTO, vocab])
        return logits, tok

    def finish(self):
        """Advances the counters, numbers the states, serialises."""
        nc, nw = len(self.caches), len(self.windows)
        if nc:
            self.op(OP.STATE_ADVANCE, [0, nc, ROWS_AUTO])
        if nw:
            self.op(OP.STATE_ADVANCE, [nc, nw, 1])
        base = {"cache": 0, "window": nc, "plain": nc + nw}
        sizes = self.caches + self.windows + self.plain
        if len(sizes) > 64:
            raise ValueError("%d states: a runlist holds at most 64" % len(sizes))
        if sizes:
            self.b.add_states(sizes)
        for idx, i, kind, k in self._state_args:
            self.b.ops[idx][1][i] = ST(base[kind] + k)
        return self.b.build()
