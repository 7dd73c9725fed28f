"""Row-count runlists: one op list that runs any number of token rows of a sequence from the states earlier runs left
(prompts whole or in portions, and single decoded tokens), written with the executor's own row ops.

`RowsEmitter` holds the mechanisms - projections, norms on the residual stream, latent attention, grouped-query attention
over a window, the delta rule with a decay per key channel, dense feed-forwards, the picked-row head - each with its sizes
and constants as arguments; a model design (ripidra.py, supevik.py) strings them together. Activations are bf16 or fp32,
weights bf16, the residual stream fp32.

Temps are named and reused from layer to layer: a layer's intermediate faces share the memory of the layer before.
"""
import math
import struct

import numpy as np

from .checkpoint import bf16_to_f32
from .wtop import COL_ALIGN, DT_BF16, DT_F32, LIN_GELU_GATE, LIN_RELU2, LIN_X_BF16, LIN_Y_BF16, OP, ROWS_AUTO, S, SEL_AUTO, ST, BlobBuilder


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


def yarn_scaling(dims, base, factor, original, fast, slow):
    """(factor on each pair's angle, factor on cosine and sine) of YaRN context extension: pairs that turn more than `fast`
    times over the original context keep their angle, those below `slow` turns have it divided by `factor`."""
    def at(turns):
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(fast)), 0), min(math.ceil(at(slow)), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return ramp / factor + (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rope_halves(positions, dims, base, scaling=None):
    """fp32 [positions][dims / 2][cos, sin] for components i and i + dims / 2 turned by p * base^(-2i / dims); scaling:
    the arguments of yarn_scaling by name."""
    f, mag = np.float64(base) ** (-np.arange(0, dims, 2, dtype=np.float64) / dims), 1.0
    if scaling:
        by, mag = yarn_scaling(dims, base, scaling["factor"], scaling["original"], scaling["fast"], scaling["slow"])
        f = f * by
    ang = np.arange(positions, dtype=np.float64)[:, None] * f
    return (np.stack([np.cos(ang), np.sin(ang)], axis=-1) * mag).astype(np.float32)


RING_ALIGN = 128        # rows of a position ring are a multiple of the largest tile that is read from it


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
    def embed(self, table, vocab, width, scale=1.0, act="act", col=0, stride=0):
        """x = table rows * scale; their activation copy goes to columns `col` .. of temp `act` (None: no copy)."""
        copy = self.temp(act) if act and (self.bf16 or act != "act") else 0
        self.op(OP.EMBED_ROWS, [table, S(self.face), self.temp("x"), copy, ROWS_AUTO, width, vocab, self.dt, bits(scale), stride, col])

    def act(self):
        """The residual stream as projections read it: its bf16 copy, or the stream itself in fp32."""
        return self.temp("act") if self.bf16 else self.temp("x")

    def linear(self, x, w, out, K, N, y_act=True, relu2=False, rows=ROWS_AUTO, col=0, stride=0, bias=0, gelu_gate=False):
        fl = (LIN_X_BF16 if self.bf16 else 0) | (LIN_Y_BF16 if self.bf16 and y_act else 0) | (LIN_RELU2 if relu2 else 0)
        t = self.temp(out)
        self.op(OP.LINEAR, [x, w, t, rows, K, N, fl | (LIN_GELU_GATE if gelu_gate else 0), col, stride, bias])
        return t

    def tanh_params(self, key, alpha, w, b):
        """Slot of an element-wise norm tanh(alpha z) w + b; arguments: zero-argument callables giving bf16 bits."""
        def make():
            a, w_, b_ = (bf16_to_f32(np.asarray(f())).reshape(-1) for f in (alpha, w, b))
            if a.size != 1:
                raise ValueError("%s: %d factors in front of tanh, expected one" % (key, a.size))
            return np.concatenate([a, np.zeros(3, np.float32), w_, b_])
        return self.slot((key, "tanh"), make)

    def tanh_resid(self, y, width, p=0, add=True, to_x=True, then=0, act="act", col=0, stride=0, rows=ROWS_AUTO):
        """x <- x + t(y, p) (add=False: t(y, p)); temp `act` (None: not written) gets t(x, then) from column `col` on."""
        x = self.temp("x")
        self.op(OP.TANH_RESID, [y, p, x if add else 0, x if to_x else 0, then, self.temp(act) if act else 0, rows, width,
                                2 if self.bf16 else 0, stride, col])

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

    def window_attention(self, key, x, width, heads, kv_heads, dim, vdim, window, rot, scale, eps, w):
        """Grouped-query attention of rows x over the last `window` positions. rot: {dims, base, scaling}. w: q, k, v, g, o
        and the biases q_b, k_b, v_b, the head norms q_norm, k_norm (None where the design has none; zero-argument callables)."""
        at, cols = [], 0
        for n in (heads * dim, kv_heads * dim, kv_heads * vdim) + ((heads * vdim,) if w["g"] else ()):
            at.append(cols)
            cols += up(n)

        def bias():
            out = np.zeros(cols, np.float32)
            for a, n in zip(at, ("q_b", "k_b", "v_b")):
                v = bf16_to_f32(w[n]())
                out[a:a + v.size] = v
            return out
        w_in = self.slot((key, "in"), lambda: join_rows([w[n]() for n in "qkvg" if w[n]])[0])
        b_in = self.slot((key, "bias"), bias) if w["q_b"] else 0
        norms = self.slot((key, "norms"), lambda: bf16_to_f32(np.concatenate([w["q_norm"](), w["k_norm"]()]))) if w["q_norm"] else 0
        dims = rot["dims"] if rot else 0
        table = self.slot(("halves", dims, float(rot["base"]), tuple(sorted((rot.get("scaling") or {}).items()))),
                          lambda: rope_halves(self.nslots, dims, rot["base"], rot.get("scaling"))) if dims else 0
        row = up(kv_heads * (dim + vdim))
        ring = min(up(self.nslots, RING_ALIGN), up(window - 1 + self.max_rows, RING_ALIGN))
        st = self._state("cache", ring * row * self.es)
        y = self.linear(x, w_in, "proj", width, cols, bias=b_in)
        q, out = self.temp("q"), self.temp("heads")
        self.op(OP.HEADS_APPEND, [y, norms, table, q, st, ROWS_AUTO, heads, kv_heads, dim, vdim, dims, bits(eps), cols, self.nslots, self.dt])
        self.op(OP.WINDOW_ATTEND, [q, y, st, out, ROWS_AUTO, heads, kv_heads, dim, vdim, window, bits(scale), at[3] if w["g"] else 0xFFFFFFFF, cols, self.dt])
        return self.linear(out, self.slot((key, "o"), w["o"]), "mix", heads * vdim, width, y_act=False)

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

    def dense_gelu_gate(self, key, x, width, ff, w):
        """(gelu(gate x) * up x) through `down`; w: gate, up, down."""
        w_in = self.slot((key, "gate_up"), lambda: np.stack([w["gate"](), w["up"]()], axis=1).reshape(2 * ff, width))
        h = self.linear(x, w_in, "ff", width, 2 * ff, gelu_gate=True)
        return self.linear(h, self.slot((key, "down"), w["down"]), "mix", ff, width, y_act=False)

    def pick(self, width):
        p = self.temp("picked")
        self.op(OP.PICK_ROWS, [self.temp("x"), S(self.face), self.max_rows, p, SEL_AUTO, width])
        return p

    def choose(self, h, table, vocab, width):
        """Logits (fp32) of picked rows h and the greedy choice."""
        logits = self.linear(h, table, "logits", width, vocab, y_act=False, rows=SEL_AUTO)
        tok = self.temp("token")
        self.op(OP.ARGMAX_ROWS, [logits, tok, SEL_AUTO, vocab])
        return logits, tok

    def tanh_head(self, p, table, vocab, width):
        """Picked rows -> element-wise norm -> logits and the greedy choice."""
        self.tanh_resid(self.pick(width), width, add=False, to_x=False, then=p, act="picked_act", rows=SEL_AUTO)
        return self.choose(self.temp("picked_act"), table, vocab, width)

    def head(self, norm_w, table, vocab, width, eps, about_one):
        """Picked rows -> norm -> logits (fp32) and the greedy choice."""
        p, h = self.pick(width), self.temp("picked_act")
        self.op(OP.NORM_RESID, [p, norm_w, 0, 0, h, SEL_AUTO, width, (1 if about_one else 0) | (2 if self.bf16 else 0), bits(eps)])
        return self.choose(h, table, vocab, width)

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
