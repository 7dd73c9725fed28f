"""Supevik: a decoder of window attention layers with a looped middle, written as a row-count runlist.

Every sublayer has a norm in front and one behind it, and the norm is element by element: tanh(alpha z) w + b. Queries and
keys are RMS-normed per head and turned by YaRN-scaled rotations, attention sees a window of positions, its output is gated
element by element. A range of layers runs several times over with the same weights, each pass with caches of its own and
entered through a projection of the stream beside the embedding. Sizes and constants come from config.json.
"""
from dataclasses import dataclass, field

from .rowlists import RowsEmitter, up


@dataclass
class Layer:
    type: str
    mixer: dict
    mlp: dict = None


@dataclass
class SupevikConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: list = field(default_factory=list)
    loop: tuple = None               # (start, stop, times)
    name: str = "Supevik"

    @classmethod
    def from_json(cls, c):
        layers = []
        for i, e in enumerate(c["layers"]):
            if e["type"] not in MIXERS:
                raise ValueError("layer %d: mixer %r" % (i, e["type"]))
            mlp = e.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError("layer %d: feed-forward %r" % (i, mlp["kind"]))
            layers.append(Layer(e["type"], e["mixer"], mlp))
        loop = c.get("loop")
        if loop is not None:
            loop = (loop["start"], loop["stop"], loop["times"])
            if not (0 <= loop[0] < loop[1] <= len(layers) and loop[2] >= 1):
                raise ValueError("loop %r of %d layers" % (loop, len(layers)))
        return cls(c["vocab"], c["width"], c["norm"]["eps"], c["embedding"]["scale"], layers, loop)

    def runs(self):
        """Layer runs in order: (layer, True where a pass of the loop begins)."""
        n = len(self.layers)
        start, stop, times = self.loop or (n, n, 0)
        out = [(i, False) for i in range(start)]
        for _ in range(times):
            out += [(i, i == start) for i in range(start, stop)]
        return out + [(i, False) for i in range(stop, n)]


def _attention(e, cfg, t, pre, m, x):
    W, H, G, D, V = cfg.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot, window = m["rot"], m["mask"]["size"]
    if H % G or rot["dims"] > D or rot["dims"] % 2 or window < 1:
        raise ValueError("%s: %d heads over %d, rotation of %d in %d dimensions, window %d" % (pre, H, G, rot["dims"], D, window))
    shapes = {"q": (H * D, W), "k": (G * D, W), "v": (G * V, W), "q.b": (H * D,), "k.b": (G * D,), "v.b": (G * V,),
              "q.norm": (D,), "k.norm": (D,), "g": (H * V, W), "o": (W, H * V)}
    w = {n.replace(".", "_"): (lambda n=n, s=s: t.bf16(pre + "mix." + n, s)) for n, s in shapes.items()}
    return e.window_attention(pre, x, W, H, G, D, V, window, rot, m["scale"], cfg.eps, w)


MIXERS = {"attention": _attention}


def build_runlist(cfg, t, dtype="bfloat16", max_tokens=2048, max_rows=2048, max_sel=64):
    """(blob, manifest) of a model: `t` holds the tensors by name (checkpoint.Tensors). max_tokens: positions a sequence may
    have; max_rows: token rows of the largest run; max_sel: rows whose logits one run can give."""
    nslots = up(max(max_tokens, 64), 64)
    max_rows = min(max_rows, nslots)
    max_sel = min(max_sel, max_rows)
    e = RowsEmitter(dtype, nslots, max_rows, max_sel)
    W, V = cfg.width, cfg.vocab

    def norm(name):
        return e.tanh_params(name, lambda: t.bf16(name + ".alpha"), lambda: t.bf16(name, (W,)), lambda: t.bf16(name + ".b", (W,)))
    # steps between the sublayers: what the stream's next reader wants beside it
    runs = cfg.runs()
    loop_w = e.slot("loop.in", lambda: t.bf16("loop.in", (W, 2 * W))) if cfg.loop else 0
    beside = dict(act="pass", stride=2 * W)         # [stream | embedding], the operand of a pass's entry

    def reader(k):
        """Arguments of tanh_resid for the activations run k starts from."""
        if k == len(runs):
            return dict(act=None)
        i, enter = runs[k]
        return beside if enter else dict(then=norm("l%d.norm1" % i))
    if cfg.loop:
        e.embed(e.slot("embed", lambda: t.bf16("embed", (V, W))), V, W, cfg.embed_scale, col=W, **beside)
    else:
        e.embed(e.slot("embed", lambda: t.bf16("embed", (V, W))), V, W, cfg.embed_scale, act=None)
    if runs:
        e.tanh_resid(e.temp("x"), W, add=False, to_x=False, **reader(0))
    marks = []
    for k, (i, enter) in enumerate(runs):
        layer, pre, act = cfg.layers[i], "l%d." % i, e.temp("act")
        if enter:
            y = e.linear(e.temp("pass"), loop_w, "mix", 2 * W, W, y_act=False)
            e.tanh_resid(y, W, add=False, then=norm(pre + "norm1"))
        y = MIXERS[layer.type](e, cfg, t, pre, layer.mixer, act)
        if layer.mlp is not None:
            e.tanh_resid(y, W, norm(pre + "norm1b"), then=norm(pre + "norm2"))
            ff = layer.mlp["ff"]
            w = {n: (lambda n=n, s=s: t.bf16(pre + "mlp." + n, s)) for n, s in (("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff)))}
            y = e.dense_gelu_gate(pre, act, W, ff, w)
            e.tanh_resid(y, W, norm(pre + "norm2b"), **reader(k + 1))
        else:
            e.tanh_resid(y, W, norm(pre + "norm1b"), **reader(k + 1))
        marks.append(len(e.b.ops))
    logits, token = e.tanh_head(norm("final.norm"), e.slot("head", lambda: t.bf16("head", (V, W))), V, W)
    man = dict(config=cfg.name, dtype=dtype, vocab=V, width=W, nslots=nslots, max_rows=max_rows, max_sel=max_sel, logits_temp=logits,
               token_temp=token, stream_temp=e.temp("x"), layer_end=marks, input_slot=e.face)
    blob = e.finish()
    man["n_ops"] = len(e.b.ops)
    return blob, man
