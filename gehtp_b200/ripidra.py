"""Ripidra: a decoder of latent-attention and channel-decay delta-rule layers, written as a row-count runlist.

There is no norm in front of a sublayer: mixers and feed-forwards take the residual stream, and an RMS norm sits between
their output and the addition (its weights are deviations from one). A layer may borrow another layer's weights while it
keeps its own cache or state. Embedding and head are one table. Sizes and constants come from config.json and from
tensor shapes.
"""
from dataclasses import dataclass, field

from .rowlists import RowsEmitter, up


@dataclass
class Layer:
    type: str
    mixer: dict
    mlp: dict = None
    weights_of: int = None


@dataclass
class RipidraConfig:
    vocab: int
    width: int
    eps: float
    layers: list = field(default_factory=list)
    name: str = "Ripidra"

    @classmethod
    def from_json(cls, c):
        layers = []
        for i, e in enumerate(c["layers"]):
            if e["type"] not in MIXERS:
                raise ValueError("layer %d: mixer %r" % (i, e["type"]))
            mlp = e.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError("layer %d: feed-forward %r" % (i, mlp["kind"]))
            src = e.get("weights_of")
            if src is not None and not (0 <= src < len(c["layers"]) and src != i):
                raise ValueError("layer %d: weights of layer %r" % (i, src))
            layers.append(Layer(e["type"], e["mixer"], mlp, src))
        return cls(c["vocab"], c["width"], c["norm"]["eps"], layers)

    def owner(self, i):
        """The layer whose tensors layer i uses."""
        seen = set()
        while self.layers[i].weights_of is not None:
            if i in seen:
                raise ValueError("layer %d: its weights lead back to itself" % i)
            seen.add(i)
            i = self.layers[i].weights_of
        return i


def _latent(e, cfg, t, pre, m):
    W, H, D, R, V, C = cfg.width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    if m["rot"]["dims"] != R:
        raise ValueError("%s: rotates %d of %d rotary dimensions" % (pre, m["rot"]["dims"], R))
    shapes = {"q": (H * (D + R), W), "dkv": (C + R, W), "dkv.norm": (C,), "uk": (H * D, C), "uv": (H * V, C), "g": (H, W), "o": (W, H * V)}
    w = {n.replace(".", "_"): (lambda n=n, s=s: t.bf16(pre + "mix." + n, s)) for n, s in shapes.items()}
    return e.latent_attention(pre, W, H, D, R, V, C, m["rot"]["base"], m["scale"], cfg.eps, w)


def _delta(e, cfg, t, pre, m):
    W, H, KH, D, V, taps = cfg.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    if H % KH:
        raise ValueError("%s: %d heads over %d key heads" % (pre, H, KH))
    ra, rg = t.shape(pre + "mix.a1")[0], t.shape(pre + "mix.g1")[0]
    shapes = {"q": (KH * D, W), "k": (KH * D, W), "v": (H * V, W), "q.conv": (KH * D, taps), "k.conv": (KH * D, taps),
              "v.conv": (H * V, taps), "b": (H, W), "A_log": (H,), "norm": (V,), "a1": (ra, W), "a2": (H * D, ra),
              "dt_bias": (H * D,), "g1": (rg, W), "g2": (H * V, rg), "o": (W, H * V)}
    w = {n.replace(".", "_").lower(): (lambda n=n, s=s: t.bf16(pre + "mix." + n, s)) for n, s in shapes.items()}
    return e.channel_delta(pre, W, H, KH, D, V, taps, ra, rg, cfg.eps, w)


MIXERS = {"latent_attention": _latent, "channel_delta": _delta}


def build_runlist(cfg, t, dtype="bfloat16", max_tokens=2048, max_rows=2048, max_sel=64):
    """(blob, manifest) of a model: `t` holds the tensors by name (checkpoint.Tensors). max_tokens: positions the caches
    hold; max_rows: token rows of the largest run; max_sel: rows whose logits one run can give."""
    from .checkpoint import bf16_to_f32
    nslots = up(max(max_tokens, 64), 64)
    max_rows = min(max_rows, nslots)
    max_sel = min(max_sel, max_rows)
    e = RowsEmitter(dtype, nslots, max_rows, max_sel)
    W, V = cfg.width, cfg.vocab
    table = e.slot("embed", lambda: t.bf16("embed", (V, W)))
    e.embed(table, V, W)

    def norm(name):
        return e.slot(name, lambda: bf16_to_f32(t.bf16(name, (W,))))
    marks = []
    for i, layer in enumerate(cfg.layers):
        pre = "l%d." % cfg.owner(i)
        e.add_norm(MIXERS[layer.type](e, cfg, t, pre, layer.mixer), norm(pre + "norm1"), W, cfg.eps, True)
        if layer.mlp is not None:
            ff = layer.mlp["ff"]
            w = {n: (lambda n=n, s=s: t.bf16(pre + "mlp." + n, s)) for n, s in (("up", (ff, W)), ("down", (W, ff)))}
            e.add_norm(e.dense_relu2(pre, W, ff, w), norm(pre + "norm2"), W, cfg.eps, True)
        marks.append(len(e.b.ops))
    logits, token = e.head(norm("final.norm"), table, V, W, cfg.eps, True)
    man = dict(config=cfg.name, dtype=dtype, vocab=V, width=W, nslots=nslots, max_rows=max_rows, max_sel=max_sel, logits_temp=logits,
               token_temp=token, stream_temp=e.temp("x"), layer_end=marks, input_slot=e.face)
    blob = e.finish()
    man["n_ops"] = len(e.b.ops)
    return blob, man
