"""The Supevik design through the engine against the plain statement in supevik_oracle.py: every mechanism alone, whole
prompts against portions and token-by-token decoding, window edges, wrapping position rings, looped layers, generation
through the scheduler."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import supevik_oracle as oracle
from gehtp_b200.checkpoint import ArrayTensors, bf16_to_f32, f32_to_bf16, write_safetensors
from gehtp_b200.registry import Model, load_model
from gehtp_b200.rowlists import RowsEmitter, bits, rope_halves, yarn_scaling
from gehtp_b200.session import Request, Scheduler, Session
from gehtp_b200.wtop import LIN_GELU_GATE, LIN_X_BF16, LIN_Y_BF16, OP, ROWS_AUTO, SEL_AUTO, Engine, EngineError, S, parse_blob

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
YARN = dict(factor=3.0, fast=8.0, slow=1.5, original=200)


def layer(heads=6, kv_heads=2, dim=24, vdim=40, window=19, base=3000.0, rot=12, scaling=YARN, scale=0.23, ff=88):
    r = dict(base=base, dims=rot)
    if scaling:
        r["scaling"] = scaling
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=window), rot=r, scale=scale)
    return dict(type="attention", mixer=m, mlp=dict(kind="dense", ff=ff) if ff else None)


def make(layers, loop=None, vocab=130, width=72, eps=1e-4, emb=3.0, seed=0, sharp=1.0):
    """(config, tensors as float32 holding bf16 values); sharp: factor on the query norm, so that single keys stand out.
    loop: (start, stop, times)."""
    cfg = dict(architecture="Supevik", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=emb), layers=layers)
    if loop:
        cfg["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    rng = np.random.default_rng(seed)
    t = {}

    def put(name, *shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        t[name] = bf16_to_f32(f32_to_bf16(rng.standard_normal(shape).astype(np.float32) * np.float32(std) + np.float32(mean)))

    def norm(name):
        put(name, width, std=0.3, mean=1.0)
        put(name + ".b", width, std=0.2)
        put(name + ".alpha", 1, std=0.1, mean=0.6)
    put("embed", vocab, width, std=0.4)
    put("head", vocab, width)
    norm("final.norm")
    if loop:
        put("loop.in", width, 2 * width)
    for i, e in enumerate(layers):
        p, m = "l%d." % i, e["mixer"]
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if e["mlp"] else ()):
            norm(p + n)
        q = p + "mix."
        for n, c in (("q", H * D), ("k", G * D), ("v", G * V)):
            put(q + n, c, width)
            put(q + n + ".b", c, std=0.4)
        put(q + "q.norm", D, std=0.2 * sharp, mean=sharp)
        put(q + "k.norm", D, std=0.2, mean=1.0)
        put(q + "g", H * V, width)
        put(q + "o", width, H * V)
        if e["mlp"]:
            put(p + "mlp.gate", e["mlp"]["ff"], width)
            put(p + "mlp.up", e["mlp"]["ff"], width)
            put(p + "mlp.down", width, e["mlp"]["ff"])
    return cfg, t


def ids(n, vocab=130, seed=1):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def session(cuda, mt, dtype, **kw):
    kw.setdefault("max_tokens", 512)
    return Session(Model(mt[0], ArrayTensors(mt[1])), dtype, lib=cuda, **kw)


def row_errors(got, want):
    """Error of each row, mean taken off, over the root mean square of all wanted rows."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    return np.sqrt((d ** 2).mean(axis=-1)) / np.sqrt((want ** 2).mean())


def rel(got, want):
    return float(row_errors(got, want).max())


def close(got, want, dtype):
    e = row_errors(got, want)
    return bool(e.max() < 3e-5 if dtype == "float32" else e.max() < 6e-2 and np.median(e) < 2e-2)


def run_cut(s, tok, cut):
    """Logits of every token, fed in portions of the given sizes."""
    s.reset()
    at, rows = 0, []
    for n in cut:
        rows.append(s.feed(tok[at:at + n], range(n)))
        at += n
    assert at == len(tok)
    return np.concatenate(rows)


DTYPES = ["float32", "bfloat16"]
MIX = [layer(), layer(heads=2, kv_heads=2, dim=64, vdim=64, window=150, rot=64, base=500.0, ff=None), layer(heads=3, kv_heads=1, dim=16, vdim=8, window=5)]
LOOP = (1, 3, 2)


# ------------------------------------------------------------------ CPU: oracle, reader, runlist
def test_oracle_mechanisms():
    """The plain statement's own pieces on cases with known answers."""
    assert oracle.window_mask(4, 2).astype(int).tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    assert np.allclose(oracle.tanh_norm(np.array([0.0, 1e9]), 0.5, np.array([2.0, 3.0]), np.array([1.0, -1.0])), [1.0, 2.0])
    z = np.linspace(-6, 6, 25)
    assert np.allclose(oracle.gelu_tanh(z), z * oracle.sigmoid(2 * np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)))
    assert oracle.schedule(dict(layers=[0] * 4, loop=dict(start=1, stop=3, times=2))) == [(0, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    x = np.array([[1.0, 2.0, 3.0, 4.0, 5.0]])
    got = oracle.rotate_halves(x, [1], dict(dims=4, base=100.0))
    c, s, c2, s2 = np.cos(1), np.sin(1), np.cos(0.1), np.sin(0.1)
    assert np.allclose(got, [[c - 3 * s, 2 * c2 - 4 * s2, 3 * c + s, 4 * c2 + 2 * s2, 5]])


@pytest.mark.parametrize("dims,scaling", [(12, None), (12, YARN), (32, dict(factor=8.0, fast=32.0, slow=1.0, original=4096)),
                                          (4, dict(factor=2.0, fast=1e6, slow=1e-6, original=64)), (2, dict(factor=1.0, fast=2.0, slow=2.0, original=10))])
def test_rotation_table(dims, scaling):
    rot = dict(dims=dims, base=700.0, **({"scaling": scaling} if scaling else {}))
    tab = rope_halves(40, dims, 700.0, scaling)
    f, mag = oracle.frequencies(rot)
    a = np.arange(40)[:, None] * f
    assert tab.shape == (40, dims // 2, 2)
    assert np.abs(tab - np.stack([np.cos(a), np.sin(a)], -1) * mag).max() < 1e-6
    if scaling:
        by, m = yarn_scaling(dims, 700.0, scaling["factor"], scaling["original"], scaling["fast"], scaling["slow"])
        assert abs(m - mag) < 1e-12 and (by <= 1.0).all() and (by >= 1.0 / scaling["factor"] - 1e-12).all()


def test_registry_reads_the_config(tmp_path):
    cfg, t = make(MIX, LOOP)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), t)
    m = load_model(str(tmp_path))
    assert m.architecture == "Supevik" and m.config.runs() == oracle.schedule(cfg)
    for bad in (dict(cfg, layers=[dict(layer(), type="other")]), dict(cfg, layers=[dict(layer(), mlp=dict(kind="routed", ff=8))]),
                dict(cfg, loop=dict(start=2, stop=2, times=1)), dict(cfg, loop=dict(start=1, stop=9, times=1)), dict(cfg, loop=dict(start=0, stop=1, times=0))):
        with pytest.raises(ValueError):
            Model(bad, ArrayTensors(t))
    for bad in (layer(heads=5), layer(rot=26), layer(rot=7), layer(window=0)):
        with pytest.raises(ValueError):
            Model(dict(cfg, layers=[bad] + MIX[1:]), ArrayTensors(t)).runlist()
    with pytest.raises(ValueError):                     # a tensor of another shape than the configuration says
        Model(dict(cfg, layers=[layer(vdim=48)] + MIX[1:]), ArrayTensors(t)).runlist()


@pytest.mark.parametrize("dtype", DTYPES)
def test_passes_share_weights_and_own_their_rings(cuda, dtype):
    cfg, t = make(MIX, LOOP)
    blob, man = Model(cfg, ArrayTensors(t)).runlist(dtype, max_tokens=1000, max_rows=40, max_sel=3)
    rc, b = parse_blob(cuda, blob)
    assert rc == 0 and man["nslots"] == 1024
    ops = [(o.opcode, list(o.args[:o.n_args])) for o in b.ops[:b.n_ops]]
    app = [a for c, a in ops if c == OP.HEADS_APPEND]
    # runs: layer 0, (1, 2), (1, 2)
    assert len(app) == 5 and len({a[4] for a in app}) == 5
    assert app[1][1] == app[3][1] != app[0][1] and app[2][1] == app[4][1]
    tanh = [a for c, a in ops if c == OP.TANH_RESID]
    # first norm, per run one or two behind the sublayers, two pass entries, the head's
    assert len(tanh) == 1 + (2 + 1 + 2 + 1 + 2) + 2 + 1
    assert [a for c, a in ops if c == OP.STATE_ADVANCE] == [[0, 5, ROWS_AUTO]]
    # windows of 19 and 5 positions and runs of 40 rows fit in 128 ring rows, 150 take 256
    n, base = np.frombuffer(blob, np.uint8), b.weight_off
    sizes = next(np.frombuffer(n[base + s.offset:base + s.offset + s.len].tobytes(), np.uint32) for s in b.slots[:b.n_slots] if s.addr == 0xFFFFFFFB)
    es = 2 if dtype == "bfloat16" else 4
    assert sizes.tolist() == [5, 128 * 2 * 64 * es] + [256 * 2 * 128 * es, 128 * 24 * es] * 2
    assert cfg["layers"][1]["mlp"] is None and man["layer_end"] == sorted(man["layer_end"]) and len(man["layer_end"]) == 5


def test_row_ops_are_validated(cuda):
    e = RowsEmitter("float32", 64, 8, 2)
    tab = e.slot("t", lambda: np.zeros((4, 8), np.uint16))
    e.embed(tab, 4, 8)
    for op, args in ((OP.TANH_RESID, [1, S(99), 0, 1, 0, 0, ROWS_AUTO, 8, 0, 0, 0]), (OP.HEADS_APPEND, [1, 0, S(99)] + [0] * 12),
                     (OP.LINEAR, [1, tab, 2, ROWS_AUTO, 8, 4, 0, 0, 0, S(99)])):
        e.b.ops[1:] = [(op, args)]
        assert parse_blob(cuda, e.b.build())[0] == -12
        e.b.ops[1:] = [(op, args[:-1])]
        assert parse_blob(cuda, e.b.build())[0] == -11


# ------------------------------------------------------------------ GPU: single ops
def run_ops(cuda, emit, rows, sel=1, dtype="bfloat16", vocab=512, width=64, fuse=1, max_rows=512):
    """Runs EMBED_ROWS of ids 0..rows-1 and the ops of emit(emitter, table slot); returns (engine, emitter, x rows)."""
    cuda.gehtp_cuda_set_fusion(fuse)
    tab = bf16_to_f32(f32_to_bf16(np.random.default_rng(3).standard_normal((vocab, width)).astype(np.float32)))
    e = RowsEmitter(dtype, 512, max_rows, 8)
    t = e.slot("t", lambda: f32_to_bf16(tab))
    emit(e, t)
    eng = Engine(cuda, e.finish())
    eng.set_rows(rows, sel)
    face = np.zeros(max_rows + 8, np.int32)
    face[:rows] = np.arange(rows)
    face[max_rows:max_rows + sel] = (np.arange(sel) * 7 + rows - 1) % rows
    eng.run_io(face, e.temp("x"), None)
    return eng, e, tab[:rows]


@pytest.fixture(autouse=True)
def fusion_on(cuda):
    yield
    cuda.gehtp_cuda_set_fusion(1)


def faces(eng, e, name, rows, bf):
    a = eng.temp(e.temp(name), np.uint16 if bf else np.float32).reshape(rows, -1)
    return bf16_to_f32(a) if bf else a


def params(rng, width):
    a, w, b = np.float32(0.7), rng.standard_normal(width).astype(np.float32), rng.standard_normal(width).astype(np.float32)
    return np.concatenate([[a], np.zeros(3, np.float32), w, b]).astype(np.float32), (float(a), w.astype(np.float64), b.astype(np.float64))


@pytest.mark.gpu
@pytest.mark.parametrize("width", [64, 50, 1028, 2560])
@pytest.mark.parametrize("dtype", DTYPES)
def test_scaled_embedding_beside_the_stream(cuda, width, dtype):
    """Scaled rows in the right half of a joined operand, the stream written to its left half."""
    def emit(e, t):
        e.embed(t, 512, width, 2.5, act="pair", col=width, stride=2 * width)
        e.tanh_resid(e.temp("x"), width, add=False, to_x=False, act="pair", stride=2 * width)
    eng, e, x = run_ops(cuda, emit, 9, dtype=dtype, width=width)
    x = x * np.float32(2.5)
    assert np.array_equal(eng.temp(e.temp("x"), np.float32).reshape(9, width), x)
    pair = faces(eng, e, "pair", 9, e.bf16)
    want = bf16_to_f32(f32_to_bf16(x)) if e.bf16 else x
    assert np.array_equal(pair[:, :width], want) and np.array_equal(pair[:, width:], want)
    eng.shutdown()


@pytest.mark.gpu
@pytest.mark.parametrize("width", [64, 50, 1028, 2560])
@pytest.mark.parametrize("dtype", DTYPES)
def test_tanh_norms_and_residual(cuda, width, dtype):
    rng = np.random.default_rng(width)
    (p, pv), (q, qv) = params(rng, width), params(rng, width)
    rows, sel = 9, 4

    def emit(e, t):
        e.embed(t, 512, width)
        ps, qs = e.slot("p", lambda: p), e.slot("q", lambda: q)
        fl = 2 if e.bf16 else 0
        e.op(OP.TANH_RESID, [e.temp("x"), ps, e.temp("x"), e.temp("s"), qs, e.temp("a"), ROWS_AUTO, width, fl, 0, 0])
        e.op(OP.TANH_RESID, [e.temp("s"), ps, 0, e.temp("n"), 0, 0, ROWS_AUTO, width, fl, 0, 0])
        e.op(OP.PICK_ROWS, [e.temp("s"), S(e.face), e.max_rows, e.temp("picked"), SEL_AUTO, width])
        e.op(OP.TANH_RESID, [e.temp("picked"), 0, 0, 0, qs, e.temp("head"), SEL_AUTO, width, fl, 0, 0])
    for fuse in (1, 0):
        eng, e, x = run_ops(cuda, emit, rows, sel, dtype, width=width, fuse=fuse)
        x = x.astype(np.float64)
        s = x + oracle.tanh_norm(x, *pv)
        assert np.abs(faces(eng, e, "s", rows, False) - s).max() < 3e-6
        assert np.abs(faces(eng, e, "n", rows, False) - oracle.tanh_norm(s, *pv)).max() < 3e-6
        near = lambda got, want: (np.abs(got - want) <= ((4e-3 * np.abs(want) + 1e-5) if e.bf16 else 3e-6)).all()
        assert near(faces(eng, e, "a", rows, e.bf16), oracle.tanh_norm(s, *qv))
        at = (np.arange(sel) * 7 + rows - 1) % rows
        assert near(faces(eng, e, "head", sel, e.bf16), oracle.tanh_norm(s, *qv)[at])
        eng.shutdown()


@pytest.mark.gpu
@pytest.mark.parametrize("K,N", [(64, 128), (24, 6), (72, 258), (320, 24), (8, 130), (20, 34), (1024, 136), (64, 2)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_projection_epilogues(cuda, K, N, dtype):
    """Bias, gated gelu, and the residual sum with its norms behind every projection path, fused and op by op."""
    rng = np.random.default_rng(K * N)
    w = bf16_to_f32(f32_to_bf16(rng.standard_normal((N, K)).astype(np.float32) / np.float32(K ** 0.5)))
    bias = rng.standard_normal(N).astype(np.float32)
    (p, pv), (q, qv) = params(rng, N), params(rng, N)
    for rows in (1, 2, 9, 31, 33, 130, 300):
        def emit(e, t):
            e.embed(t, 512, K)
            ws, bs, ps, qs = (e.slot(n, lambda a=a: a) for n, a in (("w", f32_to_bf16(w)), ("b", bias), ("p", p), ("q", q)))
            xf, yf = (LIN_X_BF16, LIN_Y_BF16) if e.bf16 else (0, 0)
            e.op(OP.LINEAR, [e.act(), ws, e.temp("yb"), ROWS_AUTO, K, N, xf | yf, 0, 0, bs])
            e.op(OP.LINEAR, [e.act(), ws, e.temp("yf"), ROWS_AUTO, K, N, xf, 0, 0, bs])
            e.op(OP.LINEAR, [e.act(), ws, e.temp("h"), ROWS_AUTO, K, N, xf | yf | LIN_GELU_GATE, 0, 0, 0])
            for to, add in (("r", 0), ("r", 1)):
                e.op(OP.LINEAR, [e.act(), ws, e.temp("y"), ROWS_AUTO, K, N, xf, 0, 0, 0])
                e.op(OP.TANH_RESID, [e.temp("y"), ps if add else 0, e.temp(to) if add else 0, e.temp(to), qs, e.temp("a"), ROWS_AUTO, N, 2 if e.bf16 else 0, N + 8, 8])
        for fuse in (1, 0):
            eng, e, x = run_ops(cuda, emit, rows, dtype=dtype, width=K, fuse=fuse)
            y = x.astype(np.float64) @ w.T.astype(np.float64)
            tol = 2e-5 * max(1.0, np.abs(y).max())
            assert np.abs(faces(eng, e, "yf", rows, False) - (y + bias)).max() < tol, (rows, fuse)
            close_b = lambda got, want: (np.abs(got - want) <= ((8e-3 * np.abs(want) + 2e-3) if e.bf16 else 2 * tol)).all()
            assert close_b(faces(eng, e, "yb", rows, e.bf16), y + bias), (rows, fuse)
            assert close_b(faces(eng, e, "h", rows, e.bf16), oracle.gelu_tanh(y[:, 0::2]) * y[:, 1::2]), (rows, fuse)
            r = y + oracle.tanh_norm(y, *pv)
            assert np.abs(faces(eng, e, "r", rows, False) - r).max() < 2 * tol, (rows, fuse)
            assert close_b(faces(eng, e, "a", rows, e.bf16)[:, 8:], oracle.tanh_norm(r, *qv)), (rows, fuse)
            eng.shutdown()


# ------------------------------------------------------------------ GPU: mechanisms and whole models
SINGLE = {
    "plain": layer(),
    "no feed-forward": layer(ff=None),
    "no scaling": layer(scaling=None, rot=24),
    "one head, window of one": layer(heads=1, kv_heads=1, dim=8, vdim=8, rot=2, window=1, ff=None),
    "window of two": layer(window=2),
    "window past the context": layer(window=5000),
    "a key head per head": layer(heads=5, kv_heads=5, dim=16, vdim=24, rot=16),
    "many heads to a key head": layer(heads=20, kv_heads=1, dim=32, vdim=16, window=40),
    "odd sizes": layer(heads=3, kv_heads=1, dim=13, vdim=11, rot=6, ff=37),
    "64 / 64": layer(heads=4, kv_heads=2, dim=64, vdim=64, rot=32, window=33),
    "128 / 64, odd group": layer(heads=3, kv_heads=1, dim=128, vdim=64, rot=96, scale=0.1),
    "64 / 128, a key head per head": layer(heads=2, kv_heads=2, dim=64, vdim=128, rot=64, window=30),
    "128 / 128": layer(heads=8, kv_heads=2, dim=128, vdim=128, rot=128, scale=0.09, window=61, ff=200),
    "wide values": layer(heads=2, kv_heads=1, dim=40, vdim=200, rot=8),
    "values beyond the tiled kernels": layer(heads=2, kv_heads=1, dim=16, vdim=264, rot=8),
    "keys of 320": layer(heads=2, kv_heads=1, dim=320, vdim=24, rot=10, scale=0.05),
}


@pytest.mark.gpu
@pytest.mark.parametrize("name", list(SINGLE))
def test_layer_alone(cuda, name):
    """One layer: prompt, a short portion, decoding behind it, and the one-kernel-per-op plan."""
    mt = make([SINGLE[name]], seed=len(name), width=75 if name == "odd sizes" else 72)
    tok = ids(90)
    want = oracle.run(*mt, tok)[0]
    for dtype in DTYPES:
        for fuse in (1, 0):
            cuda.gehtp_cuda_set_fusion(fuse)
            s = session(cuda, mt, dtype, max_tokens=128)
            assert close(run_cut(s, tok, [80, 5, 1, 1, 1, 1, 1]), want, dtype), (dtype, fuse)
            s.close()
    cuda.gehtp_cuda_set_fusion(1)


@pytest.mark.gpu
@pytest.mark.parametrize("loop", [None, (0, 1, 1), (0, 3, 2), (1, 2, 3), (2, 3, 2), (1, 3, 4)])
def test_loops(cuda, loop):
    mt = make(MIX, loop, seed=4)
    tok = ids(40)
    want, trail = oracle.run(*mt, tok)
    for dtype in DTYPES:
        s = session(cuda, mt, dtype)
        assert len(s.man["layer_end"]) == len(trail)
        assert close(run_cut(s, tok, [30, 7, 1, 1, 1]), want, dtype), dtype
        s.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_stream_after_every_layer_run(cuda, dtype):
    mt = make(MIX, LOOP, seed=5)
    tok = ids(20)
    trail = oracle.run(*mt, tok)[1]
    s = session(cuda, mt, dtype)
    s.feed(tok, [0])                                      # injects the input face
    s.reset()
    s.engine.set_rows(20, 1)
    at = 0
    for i, end in enumerate(s.man["layer_end"]):
        s.engine.run_range(at, end - at)
        at = end
        assert close(s.engine.temp(s.man["stream_temp"], np.float32).reshape(20, -1), trail[i], dtype), i
    s.close()


CUTS = [[1] * 60, [2] * 30, [3, 2, 40, 2, 13], [59, 1], [1, 59], [17, 16, 15, 12], [33, 27], [4, 5, 8, 9, 16, 18]]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_agree_with_the_whole_prompt(cuda, dtype):
    mt = make(MIX, LOOP, seed=6, sharp=2.0 if dtype == "float32" else 1.0)
    tok = ids(60, seed=2)
    want = oracle.run(*mt, tok)[0]
    s = session(cuda, mt, dtype)
    assert close(run_cut(s, tok, [60]), want, dtype)
    for cut in CUTS:
        assert close(run_cut(s, tok, cut), want, dtype), cut
    s.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("max_rows", [7, 16, 100])
def test_ring_wraps(cuda, dtype, max_rows):
    """Sequences several times as long as the ring, in portions, by single tokens, and cut by the session itself."""
    mt = make([layer(window=19, dim=64, vdim=64), layer(window=100, dim=128, vdim=128, heads=2, kv_heads=1, rot=128, scale=0.1)], (0, 1, 2), seed=7)
    tok = ids(620)
    want = oracle.run(*mt, tok)[0]
    s = session(cuda, mt, dtype, max_tokens=640, max_rows=max_rows, max_sel=max_rows)
    assert close(run_cut(s, tok, [620]), want, dtype)
    assert close(run_cut(s, tok, [300] + [1] * 20 + [130, 2, 3, 5, 160]), want, dtype)
    s.reset()
    s.feed(tok[:500])
    got = np.concatenate([s.feed([t], [0]) for t in tok[500:]])
    assert close(got, want[500:], dtype)
    s.close()


@pytest.mark.gpu
@pytest.mark.parametrize("n", [1, 2, 3, 15, 16, 17, 63, 64, 65, 127, 128, 129, 255, 257, 300])
def test_lengths_around_the_tiles(cuda, n):
    """A prompt of n tokens, a portion of 9 and five decoded ones, with keys that stand out, at the sizes of both prompt kernels."""
    tok = ids(n + 14, seed=n)
    for sizes in (dict(dim=128, vdim=64, rot=32, scale=0.1), dict(dim=48, vdim=32)):
        mt = make([layer(window=130, **sizes), layer(window=33, **sizes)], seed=n, sharp=2.0)
        want = oracle.run(*mt, tok)[0]
        for dtype in DTYPES:
            s = session(cuda, mt, dtype)
            assert close(run_cut(s, tok, [n, 9, 1, 1, 1, 1, 1]), want, dtype), (dtype, sizes)
            s.close()


def far_key_model(window, dim, vdim, heads, kv_heads, seed=11):
    """One layer in which token 1's query matches token 0's key far above all others: the query of token 1 is made from the
    key of token 0 through the projections. Only two components turn with the position."""
    cfg, t = make([layer(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, window=window, rot=2, scaling=None, scale=40.0 / dim, ff=None)], seed=seed)
    f = lambda n: t["l0." + n].astype(np.float64)
    h = oracle.tanh_norm(t["embed"][:2].astype(np.float64) * cfg["embedding"]["scale"], f("norm1.alpha"), f("norm1"), f("norm1.b"))
    key = (f("mix.k") @ h[0] + f("mix.k.b")).reshape(kv_heads, dim)
    key = oracle.rms_unit(key, cfg["norm"]["eps"]) * f("mix.k.norm")
    q = f("mix.q").reshape(heads, dim, -1)
    t["l0.mix.q.norm"][:] = 1.0
    for i in range(heads):
        # rank-one change: the query of embedding 1 becomes a multiple of the key of embedding 0
        have = q[i] @ h[1] + f("mix.q.b").reshape(heads, dim)[i]
        q[i] += np.outer(4.0 * key[i // (heads // kv_heads)] - have, h[1]) / (h[1] @ h[1])
    t["l0.mix.q"] = bf16_to_f32(f32_to_bf16(q.reshape(heads * dim, -1).astype(np.float32)))
    return cfg, t


@pytest.mark.gpu
@pytest.mark.parametrize("window,dim,vdim,heads,kv_heads", [(128, 128, 128, 4, 2), (100, 64, 64, 3, 1), (257, 128, 64, 2, 2), (64, 40, 24, 4, 1), (3, 64, 64, 2, 1)])
def test_window_edges(cuda, window, dim, vdim, heads, kv_heads):
    """The one token whose key the last query looks for is the oldest the window holds, or the one before that, or stands at
    a tile border inside it - in a prompt, at the end of a portion and in decoding, at last positions off and on tiles."""
    mt = far_key_model(window, dim, vdim, heads, kv_heads)
    for n in (300, 385, window + 1):
        inside = sorted({max(n - window, 0), n - 2} | {p for p in (128, 255, 256, 272, 320) if n - window <= p < n - 1})
        for place in [n - window - 1] + inside:
            if not 0 <= place < n - 1:
                continue
            tok = [2 + i % 100 for i in range(n)]
            tok[place], tok[-1] = 0, 1
            want = oracle.run(*mt, tok)[0][-1:]
            other = list(tok)
            other[place] = 5
            seen = rel(oracle.run(*mt, other)[0][-1:], want)
            assert seen > 0.15 if place >= n - window else seen == 0.0           # the key decides the row, or has no part in it
            for dtype in DTYPES:
                s = session(cuda, mt, dtype)
                assert close(s.feed(tok, [n - 1]), want, dtype), (n, place, dtype)
                s.reset()
                s.feed(tok[:n - 1])
                assert close(s.feed(tok[n - 1:], [0]), want, dtype), (n, place, dtype)
                s.reset()
                cut = max(n - 20, 1)
                s.feed(tok[:cut])
                assert close(s.feed(tok[cut:], [n - 1 - cut]), want, dtype), (n, place, dtype)
                s.reset()
                s.feed(tok[:n - 2])
                assert close(s.feed(tok[n - 2:], [1]), want, dtype), (n, place, dtype)
                s.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dim,vdim", [(128, 128), (32, 16)])
def test_maximum_that_grows(cuda, dim, vdim):
    """Scores far above those of earlier tiles, so that what a row has summed up is rescaled more than once."""
    mt = make([layer(window=700, dim=dim, vdim=vdim, rot=2, scaling=None, scale=30.0 / dim, heads=2, kv_heads=1, ff=None)], seed=3, sharp=4.0)
    tok = ids(600, seed=9)
    want = oracle.run(*mt, tok)[0]
    for dtype in DTYPES:
        s = session(cuda, mt, dtype, max_tokens=640)
        pick = list(range(0, 600, 13)) + [599]
        e = row_errors(s.feed(tok, sorted(pick)), want[sorted(pick)])
        # sharp softmax: which of two near-equal keys wins follows the roundings of bf16 queries and keys
        assert e.max() < 3e-4 if dtype == "float32" else np.median(e) < 5e-2, dtype
        s.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_states_are_given_back(cuda, dtype):
    """A request after another one gives the bits it gives alone."""
    mt = make(MIX, LOOP, seed=9)
    a, b = ids(190, seed=4), ids(40, seed=5)
    s = session(cuda, mt, dtype)

    def run(tok):
        s.reset()
        return np.concatenate([s.feed(tok[:-6], [len(tok) - 7])] + [s.feed([t], [0]) for t in tok[-6:]])
    alone = run(b)
    run(a)
    assert np.array_equal(alone, run(b))
    assert close(alone, oracle.run(*mt, b)[0][-7:], dtype)
    s.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(cuda, dtype):
    mt = make(MIX, LOOP, seed=10)
    tok = ids(220, seed=6)
    want = oracle.run(*mt, tok)[0]
    s = session(cuda, mt, dtype)
    got = np.concatenate([s.feed(tok[:10], [9])] + [s.feed([t], [0]) for t in tok[10:]])
    assert close(got, want[9:], dtype)
    s.close()


@pytest.mark.gpu
def test_replayed_graph_gives_the_eager_bits(cuda):
    mt = make(MIX, LOOP, seed=12)
    tok = ids(30)

    def run(graph):
        cuda.gehtp_cuda_set_graph(graph)
        s = session(cuda, mt, "bfloat16")
        got = np.concatenate([s.feed(tok[:5], [4])] + [s.feed([t], [0]) for t in tok[5:]])
        s.close()
        return got
    a, b = run(0), run(1)
    cuda.gehtp_cuda_set_graph(1)
    assert np.array_equal(a, b)


def greedy(mt, prompt, n):
    tok = list(prompt)
    for _ in range(n):
        tok.append(int(oracle.run(*mt, tok)[0][-1].argmax()))
    return tok[len(prompt):]


@pytest.mark.gpu
def test_generation_through_the_scheduler(cuda):
    mt = make(MIX, LOOP, seed=13)
    prompts = [ids(12, seed=1), ids(1, seed=2), ids(33, seed=3)]
    s = session(cuda, mt, "float32", max_rows=10)
    sch = Scheduler(s)
    for i, p in enumerate(prompts):
        sch.submit(Request(i, p, 8))
    sch.submit(Request("bad", [5000], 3))
    first = greedy(mt, prompts[0], 8)
    sch.submit(Request("stop", prompts[0], 8, stop=(first[2],)))
    done = sch.run()
    for r, p in zip(done, prompts):
        assert r.tokens == greedy(mt, p, 8)
    assert done[3].error and done[4].tokens == first[:first.index(first[2]) + 1]
    s.close()


@pytest.mark.gpu
def test_command_line(cuda, tmp_path):
    """The command line generates; bin/trace_run gives the session's logits."""
    mt = make(MIX, LOOP, seed=14)
    (tmp_path / "config.json").write_text(json.dumps(mt[0]))
    write_safetensors(str(tmp_path / "model.safetensors"), mt[1])
    tok = ids(20)
    run = lambda *a, **k: subprocess.run(a, cwd=ROOT, capture_output=True, text=True, timeout=300, **k)
    r = run(sys.executable, "-m", "gehtp_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt", ",".join(map(str, tok)), "--max-new", "5")
    assert r.returncode == 0, r.stderr
    assert [int(x) for x in r.stdout.split(",")] == greedy(mt, tok, 5)
    lines = [json.dumps(dict(step=0, entries=[dict(id="q", tokens=tok[:15], want=[3, 14])], end=[])),
             json.dumps(dict(step=1, entries=[dict(id="q", tokens=tok[15:], want=[4])], end=["q"]))]
    r = run(os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "bfloat16", "--out", str(tmp_path), "--max-tokens", "64",
            input="\n".join(lines) + "\n")
    assert r.returncode == 0 and r.stdout.split("\n")[:2] == ["done 0", "done 1"], r.stderr
    got = np.concatenate([np.fromfile(str(tmp_path / ("%d.f32" % n)), np.float32).reshape(-1, 130) for n in (0, 1)])
    assert close(got, oracle.run(*mt, tok)[0][[3, 14, 19]], "bfloat16")


@pytest.mark.gpu
def test_limits_are_reported(cuda):
    mt = make(MIX, LOOP, seed=15)
    s = session(cuda, mt, "bfloat16", max_tokens=200, max_rows=16, max_sel=2)
    for _ in range(2):                                    # 256 positions whatever the rings hold
        s.reset()
        s.feed(ids(256))
        with pytest.raises(ValueError):
            s.feed([1])
        s.position = 0
        with pytest.raises(EngineError, match="context too long"):
            s.feed([1])
    s.close()
    # a ring too small for the window and the rows of a run is refused, not overrun
    e = RowsEmitter("bfloat16", 512, 64, 8)
    t = e.slot("t", lambda: np.zeros((16, 80), np.uint16))
    e.embed(t, 16, 80, act="act")
    st = e._state("cache", 128 * 64 * 2)
    rope = e.slot("r", lambda: rope_halves(512, 4, 100.0))
    e.op(OP.HEADS_APPEND, [e.temp("act"), 0, rope, e.temp("q"), st, ROWS_AUTO, 1, 1, 16, 48, 4, bits(1e-5), 80, 512, 1])
    e.op(OP.WINDOW_ATTEND, [e.temp("q"), 0, st, e.temp("o"), ROWS_AUTO, 1, 1, 16, 48, 66, bits(1.0), 0xFFFFFFFF, 80, 1])
    eng = Engine(cuda, e.finish())
    eng.set_rows(4, 1)
    with pytest.raises(EngineError, match="exceed a ring"):
        eng.run_io(np.zeros(72, np.int32), 1, None)
    eng.shutdown()
