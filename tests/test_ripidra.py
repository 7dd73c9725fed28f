"""The Ripidra design through the engine against the plain statement in ripidra_oracle.py: every mechanism alone, whole
prompts against portions and token-by-token decoding, sizes off every tile, generation through the scheduler."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import ripidra_oracle as oracle
from gehtp_b200.checkpoint import ArrayTensors, Tensors, bf16_to_f32, f32_to_bf16, write_safetensors
from gehtp_b200.registry import Model, load_model
from gehtp_b200.rowlists import RowsEmitter, join_rows, latent_row, rope_pairs
from gehtp_b200.session import Request, Scheduler, Session
from gehtp_b200.trace import replay
from gehtp_b200.wtop import LIN_RELU2, LIN_X_BF16, LIN_Y_BF16, OP, ROWS_AUTO, SEL_AUTO, EngineError, S, parse_blob

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def latent(heads=3, dim=24, rot_dim=16, vdim=40, kv_rank=48, base=5000.0, scale=0.17, ff=96, **kw):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale, rot=dict(base=base, dims=rot_dim))
    return dict(type="latent_attention", mixer=m, mlp=dict(kind="dense", ff=ff) if ff else None, **kw)


def delta(heads=4, kv_heads=2, dim=32, vdim=24, conv=4, ff=96, **kw):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)
    return dict(type="channel_delta", mixer=m, mlp=dict(kind="dense", ff=ff) if ff else None, **kw)


def make(layers, vocab=120, width=80, eps=1e-5, seed=0, rank_a=16, rank_g=8, sharp=1.0, slow=0.0):
    """(config, tensors as float32 holding bf16 values). sharp: factor on the query projections, so that single keys
    stand out; slow: shift of the decay bias, so that old tokens stay in the state."""
    cfg = dict(architecture="Ripidra", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    rng = np.random.default_rng(seed)
    t = {}

    def put(name, *shape, std=None, mean=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        t[name] = bf16_to_f32(f32_to_bf16(rng.standard_normal(shape).astype(np.float32) * np.float32(std) + np.float32(mean)))
    put("embed", vocab, width, std=1.0)
    put("final.norm", width, std=0.2)
    for i, e in enumerate(layers):
        if e.get("weights_of") is not None:
            continue
        p, m = "l%d." % i, e["mixer"]
        put(p + "norm1", width, std=0.3)
        if e["mlp"]:
            put(p + "norm2", width, std=0.3)
            put(p + "mlp.up", e["mlp"]["ff"], width)
            put(p + "mlp.down", width, e["mlp"]["ff"])
        q = p + "mix."
        if e["type"] == "latent_attention":
            put(q + "q", m["heads"] * (m["dim"] + m["rot_dim"]), width, std=sharp * width ** -0.5)
            put(q + "dkv", m["kv_rank"] + m["rot_dim"], width)
            put(q + "dkv.norm", m["kv_rank"], std=0.3, mean=1.0)
            put(q + "uk", m["heads"] * m["dim"], m["kv_rank"])
            put(q + "uv", m["heads"] * m["vdim"], m["kv_rank"])
            put(q + "g", m["heads"], width)
            put(q + "o", width, m["heads"] * m["vdim"])
        else:
            kd, vd, hd = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"], m["heads"] * m["dim"]
            for n, c in (("q", kd), ("k", kd), ("v", vd)):
                put(q + n, c, width)
                put(q + n + ".conv", c, m["conv"], std=0.6)
            put(q + "b", m["heads"], width)
            put(q + "A_log", m["heads"], std=0.5)
            put(q + "dt_bias", hd, std=0.5, mean=-slow)
            put(q + "norm", m["vdim"], std=0.3, mean=1.0)
            put(q + "a1", rank_a, width)
            put(q + "a2", hd, rank_a)
            put(q + "g1", rank_g, width)
            put(q + "g2", vd, rank_g)
            put(q + "o", width, vd)
    return cfg, t


def ids(n, vocab=120, seed=1):
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
    """fp32: every row within 3e-5. bf16: rounding differs from row to row (a mixer output that nearly cancels is
    normed up, and its rounding with it): no row beyond 8e-2, half of them within 1.5e-2."""
    e = row_errors(got, want)
    return bool(e.max() < 3e-5 if dtype == "float32" else e.max() < 8e-2 and np.median(e) < 1.5e-2)


DTYPES = ["float32", "bfloat16"]
MIX = [latent(), delta(), latent(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=32, base=300.0, scale=0.3, ff=None), delta(weights_of=1),
       latent(weights_of=0)]


# ------------------------------------------------------------------ CPU: reader, runlist, session logic
def test_safetensors_round_trip(tmp_path):
    cfg, t = make(MIX)
    path = str(tmp_path / "model.safetensors")
    write_safetensors(path, t)
    r = Tensors(path)
    assert sorted(r.names()) == sorted(t)
    for k, a in t.items():
        assert r.shape(k) == a.shape and np.array_equal(r.f32(k), a)
    with pytest.raises(KeyError):
        r.raw("nothing")
    with pytest.raises(ValueError):
        r.bf16("embed", (1, 2))
    with open(path, "r+b") as f:
        f.truncate(os.path.getsize(path) - 4)
    with pytest.raises(ValueError):
        [Tensors(path).raw(k) for k in t]


def test_registry_reads_the_config(tmp_path):
    cfg, t = make(MIX)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), t)
    m = load_model(str(tmp_path))
    assert m.architecture == "Ripidra" and [m.config.owner(i) for i in range(5)] == [0, 1, 2, 1, 0]
    for bad in (dict(cfg, architecture="other"), dict(cfg, layers=[dict(latent(), type="other")]),
                dict(cfg, layers=[dict(latent(), mlp=dict(kind="routed", ff=8))]), dict(cfg, layers=[latent(weights_of=3)])):
        with pytest.raises(ValueError):
            Model(bad, ArrayTensors(t))
    loop = Model(dict(cfg, layers=[latent(weights_of=1), latent(weights_of=0)]), ArrayTensors(t))
    with pytest.raises(ValueError):
        loop.runlist()


@pytest.mark.parametrize("dtype", DTYPES)
def test_runlist_shares_weights_and_numbers_states(cuda, dtype):
    cfg, t = make(MIX)
    blob, man = Model(cfg, ArrayTensors(t)).runlist(dtype, max_tokens=100, max_rows=40, max_sel=3)
    assert man["nslots"] == 128 and man["max_rows"] == 40 and man["max_sel"] == 3
    rc, b = parse_blob(cuda, blob)
    assert rc == 0
    ops = [(o.opcode, list(o.args[:o.n_args])) for o in b.ops[:b.n_ops]]
    lat = [a for c, a in ops if c == OP.LATENT_ATTEND]
    dlt = [a for c, a in ops if c == OP.CHANNEL_DELTA]
    # layers 0 and 4 (1 and 3) use one weight slot each, and a state of their own
    assert lat[0][3] == lat[2][3] != lat[1][3] and len({a[2] for a in lat}) == 3
    assert dlt[0][3] == dlt[1][3] and dlt[0][5] != dlt[1][5]
    adv = [a for c, a in ops if c == OP.STATE_ADVANCE]
    assert adv == [[0, 3, ROWS_AUTO], [3, 2, 1]]
    assert sum(c == OP.NORM_RESID for c, _ in ops) == 5 + 4 + 1
    with pytest.raises(ValueError):
        Model(cfg, ArrayTensors(t)).runlist("float16")


def test_join_rows_and_tables():
    a, b = np.ones((3, 4), np.uint16), np.full((9, 4), 2, np.uint16)
    m, at = join_rows([a, b])
    assert at == [0, 8] and m.shape == (24, 4) and (m[3:8] == 0).all() and (m[8:17] == 2).all() and (m[17:] == 0).all()
    assert latent_row(48, 16) == 64 and latent_row(33, 4) == 48
    tab = rope_pairs(5, 6, 100.0)
    x = np.random.default_rng(0).standard_normal((5, 6))
    c, s = tab[..., 0], tab[..., 1]
    got = np.stack([x[:, 0::2] * c - x[:, 1::2] * s, x[:, 1::2] * c + x[:, 0::2] * s], axis=-1).reshape(5, 6)
    assert np.abs(got - oracle.rotate_pairs(x, np.arange(5), 100.0)).max() < 1e-6


def test_row_ops_are_validated(cuda):
    """Arity and slot references of the row ops are checked by the parser like those of the reference's ops."""
    e = RowsEmitter("float32", 64, 8, 2)
    tab = e.slot("t", lambda: np.zeros((4, 8), np.uint16))
    e.embed(tab, 4, 8)
    e.b.add_op(OP.LINEAR, [1, S(99), 9, ROWS_AUTO, 8, 8, 0, 0, 0, 0])
    assert parse_blob(cuda, e.finish())[0] == -12
    e.b.ops[-1] = (OP.LINEAR, [1, tab, 9])
    assert parse_blob(cuda, e.b.build())[0] == -11
    e.b.ops[-1] = (0x14E, [])
    assert parse_blob(cuda, e.b.build())[0] == -10


class FakeSession:
    """Logits that tell the tokens fed so far, so that the replay and scheduling logic can be checked without a GPU."""
    def __init__(self):
        self.seen, self.resets = [], 0

    def reset(self):
        self.seen, self.resets = [], self.resets + 1

    def feed(self, tokens, want=()):
        base = len(self.seen)
        self.seen += tokens
        return np.array([[base + w, sum(self.seen[:base + w + 1])] for w in want], np.float32).reshape(-1, 2)

    def generate(self, prompt, n, stop=()):
        if not prompt:
            raise ValueError("no tokens")
        self.reset()
        return [len(prompt) + i for i in range(n)]


def test_replay_writes_the_wanted_rows(tmp_path):
    steps = [dict(step=0, entries=[dict(id="a", tokens=[5, 7, 1], want=[2, 0])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=[4], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=[2], want=[0])], end=["a"]),
             dict(step=3, entries=[dict(id="b", tokens=[9], want=[0])], end=["b"])]
    out, s = [], FakeSession()
    replay(s, [json.dumps(x) + "\n" for x in steps], str(tmp_path), out.append)
    assert out == ["done %d" % i for i in range(4)]
    read = lambda n: np.fromfile(str(tmp_path / ("%d.f32" % n)), "<f4").reshape(-1, 2).tolist()
    assert read(0) == [[2, 13], [0, 5]] and read(2) == [[4, 19]] and read(3) == [[0, 9]]
    assert not (tmp_path / "1.f32").exists()
    with pytest.raises(ValueError):
        replay(FakeSession(), [json.dumps(dict(step=0, entries=[dict(id="a", tokens=[1], want=[])], end=[])),
                               json.dumps(dict(step=1, entries=[dict(id="b", tokens=[1], want=[])], end=[]))], str(tmp_path), out.append)


def test_scheduler_serves_in_order_and_keeps_going():
    sch = Scheduler(FakeSession())
    for i, p in enumerate(([1, 2], [], [3])):
        sch.submit(Request(i, p, 2))
    r = sch.run()
    assert [x.id for x in r] == [0, 1, 2] and r[0].tokens == [2, 3] and r[1].error == "no tokens" and r[2].tokens == [1, 2]


def test_portions_respect_both_limits():
    s = Session.__new__(Session)
    s.man = dict(max_rows=10, max_sel=2)
    got = list(s._portions(25, [0, 3, 4, 9, 24]))
    assert [(a, b, w) for a, b, w in got] == [(0, 4, [0, 3]), (4, 14, [4, 9]), (14, 24, []), (24, 25, [24])]


def test_oracle_mechanisms():
    """The plain statement's own pieces on cases with known answers."""
    x = np.arange(12.0).reshape(4, 3)
    w = np.zeros((3, 3))
    w[:, 2], w[:, 1] = 1.0, 10.0
    assert np.array_equal(oracle.causal_conv(x, w)[2], x[2] + 10 * x[1]) and np.array_equal(oracle.causal_conv(x, w)[0], x[0])
    k = np.zeros((2, 1, 2)); k[:, 0, 0] = 1.0
    v = np.array([[[3.0]], [[5.0]]])
    o = oracle.delta_recurrence(k, k, v, np.full((2, 1, 2), 0.5), np.ones((2, 1)))
    assert np.allclose(o[:, 0, 0], [3.0, 5.0])            # a full step replaces what the key held
    o = oracle.delta_recurrence(k, k, v, np.full((2, 1, 2), 0.5), np.array([[1.0], [0.0]]))
    assert np.allclose(o[:, 0, 0], [3.0, 1.5])            # no step: the value decays
    assert np.allclose(oracle.norm_about_one(np.array([3.0, 4.0]), np.array([0.0, 1.0]), 0.0), np.array([3.0, 8.0]) / np.sqrt(12.5))


# ------------------------------------------------------------------ GPU: single ops
def run_ops(cuda, emit, rows, sel=1, dtype="bfloat16", vocab=512, width=64, max_rows=512, fuse=1):
    """Runs EMBED_ROWS of ids 0..rows-1 and the ops of emit(emitter, table slot); returns (engine, x rows)."""
    from gehtp_b200.wtop import Engine
    cuda.gehtp_cuda_set_fusion(fuse)
    tab = bf16_to_f32(f32_to_bf16(np.random.default_rng(3).standard_normal((vocab, width)).astype(np.float32)))
    e = RowsEmitter(dtype, 512, max_rows, 8)
    t = e.slot("t", lambda: f32_to_bf16(tab))
    e.embed(t, vocab, width)
    emit(e, t)
    eng = Engine(cuda, e.finish())
    eng.set_rows(rows, sel)
    face = np.zeros(max_rows + 8, np.int32)
    face[:rows] = np.arange(rows)
    face[max_rows:max_rows + sel] = (np.arange(sel) * 7 + rows - 1) % rows
    eng.run_io(face, 1, None)
    cuda.gehtp_cuda_set_fusion(1)
    return eng, e, tab[:rows]


@pytest.mark.gpu
@pytest.mark.parametrize("K,N", [(64, 128), (24, 5), (72, 257), (320, 24), (8, 130), (20, 33), (64, 1)])
def test_projection_shapes(cuda, K, N):
    """Every projection path by row count, with strided inputs and sizes off the tiles."""
    w = bf16_to_f32(f32_to_bf16(np.random.default_rng(K * N).standard_normal((N, K)).astype(np.float32) / np.float32(K ** 0.5)))
    width = max(K + 8, 64) + (-K) % 8
    for dtype in DTYPES:
        for rows in (1, 2, 9, 31, 33, 130, 300):
            def emit(e, t):
                ws = e.slot("w", lambda: f32_to_bf16(w))
                fl = LIN_X_BF16 if e.bf16 else 0
                e.op(OP.LINEAR, [e.act(), ws, e.temp("y"), ROWS_AUTO, K, N, fl, 8, width, 0])
                e.op(OP.LINEAR, [e.act(), ws, e.temp("r"), ROWS_AUTO, K, N, fl | (LIN_Y_BF16 if e.bf16 else 0) | LIN_RELU2, 8, width, 0])
            eng, e, x = run_ops(cuda, emit, rows, dtype=dtype, width=width)
            want = x[:, 8:8 + K].astype(np.float64) @ w.T.astype(np.float64)
            y = eng.temp(e.temp("y"), np.float32).reshape(rows, N)
            assert np.abs(y - want).max() < 2e-5 * max(1.0, np.abs(want).max()), (dtype, rows)
            r = eng.temp(e.temp("r"), np.uint16 if dtype == "bfloat16" else np.float32).reshape(rows, N)
            r = bf16_to_f32(r) if dtype == "bfloat16" else r
            want = np.maximum(want, 0) ** 2
            assert (np.abs(r - want) <= (5e-3 if dtype == "bfloat16" else 1e-4) * (want + 1e-2)).all(), (dtype, rows)
            eng.shutdown()


@pytest.mark.gpu
@pytest.mark.parametrize("width", [64, 50, 2560, 5000])
def test_norm_pick_and_choice(cuda, width):
    rng = np.random.default_rng(width)
    w = rng.standard_normal(width).astype(np.float32)
    rows, sel = 9, 4

    def emit(e, t):
        ws = e.slot("w", lambda: w)
        e.op(OP.NORM_RESID, [e.temp("x"), ws, e.temp("x"), e.temp("n"), e.temp("na"), ROWS_AUTO, width, 1 | 2, np.float32(0.5).view(np.uint32)])
        e.op(OP.NORM_RESID, [e.temp("act"), ws, 0, e.temp("p"), 0, ROWS_AUTO, width, 4, np.float32(1e-6).view(np.uint32)])
        e.op(OP.PICK_ROWS, [e.temp("x"), S(e.face), e.max_rows, e.temp("picked"), SEL_AUTO, width])
        e.op(OP.ARGMAX_ROWS, [e.temp("picked"), e.temp("tok"), SEL_AUTO, width])
    eng, e, x = run_ops(cuda, emit, rows, sel, width=width)
    f = lambda n, dt=np.float32: eng.temp(e.temp(n), dt)
    want = x + oracle.norm_about_one(x.astype(np.float64), w, 0.5)
    assert np.abs(f("n").reshape(rows, width) - want).max() < 1e-5
    assert np.array_equal(f("na", np.uint16), f32_to_bf16(f("n")))
    assert np.abs(f("p").reshape(rows, width) - oracle.rms_unit(x.astype(np.float64), 1e-6) * w).max() < 2e-5
    at = (np.arange(sel) * 7 + rows - 1) % rows
    assert np.array_equal(f("picked").reshape(sel, width), x[at])
    assert np.array_equal(f("tok", np.int32), x[at].argmax(axis=1))
    eng.shutdown()


# ------------------------------------------------------------------ GPU: mechanisms and whole models
SINGLE = {
    "latent": [latent()],
    "latent without feed-forward": [latent(ff=None)],
    "latent, one head": [latent(heads=1, dim=8, rot_dim=2, vdim=8, kv_rank=8, ff=None)],
    "latent, wide": [latent(heads=20, dim=40, rot_dim=24, vdim=72, kv_rank=200, scale=0.1)],
    "latent, odd sizes": [latent(heads=5, dim=13, rot_dim=6, vdim=11, kv_rank=21)],
    "latent, rank 300": [latent(heads=2, dim=64, rot_dim=32, vdim=130, kv_rank=300, scale=0.08)],
    "latent, rank above the split kernel": [latent(heads=2, dim=16, rot_dim=8, vdim=16, kv_rank=528, scale=0.2)],
    "delta": [delta()],
    "delta without feed-forward": [delta(ff=None)],
    "delta, one head": [delta(heads=1, kv_heads=1, dim=8, vdim=8, ff=None)],
    "delta, long taps": [delta(conv=6, dim=20, vdim=40)],
    "delta, two taps": [delta(conv=2, heads=6, kv_heads=3, dim=48, vdim=64)],
    "delta, no window": [delta(conv=1)],
    "delta, odd sizes": [delta(heads=3, kv_heads=1, dim=21, vdim=35, conv=3)],
    "delta, wide": [delta(heads=2, kv_heads=2, dim=200, vdim=136)],
    "delta, key dim above the step kernel": [delta(heads=2, kv_heads=1, dim=260, vdim=16)],
}


@pytest.mark.gpu
@pytest.mark.parametrize("name", list(SINGLE))
def test_mechanism_alone(cuda, name):
    """One layer: prompt, decoding behind it, and the one-kernel-per-op plan."""
    mt = make(SINGLE[name], seed=len(name), rank_a=12 if "odd" in name else 16, rank_g=140 if "wide" in name else 6, slow=1.0)
    tok = ids(75)
    want = oracle.run(*mt, tok)[0]
    for dtype in DTYPES:
        for fuse in (1, 0):
            cuda.gehtp_cuda_set_fusion(fuse)
            s = session(cuda, mt, dtype, max_tokens=128)
            got = [s.feed(tok[:70], range(70))] + [s.feed([t], [0]) for t in tok[70:]]
            assert close(np.concatenate(got), want, dtype), (dtype, fuse)
            s.close()
    cuda.gehtp_cuda_set_fusion(1)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_stream_after_every_layer(cuda, dtype):
    mt = make(MIX, seed=5)
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
    mt = make(MIX, seed=6, sharp=2.0 if dtype == "float32" else 1.0, slow=2.0)
    tok = ids(60, seed=2)
    want = oracle.run(*mt, tok)[0]
    s = session(cuda, mt, dtype)
    whole = s.feed(tok, range(60))
    assert close(whole, want, dtype)
    for cut in CUTS:
        s.reset()
        at, rows = 0, []
        for n in cut:
            rows.append(s.feed(tok[at:at + n], range(n)))
            at += n
        assert at == 60 and close(np.concatenate(rows), want, dtype), cut
    s.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_runs_smaller_than_a_portion(cuda, dtype):
    """A session whose runs take few rows and give few logits cuts a portion itself."""
    mt = make(MIX, seed=7)
    tok = ids(50)
    want = oracle.run(*mt, tok)[0]
    s = session(cuda, mt, dtype, max_rows=7, max_sel=3)
    assert close(s.feed(tok, range(50)), want, dtype)
    s.reset()
    pick = [49, 0, 3, 3, 20]
    assert close(s.feed(tok, pick), want[pick], dtype)
    s.close()


@pytest.mark.gpu
@pytest.mark.parametrize("n", [1, 2, 3, 31, 32, 33, 63, 64, 65, 127, 128, 129, 200])
def test_lengths_around_the_tiles(cuda, n):
    """A prompt of n tokens and five decoded ones, with keys that stand out."""
    mt = make([latent(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=64), delta(dim=64, vdim=32)], seed=n, sharp=3.0, slow=2.0)
    tok = ids(n + 5, seed=n)
    want = oracle.run(*mt, tok)[0]
    for dtype in DTYPES:
        s = session(cuda, mt, dtype)
        got = [s.feed(tok[:n], [n - 1])] + [s.feed([t], [0]) for t in tok[n:]]
        assert close(np.concatenate(got), want[n - 1:], dtype), dtype
        s.close()


def far_key_model(seed=11):
    """One attention layer in which token 1's query matches token 0's key far above all others: the query of token 1 is
    made from the key of token 0 through the projections."""
    cfg, t = make([latent(heads=2, dim=32, rot_dim=8, vdim=32, kv_rank=64, scale=0.2, base=1e8, ff=None)], seed=seed)
    e = t["embed"].astype(np.float64)
    m = cfg["layers"][0]["mixer"]
    c = oracle.rms_unit(e[0] @ t["l0.mix.dkv"][:64].T.astype(np.float64), cfg["norm"]["eps"]) * t["l0.mix.dkv.norm"]
    key = (c @ t["l0.mix.uk"].T).reshape(2, 32)
    q = t["l0.mix.q"].astype(np.float64).reshape(2, 40, -1)
    for h in range(2):
        # rank-one change: the query of embedding 1 becomes 12 * unit key of embedding 0
        have = q[h, :32] @ e[1]
        q[h, :32] += np.outer(12.0 * key[h] / np.linalg.norm(key[h]) - have, e[1]) / (e[1] @ e[1])
    t["l0.mix.q"] = bf16_to_f32(f32_to_bf16(q.reshape(80, -1).astype(np.float32)))
    return cfg, t


@pytest.mark.gpu
@pytest.mark.parametrize("place", [0, 1, 31, 32, 63, 64, 127, 128, 255, 300])
def test_one_far_key(cuda, place):
    """The one token whose key the last query looks for sits at tile and slice borders, in a prompt and in decoding."""
    mt = far_key_model()
    tok = [2 + i % 100 for i in range(310)]
    tok[place], tok[-1] = 0, 1
    want = oracle.run(*mt, tok)[0][-1:]
    other = list(tok)
    other[place] = 5
    assert rel(oracle.run(*mt, other)[0][-1:], want) > 0.3          # the far key decides the row
    for dtype in DTYPES:
        s = session(cuda, mt, dtype)
        assert close(s.feed(tok, [309]), want, dtype)
        s.reset()
        s.feed(tok[:309])
        assert close(s.feed(tok[309:], [0]), want, dtype)
        s.reset()
        s.feed(tok[:290])
        assert close(s.feed(tok[290:], [19]), want, dtype)
        s.close()


@pytest.mark.gpu
def test_old_token_stays_in_the_delta_state(cuda):
    """With decays close to one, the first token of the sequence still shows after two hundred others."""
    mt = make([delta(ff=None)], seed=3, slow=9.0)
    tok = ids(220, seed=8)
    other = [(tok[0] + 1) % 120] + tok[1:]
    want = oracle.run(*mt, tok)[0][-20:]
    assert rel(oracle.run(*mt, other)[0][-20:], want) > 1e-3
    s = session(cuda, mt, "float32")
    s.feed(tok[:200])
    got = np.concatenate([s.feed([t], [0]) for t in tok[200:]])
    assert close(got, want, "float32")
    s.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_states_are_given_back(cuda, dtype):
    """A request after another one gives the bits it gives alone."""
    mt = make(MIX, seed=9)
    a, b = ids(90, seed=4), ids(40, seed=5)
    s = session(cuda, mt, dtype)

    def run(tok):
        s.reset()
        return np.concatenate([s.feed(tok[:-6], [len(tok) - 7])] + [s.feed([t], [0]) for t in tok[-6:]])
    alone = run(b)
    run(a)
    again = run(b)
    assert np.array_equal(alone, again)
    assert close(alone, oracle.run(*mt, b)[0][-7:], dtype)
    s.close()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(cuda, dtype):
    mt = make(MIX, seed=10, slow=1.0)
    tok = ids(150, seed=6)
    want = oracle.run(*mt, tok)[0]
    s = session(cuda, mt, dtype)
    got = np.concatenate([s.feed(tok[:10], [9])] + [s.feed([t], [0]) for t in tok[10:]])
    assert close(got, want[9:], dtype)
    s.close()


@pytest.mark.gpu
def test_replayed_graph_gives_the_eager_bits(cuda):
    mt = make(MIX, seed=12)
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
    mt = make(MIX, seed=13)
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
def test_command_line_and_runner(cuda, tmp_path):
    """The command line generates; bin/trace_run and the C++ runner give the session's logits."""
    mt = make(MIX, seed=14)
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
    got = np.concatenate([np.fromfile(str(tmp_path / ("%d.f32" % n)), np.float32).reshape(-1, 120) for n in (0, 1)])
    want = oracle.run(*mt, tok)[0][[3, 14, 19]]
    assert close(got, want, "bfloat16")
    # a compiled runlist through the C++ runner: prompt of 20 rows, the logits of the last
    blob = str(tmp_path / "m.wtop")
    r = run(sys.executable, "-m", "gehtp_b200", "compile", "--model", str(tmp_path), "--out", blob, "--max-tokens", "64", "--max-sel", "4")
    assert r.returncode == 0, r.stderr
    man = json.load(open(blob + ".json"))
    face = np.zeros(man["max_rows"] + man["max_sel"], np.int32)
    face[:20], face[man["max_rows"]] = tok, 19
    face.tofile(str(tmp_path / "in.raw"))
    (tmp_path / "job.txt").write_text("blob %s\ninput %s\noutput %s\nout_temp %d\nrows 20\nsel 1\n" % (blob, tmp_path / "in.raw", tmp_path / "out.raw", man["logits_temp"]))
    r = run(os.path.join(ROOT, "gehtp_b200", "gehtp_run"), "job", str(tmp_path / "job.txt"))
    assert r.returncode == 0, r.stdout
    assert close(np.fromfile(str(tmp_path / "out.raw"), np.float32).reshape(1, 120), want[2:], "bfloat16")


@pytest.mark.gpu
def test_limits_are_reported(cuda):
    mt = make(MIX, seed=15)
    s = session(cuda, mt, "bfloat16", max_tokens=64, max_rows=16, max_sel=2)
    with pytest.raises(ValueError):
        s.feed([120])
    with pytest.raises(ValueError):
        s.feed([1, 2], [2])
    with pytest.raises(ValueError):
        s.feed([])
    for rows, sel in ((0, 0), (17, 1), (4, 3), (1, 2)):
        with pytest.raises(EngineError):
            s.engine.set_rows(rows, sel)
    s.feed(ids(64))
    with pytest.raises(ValueError):
        s.feed([1])
    s.position = 0                                        # the engine itself refuses the 65th position
    with pytest.raises(EngineError, match="context too long"):
        s.feed([1])
    s.reset()
    assert close(s.feed([3], [0]), oracle.run(*mt, [3])[0], "bfloat16")
    s.close()
