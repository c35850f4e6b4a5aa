"""Kevatar decoders (windowed attention with bounded scores, channel-wise delta rule, lightning attention, sublayers normed on their
output, a token input in every layer) against the plain restatement in oracle/kevatar_oracle.py: each mechanism alone, prompts,
portions of prompts, decoding, mixed batches, reused slots, window edges, far tokens, generation."""
import copy
import json
import os
import subprocess

import numpy as np
import pytest

import kevatar_oracle as K
from test_layered import BF16_TOL, F32_TOL, ids, rel, rows_rel

BOTH = pytest.mark.parametrize("dtype", ["f32", "bf16"])
gpu = pytest.mark.gpu
YARN = dict(factor=4.0, original=64, fast=8.0, slow=1.0)


def layer(kind, mx, ff):
    return dict(type=kind, mixer=mx, mlp=dict(kind="dense", ff=ff) if ff else None)


def attention(heads=6, kv_heads=3, dim=20, vdim=28, window=7, dims=12, base=500.0, scaling=YARN, scale=0.3, cap=6.0, kv_from=None, ff=52):
    mx = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, softcap=cap, mask=dict(size=window) if window else None,
              rot=dict(base=base, dims=dims, scaling=scaling) if dims else None)
    if kv_from is not None:
        mx["kv_from"] = kv_from
    return layer("attention", mx, ff)


def delta(heads=4, kv_heads=2, dim=18, vdim=22, conv=3, ranks=(5, 7), ff=52):
    return layer("channel_delta", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv, _ranks=ranks), ff)


def lightning(heads=5, dim=13, vdim=18, decay=None, ff=52):
    return layer("lightning", dict(heads=heads, dim=dim, vdim=vdim, decay=decay or [1.0 - 0.5 ** (1 + 2 * i) for i in range(heads)]), ff)


def config(layers, width=72, vocab=131, eps=3e-5, side=5, scale=7.0):
    return dict(architecture="Kevatar", width=width, vocab=vocab, norm=dict(eps=eps), embedding=dict(scale=scale),
                token_side=dict(dim=side) if side else None, layers=layers)


CONFIGS = {
    # odd sizes everywhere, a borrower with a longer window and constants of its own, layers without a feed-forward
    "odd": config([attention(), delta(), lightning(), attention(window=19, scale=0.2, cap=3.0, kv_from=0, ff=0), delta(heads=3, kv_heads=3, dim=16, vdim=36, conv=5, ff=0)]),
    # everything that may be absent or 1: one key head, no window, no bound, no scaling, no rotation, one tap, no token input
    "bare": config([attention(heads=4, kv_heads=1, dim=16, vdim=16, window=0, cap=None, scaling=None, dims=16, scale=0.25), lightning(heads=1, dim=16, vdim=16, decay=[1.0]),
                    delta(heads=1, kv_heads=1, dim=16, vdim=48, conv=1, ranks=(1, 1)), attention(heads=2, kv_heads=2, dim=8, vdim=24, window=1, dims=0, cap=0.0)],
                   width=64, vocab=96, side=0, scale=1.0),
    # head sizes of larger models: every tensor-core path; nine query heads on one key head
    "large": config([attention(heads=4, kv_heads=2, dim=128, vdim=128, window=100, dims=64, scale=0.08, cap=15.0, ff=256),
                     delta(heads=4, kv_heads=2, dim=128, vdim=128, conv=4, ranks=(32, 48), ff=0), lightning(heads=3, dim=128, vdim=256, decay=[0.9, 0.97, 0.999], ff=256),
                     attention(heads=9, kv_heads=1, dim=64, vdim=96, window=160, dims=32, scale=0.1, cap=20.0, ff=0), lightning(heads=5, dim=64, vdim=64, ff=0),
                     delta(heads=3, kv_heads=3, dim=64, vdim=64, conv=2, ranks=(8, 40), ff=128), delta(heads=2, kv_heads=1, dim=32, vdim=96, conv=4, ff=0),
                     attention(heads=4, kv_heads=2, dim=128, vdim=128, window=257, dims=64, scale=0.08, cap=30.0, kv_from=0, ff=0)], width=256, vocab=384, side=32),
    # wider heads than the tensor-core kernels take
    "wide": config([attention(heads=2, kv_heads=1, dim=264, vdim=40, window=33, dims=24, scale=0.06), delta(heads=2, kv_heads=1, dim=256, vdim=200, conv=4),
                    attention(heads=3, kv_heads=3, dim=200, vdim=256, window=0, dims=40, scale=0.07, scaling=None), lightning(heads=2, dim=300, vdim=40)], width=128, vocab=160, side=9),
    "attention_only": config([attention(ff=0)], side=0),
    "delta_only": config([delta(ff=0)], side=0),
    "lightning_only": config([lightning(ff=0)], side=0),
}


class Ref:
    """The oracle's logits of one sequence (or rows of them), and how far rounding alone moves each row: a row whose norms divide by
    something small magnifies it, whoever computes it."""

    def __init__(self, cfg, w, tokens, rows=None):
        self.cfg, self.w, self.tokens, self.rows = cfg, w, tokens, rows
        self.full = K.forward(cfg, w, tokens)
        self.noise_of = {}

    def __getitem__(self, rows):
        part = copy.copy(self)                            # shares the runs
        part.rows = rows
        return part

    @property
    def want(self):
        return self.full if self.rows is None else self.full[self.rows]

    def noise(self, dtype):
        if dtype not in self.noise_of:
            other = K.forward(self.cfg, self.w, self.tokens, dtype=np.float32) if dtype == "f32" else K.forward(self.cfg, self.w, self.tokens, rounded=K.to_bf16)
            self.noise_of[dtype] = rows_rel(other, self.full)
        return self.noise_of[dtype] if self.rows is None else self.noise_of[dtype][self.rows]


def agree(got, refs, dtype):
    """Every row is within the tolerance or within eight times what rounding alone does to it; in bf16 one row in twenty-five (or one)
    may be three times as far."""
    refs = refs if isinstance(refs, list) else [refs]
    r = rows_rel(got, np.concatenate([x.want for x in refs]))
    tol = F32_TOL if dtype == "f32" else BF16_TOL
    if r.max() < tol:
        return True
    over = r / np.maximum(tol, 8 * np.concatenate([x.noise(dtype) for x in refs]))
    return bool(over.max() < 1) if dtype == "f32" else bool(over.max() < 3 and (over > 1).sum() <= max(1, 0.04 * len(r)))


@pytest.fixture(scope="module")
def ctx(device):
    """models and oracle runs, built once per (configuration, dtype)"""
    import luminal_jl_b200 as L

    class Ctx:
        models, refs, weights = {}, {}, {}

        def w(self, name):
            if name not in self.weights:
                self.weights[name] = K.random_weights(CONFIGS[name], seed=17)
            return self.weights[name]

        def model(self, name, dtype):
            if (name, dtype) not in self.models:
                self.models[name, dtype] = make(L, device, CONFIGS[name], self.w(name), dtype)
            return self.models[name, dtype]

        def session(self, name, dtype, batch=1, ctx=512):
            return L.Session(self.model(name, dtype), batch, ctx)

        def ref(self, name, tokens):
            key = (name, tuple(tokens))
            if key not in self.refs:
                self.refs[key] = Ref(CONFIGS[name], self.w(name), tokens)
            return self.refs[key]
    c = Ctx()
    yield c
    for m in c.models.values():
        m.close()


def make(L, device, cfg, w, dtype):
    m = L.models.build_model(device, cfg, dtype, shapes={k: v.shape for k, v in w.items()})
    m.set_weights(w)
    assert m.missing_weights() == []
    return m


def run(session, toks, cuts):
    """every position's logits, the tokens cut into portions"""
    session.reset()
    out, at = [], 0
    for n in cuts:
        out.append(session.extend([toks[at:at + n]], [list(range(n))]))
        at += n
    assert at == len(toks)
    return np.concatenate(out)


# ---------------------------------------------------------------------------------------------------------------------------
# without a GPU
# ---------------------------------------------------------------------------------------------------------------------------
def test_configuration_reader():
    from luminal_jl_b200 import models
    cfg = CONFIGS["odd"]
    layers = models.kevatar_layers(cfg, K.tensor_shapes(cfg))
    assert [x["mixer"] for x in layers] == ["attention", "channel_delta", "lightning", "attention", "channel_delta"]
    assert layers[3]["kv_from"] == 0 and layers[3]["window"] == 19 and layers[3]["ff"] == 0 and layers[0]["rot_scaling"] == YARN
    assert (layers[1]["decay_rank"], layers[1]["gate_rank"], layers[1]["conv"]) == (5, 7, 3)
    bare = models.kevatar_layers(CONFIGS["bare"], K.tensor_shapes(CONFIGS["bare"]))
    assert bare[0]["window"] is None and bare[0]["score_cap"] is None and bare[3]["rot_dims"] == 0
    with pytest.raises(ValueError, match="shapes"):
        models.kevatar_layers(cfg, {})
    with pytest.raises(ValueError, match="mixer"):
        models.kevatar_layers(dict(layers=[layer("convolution", dict(heads=1, dim=1, vdim=1), 0)]), {})


def test_shapes_of_a_weight_file(tmp_path):
    from luminal_jl_b200 import weights
    w = K.random_weights(CONFIGS["delta_only"], 3)
    weights.write_safetensors(str(tmp_path / "a.safetensors"), w, dtype="BF16")
    assert weights.safetensors_shapes(str(tmp_path)) == {k: v.shape for k, v in w.items()}


def test_oracle_delta_rule_overwrites():
    """With beta 1 and no decay, writing to a unit key makes the state return the new value for it, whatever was there."""
    rng = np.random.default_rng(1)
    k, S = rng.standard_normal(6), rng.standard_normal((6, 4))
    k /= np.linalg.norm(k)
    v = rng.standard_normal(4)
    assert np.allclose((S + np.outer(k, v - S.T @ k)).T @ k, v)


def test_oracle_convolution():
    rng = np.random.default_rng(2)
    y, taps = rng.standard_normal((9, 3)), rng.standard_normal((3, 4))
    want = np.stack([np.convolve(y[:, c], taps[c, ::-1])[:9] for c in range(3)], axis=1)
    assert np.allclose(K.short_conv(y, taps), want)


def test_oracle_rotation():
    f, m = K.rotation(dict(base=100.0, dims=8, scaling=None))
    g, one = K.rotation(dict(base=100.0, dims=8, scaling=dict(factor=1.0, original=32, fast=4.0, slow=1.0)))
    assert np.allclose(f, g) and m == one == 1.0
    g, m = K.rotation(dict(base=10000.0, dims=64, scaling=dict(factor=8.0, original=2048, fast=32.0, slow=1.0)))
    f, _ = K.rotation(dict(base=10000.0, dims=64))
    assert np.isclose(g[0], f[0]) and np.isclose(g[-1], f[-1] / 8.0) and 1.2 < m < 1.21
    assert np.all((g <= f + 1e-12) & (g >= f / 8.0 - 1e-12))


def test_oracle_window():
    """A token outside every window changes nothing, one inside does."""
    cfg = config([attention(ff=0, window=4)], side=0)
    w = K.random_weights(cfg, 5)
    a = ids(1, 9, 131)
    b = list(a)
    b[4] = (b[4] + 1) % 131
    la, lb = K.forward(cfg, w, a), K.forward(cfg, w, b)
    assert np.allclose(la[8], lb[8]) and not np.allclose(la[7], lb[7])


# ---------------------------------------------------------------------------------------------------------------------------
# prompts, decoding, portions
# ---------------------------------------------------------------------------------------------------------------------------
@gpu
@BOTH
@pytest.mark.parametrize("name", list(CONFIGS))
def test_prompt_every_position(ctx, name, dtype):
    s = ctx.session(name, dtype)
    for n in (1, 2, 3, 17, 65, 150):
        toks = ids(n, n, CONFIGS[name]["vocab"])
        assert agree(run(s, toks, [n]), ctx.ref(name, toks), dtype), (name, n)
    s.close()


@gpu
@BOTH
@pytest.mark.parametrize("name", ["odd", "bare", "large", "wide"])
def test_decoding_equals_prompt(ctx, name, dtype):
    toks = ids(7, 140, CONFIGS[name]["vocab"])
    ref = ctx.ref(name, toks)
    s = ctx.session(name, dtype)
    assert agree(run(s, toks, [1] * 140), ref, dtype)
    assert agree(run(s, toks, [100] + [1] * 40), ref, dtype)
    s.close()


@gpu
@BOTH
@pytest.mark.parametrize("name", ["odd", "bare", "large"])
def test_portions(ctx, name, dtype):
    toks = ids(8, 330, CONFIGS[name]["vocab"])
    ref = ctx.ref(name, toks)
    s = ctx.session(name, dtype)
    for cuts in ([2] * 12 + [3, 5, 1, 1, 40, 64, 65, 63, 64], [64, 64, 64, 64, 74], [1, 329], [128, 2, 127, 2, 71], [15, 16, 17, 18, 264], [200, 128, 2], [63, 2, 65, 200],
                 [7, 8, 9, 10, 11, 285], [2] * 165):
        got = run(s, toks, cuts)
        assert agree(got, ref, dtype), (name, cuts)
    s.close()


@gpu
@BOTH
def test_layer_outputs(ctx, dtype):
    """the residual stream after every layer, from a prompt, a portion and a decoded token"""
    for name in ("odd", "bare"):
        toks = ids(3, 41, CONFIGS[name]["vocab"])
        _, ref = K.forward(CONFIGS[name], ctx.w(name), toks, return_layers=True)
        s = ctx.session(name, dtype)
        s.set_capture(True)
        for at, n in ((0, 30), (30, 10), (40, 1)):
            s.extend([toks[at:at + n]])
            for l, r in enumerate(ref):
                assert rel(s.layer_output(l), r[at + n - 1:at + n]) < (1e-5 if dtype == "f32" else 3e-2), (name, at, l)
        s.close()


@gpu
def test_long_decoding(ctx):
    """hundreds of decoded tokens on one state and one cache (bf16 graph replays), checked along the way"""
    name, toks = "large", ids(5, 700, 384)
    ref = ctx.ref(name, toks)
    s = ctx.session(name, "bf16", ctx=704)
    s.extend([toks[:40]])
    for t in range(40, 700):
        got = s.extend([[toks[t]]], [[0] if t % 60 == 0 or t > 690 else []])
        if len(got):
            assert agree(got, ref[t:t + 1], "bf16"), t
    s.close()


# ---------------------------------------------------------------------------------------------------------------------------
# far tokens and edges, made visible by weights that single one token out
# ---------------------------------------------------------------------------------------------------------------------------
def needle_weights(cfg, seed):
    """Weights under which the first layer's attention is close to a copy: token 0 asks, token 1 answers, every other key scores low.  The
    shared direction lies behind the rotated features, so distance does not turn it away."""
    w = K.random_weights(cfg, seed)
    mx, s = cfg["layers"][0]["mixer"], cfg["embedding"]["scale"]
    w["embed"] = K.to_bf16(0.3 * w["embed"])
    w["embed"][0, 0] = w["embed"][1, 1] = K.to_bf16([12.0 / s])[0]
    for n, f, heads in (("q", 0, mx["heads"]), ("k", 1, mx["kv_heads"])):
        m = w[f"l0.mix.{n}"]
        m[:, f] = 0.0
        for h in range(heads):
            m[(h + 1) * mx["dim"] - 1, f] = 4.0
    return w


@gpu
@BOTH
@pytest.mark.parametrize("sizes", [dict(scale=1.3), dict(heads=4, kv_heads=2, dim=128, vdim=128, dims=64, scale=0.08), dict(heads=2, kv_heads=2, dim=64, vdim=80, dims=16, scale=0.125)])
def test_window_edges(device, dtype, sizes):
    """One key carries most of the asking token's weight while it is in the window and none of it one position further: windows that
    end at, before and after multiples of 16, 64 and 128, in prompts, portions and decoding."""
    import luminal_jl_b200 as L
    for window in (1, 2, 40, 64, 65, 129, 300, 0):
        cfg = config([attention(ff=0, cap=20.0, window=window, **dict(dict(scale=0.5), **sizes))], width=128, vocab=64, side=0)
        w = needle_weights(cfg, 4)
        m = make(L, device, cfg, w, dtype)
        s = L.Session(m, 1, 640)
        shifts = {True: [], False: []}
        for n in (3, 200, 257, 513):
            for key in {n - 2, n - window, n - window - 1, 0, n - 130}:
                if not 0 <= key < n - 1:
                    continue
                seen = window == 0 or n - 1 - key < window
                toks = [2 + t % 60 for t in ids(n + key, n, 60)]
                toks[key], toks[-1] = 1, 0
                ref = Ref(cfg, w, toks)[-1:]
                without = list(toks)
                without[key] = 7
                shifts[seen].append(rel(K.forward(cfg, w, without)[-1:], ref.want))
                for cuts in ([n], [n - 1, 1], [n // 2, n - n // 2], [max(1, n - 3), min(3, n - 1)], [max(1, n - 40), min(40, n - 1)]):
                    s.reset()
                    at = 0
                    for c in cuts:
                        got = s.extend([toks[at:at + c]], [[c - 1]])
                        at += c
                    assert agree(got, ref, dtype), (window, n, key, cuts)
        assert all(x > 0.05 for x in shifts[True]) and all(x < 1e-9 for x in shifts[False])
        s.close()
        m.close()


@gpu
@BOTH
def test_borrowed_window_is_longer(device, dtype):
    """A borrower's window may reach past its source's: the source's cache keeps every position."""
    import luminal_jl_b200 as L
    cfg = config([attention(ff=0, window=3, cap=20.0, scale=0.5), attention(ff=0, window=90, cap=20.0, scale=0.5, kv_from=0)], width=128, vocab=64, side=0)
    w = needle_weights(cfg, 6)
    w["l0.norm1"] *= 0.05                                # what the first layer adds leaves the tokens recognisable
    w["l0.norm1"] = K.to_bf16(w["l0.norm1"])
    w["l1.mix.q"] = w["l0.mix.q"].copy()
    m = make(L, device, cfg, w, dtype)
    s = L.Session(m, 1, 256)
    for key in (0, 109, 110, 111, 150):
        toks = [2 + t % 60 for t in ids(key, 200, 60)]
        toks[key], toks[-1] = 1, 0
        ref = Ref(cfg, w, toks)
        for cuts in ([200], [150, 50], [199, 1], [100, 98, 2]):
            assert agree(run(s, toks, cuts), ref, dtype), (key, cuts)
    s.close()
    m.close()


@gpu
@BOTH
@pytest.mark.parametrize("dims", [(10, 14), (128, 128), (64, 192)])
def test_delta_remembers_one_token(device, dtype, dims):
    """Only one token writes strongly (beta) and nothing decays: its value is read hundreds of tokens later, wherever it was written."""
    import luminal_jl_b200 as L
    D, V = dims
    cfg = config([delta(heads=2, kv_heads=1, dim=D, vdim=V, conv=4, ff=0)], width=128, vocab=64, side=0, scale=1.0)
    w = K.random_weights(cfg, 9)
    p = "l0.mix."
    w["embed"][:, 1:3] = 0.0
    w["embed"][1, 1] = 4.0                               # feature 1: the writing token; feature 2: every token
    w["embed"][:, 2] = 2.0
    w[p + "b"][:] = K.to_bf16(0.02 * w[p + "b"])
    w[p + "b"][:, 1], w[p + "b"][:, 2] = 3.0, -4.0       # beta is a sigmoid of about -8, of +4 for the writer
    w[p + "A_log"][:], w[p + "dt_bias"][:] = -8.0, -4.0
    for n in "qk":                                       # a common part in every key and query
        w[p + n][:, 2] = K.to_bf16(2.0 + 0 * w[p + n][:, 2])
    m = make(L, device, cfg, w, dtype)
    s = L.Session(m, 1, 512)
    n, moved = 300, 0.0
    for key in (0, 1, 15, 16, 62, 63, 64, 65, 127, 128):
        toks = [2 + t % 60 for t in ids(key, n, 60)]
        toks[key] = 1
        ref = Ref(cfg, w, toks)
        without = list(toks)
        without[key] = 7
        moved = max(moved, rel(K.forward(cfg, w, without)[-1:], ref[-1:].want))
        for cuts in ([n], [64, 64, 172], [63, 2, 235], [129, 1, 1, 169], [5, 2, 2, 291]):
            assert agree(run(s, toks, cuts), ref, dtype), (key, cuts)
    assert moved > 0.2
    s.close()
    m.close()


@gpu
@BOTH
@pytest.mark.parametrize("dims", [(10, 14), (128, 128), (64, 64)])
@pytest.mark.parametrize("rate", [(3.0, 4.0), (-6.0, -5.0), (0.5, -1.0), (0.5, 0.0), (1.0, -0.2), (1.0, 0.0), None])
def test_delta_decays(device, dtype, dims, rate):
    """Decays from nearly none to a factor below any float within a few tokens, and both next to each other."""
    import luminal_jl_b200 as L
    D, V = dims
    cfg = config([delta(heads=4, kv_heads=2, dim=D, vdim=V, conv=2, ff=0)], width=96, vocab=64, side=0)
    w = K.random_weights(cfg, 12)
    rng = np.random.default_rng(1)
    if rate:
        w["l0.mix.A_log"][:], w["l0.mix.dt_bias"][:] = rate
    else:
        w["l0.mix.A_log"][:] = [3.0, -6.0, 1.0, -1.0]
        w["l0.mix.dt_bias"][:] = K.to_bf16(rng.choice([-8.0, -2.0, 0.0, 5.0], 4 * D))
    m = make(L, device, cfg, w, dtype)
    s = L.Session(m, 1, 512)
    toks = ids(2, 280, 64)
    ref = Ref(cfg, w, toks)
    for cuts in ([280], [64, 64, 152], [65, 2, 63, 150], [17, 15, 248], [130] + [1] * 10 + [140]):
        assert agree(run(s, toks, cuts), ref, dtype), cuts
    s.close()
    m.close()


@gpu
@BOTH
@pytest.mark.parametrize("dims", [(9, 6), (128, 128), (64, 192)])
def test_lightning_remembers_one_token(device, dtype, dims):
    """With decay 1 and faint other tokens, the state is one outer product written far back."""
    import luminal_jl_b200 as L
    D, V = dims
    cfg = config([lightning(heads=2, dim=D, vdim=V, decay=[1.0, 0.9995], ff=0)], width=128, vocab=64, side=0, scale=1.0)
    w = K.random_weights(cfg, 9)
    k = 0.05 * w["l0.mix.k"]
    k[:, 1] = w["l0.mix.k"][:, 1] * 6.0                  # only feature 1 writes strongly, and only token 1 has it
    w["l0.mix.k"] = K.to_bf16(k)
    w["embed"][:, 1] = 0.0
    w["embed"][1, :] = K.to_bf16(0.1 * w["embed"][1])
    w["embed"][1, 1] = 9.0
    w["embed"][:, 2] = 2.0
    w["l0.mix.q"][:, 2] = np.abs(k[:, 1])
    m = make(L, device, cfg, w, dtype)
    s = L.Session(m, 1, 512)
    n = 300
    for key in (0, 1, 62, 63, 64, 65, 127, 128):
        toks = [2 + t % 60 for t in ids(key, n, 60)]
        toks[key] = 1
        ref = Ref(cfg, w, toks)
        for cuts in ([n], [64, 64, 172], [63, 2, 235], [129, 1, 1, 169], [5, 2, 2, 291]):
            assert agree(run(s, toks, cuts), ref, dtype), (key, cuts)
    s.close()
    m.close()


# ---------------------------------------------------------------------------------------------------------------------------
# batches, slots
# ---------------------------------------------------------------------------------------------------------------------------
@gpu
@BOTH
@pytest.mark.parametrize("name", ["odd", "large"])
def test_mixed_batch(ctx, name, dtype):
    """prompts, portions and single tokens of unequal requests in one call, each against itself alone"""
    V = CONFIGS[name]["vocab"]
    toks = [ids(50 + i, n, V) for i, n in enumerate((200, 33, 5, 90))]
    ref = [ctx.ref(name, t) for t in toks]
    s = ctx.session(name, dtype, batch=4)
    at = [0] * 4
    for plan in ((100, 1, 2, 0), (1, 1, 1, 1), (1, 20, 1, 64), (70, 1, 0, 2), (1, 1, 1, 1), (27, 9, 0, 22)):
        part = [t[a:a + n] for t, a, n in zip(toks, at, plan)]
        got = s.extend(part, [list(range(n)) for n in plan])
        assert agree(got, [r[a:a + n] for r, a, n in zip(ref, at, plan)], dtype), plan
        at = [a + n for a, n in zip(at, plan)]
    assert list(s.positions()) == at
    s.close()


@gpu
@BOTH
def test_equal_prompts_then_decoding(ctx, dtype):
    """prompts of one length share their launches; then every sequence decodes at the same and at different positions"""
    name, V = "large", 384
    toks = [ids(80 + b, 110, V) for b in range(3)]
    ref = [ctx.ref(name, t) for t in toks]
    s = ctx.session(name, dtype, batch=3)
    for n in (70, 33):
        a = s.positions()[0]
        got = s.extend([t[a:a + n] for t in toks], [list(range(n))] * 3)
        assert agree(got, [r[a:a + n] for r in ref], dtype)
    for i in range(103, 107):
        assert agree(s.extend([[t[i]] for t in toks], [[0]] * 3), [r[i:i + 1] for r in ref], dtype)
    s.extend([toks[0][107:108], [], toks[2][107:109]])
    p = s.positions()
    assert agree(s.extend([[t[a]] for t, a in zip(toks, p)], [[0]] * 3), [r[a:a + 1] for r, a in zip(ref, p)], dtype)
    s.close()


@gpu
@BOTH
def test_slots_used_again(ctx, dtype):
    import luminal_jl_b200 as L
    name, V = "odd", 131
    pool = L.RequestPool(ctx.session(name, dtype, batch=3, ctx=256))
    reqs = {i: ids(90 + i, n, V) for i, n in enumerate((120, 9, 64, 31, 200, 2, 77))}
    live, at, todo, step = [], {}, list(reqs), 0
    while live or todo:
        while todo and len(live) < 3:
            live.append(todo.pop(0))
            at[live[-1]] = 0
        sizes = [(1, 30, 2, 64, 7)[(step + k) % 5] for k in range(len(live))]
        entries = []
        for r, n in zip(live, sizes):
            part = reqs[r][at[r]:at[r] + n]
            entries.append((r, part, list(range(len(part)))))
        for (r, part, _), got in zip(entries, pool.step(entries)):
            assert agree(got, ctx.ref(name, reqs[r])[at[r]:at[r] + len(part)], dtype), (r, at[r])
            at[r] += len(part)
        done = [r for r in live if at[r] == len(reqs[r])]
        pool.end(done)
        live = [r for r in live if r not in done]
        step += 1
    pool.session.close()


@gpu
@BOTH
def test_wide_batches(ctx, dtype):
    """sixteen, thirty-two and more sequences than one weight pass serves, decoded together"""
    name, V = "odd", 131
    for B in (16, 17, 32, 40):
        toks = [ids(300 + b, 3 + b % 7, V) for b in range(B)]
        s = ctx.session(name, dtype, batch=B, ctx=64)
        got = s.extend(toks, [[len(t) - 1] for t in toks])
        assert agree(got, [ctx.ref(name, t)[-1:] for t in toks], dtype)
        nxt = ids(B, B, V)
        got = s.extend([[t] for t in nxt], [[0]] * B)
        assert agree(got, [ctx.ref(name, t + [x])[-1:] for t, x in zip(toks, nxt)], dtype)
        s.close()


@gpu
def test_positions_of_a_recurrent_state(ctx, device):
    import luminal_jl_b200 as L
    s = ctx.session("odd", "f32", batch=2, ctx=64)
    s.extend([[1, 2, 3], [4, 5]])
    with pytest.raises(L.LuminalB200Error, match="recurrent state"):
        s.set_position(1)
    s.set_positions([0, 2])                              # one slot is emptied, the other left alone
    got = s.extend([[7, 8], [9]], [[1], [0]])
    assert agree(got, [ctx.ref("odd", [7, 8])[-1:], ctx.ref("odd", [4, 5, 9])[-1:]], "f32")
    s.close()


# ---------------------------------------------------------------------------------------------------------------------------
# generation through the framework's own entry points
# ---------------------------------------------------------------------------------------------------------------------------
def oracle_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(K.forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]


@gpu
def test_greedy_generation(ctx):
    import luminal_jl_b200 as L
    name, V = "odd", 131
    prompts = [ids(70 + b, 12, V) for b in range(3)]
    want = np.array([oracle_greedy(CONFIGS[name], ctx.w(name), p, 20) for p in prompts])
    s = ctx.session(name, "f32", batch=3, ctx=64)
    assert np.array_equal(L.greedy_generate(s, np.array(prompts), 20), want)
    s.reset()
    first = s.prefill(np.array(prompts)).argmax(-1).astype(np.int32)
    assert np.array_equal(first, want[:, 0])
    assert np.array_equal(s.decode_n(first, 19).T, want[:, 1:])        # device-resident loop
    s.reset()                                                          # continue from the prompt's own best token
    s.prefill_ragged(prompts)
    assert np.array_equal(s.decode_n(None, 19).T, want[:, 1:])
    s.close()


@gpu
@BOTH
def test_pool_generation(ctx, dtype):
    """continuous batching: five requests over two slots give what each gives alone"""
    import luminal_jl_b200 as L
    name, V = "odd", 131
    prompts = {i: ids(40 + i, n, V) for i, n in enumerate((20, 3, 50, 1, 9))}
    pool = L.RequestPool(ctx.session(name, dtype, batch=2, ctx=128))
    got = pool.generate(prompts, 8)
    for i, p in prompts.items():
        if dtype == "f32":
            assert got[i] == oracle_greedy(CONFIGS[name], ctx.w(name), p, 8)
        else:                                            # bf16: every chosen token is within rounding of the best
            ref = ctx.ref(name, p + got[i])
            for j, t in enumerate(got[i]):
                row = ref.full[len(p) - 1 + j]
                assert row.max() - row[t] < 4 * BF16_TOL * row.std()
    pool.session.close()


@gpu
def test_model_folder_and_replay(device, tmp_path):
    """a folder with config.json and bf16 safetensors through load_model and through bin/trace_run"""
    import luminal_jl_b200 as L
    cfg = copy.deepcopy(CONFIGS["odd"])
    w = K.random_weights(cfg, 21)
    for x in cfg["layers"]:
        x["mixer"].pop("_ranks", None)                   # the loader takes them from the tensors
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    L.weights.write_safetensors(str(folder / "model.safetensors"), w, dtype="BF16")
    toks = ids(1, 30, 131)
    ref = K.forward(cfg, w, toks)
    m = L.load_model(device, str(folder), "f32")
    s = L.Session(m, 1, 64)
    assert rel(s.extend([toks], [[29]]), ref[29:]) < F32_TOL
    s.close()
    m.close()
    steps = [dict(step=0, entries=[dict(id="x", tokens=toks[:20], want=[0, 19])], end=[]),
             dict(step=1, entries=[dict(id="x", tokens=toks[20:21], want=[])], end=[]),
             dict(step=2, entries=[dict(id="x", tokens=toks[21:], want=[8])], end=["x"]),
             dict(step=3, entries=[dict(id="y", tokens=toks[:3], want=[2])], end=["y"])]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype, t in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "30"],
                           input="\n".join(json.dumps(x) for x in steps) + "\n", capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr[-2000:]
        for n, rows in ((0, [0, 19]), (2, [29]), (3, [2])):
            got = np.fromfile(out / f"{n}.f32", "<f4").reshape(len(rows), -1)
            assert rel(got, ref[rows]) < t


@gpu
def test_bad_configurations_are_refused(device):
    import luminal_jl_b200 as L
    for layers, what in (([attention(kv_from=0)], "kv_from"), ([attention(), attention(kv_from=0, vdim=12)], "widths"), ([delta(), attention(kv_from=0)], "widths"),
                         ([attention(heads=4, kv_heads=3)], "key heads"), ([lightning(heads=2, decay=[0.5, 1.5])], "decay"), ([attention(dim=8, dims=12)], "rotated"),
                         ([delta(dim=300)], "256"), ([delta(conv=17)], "taps")):
        cfg = config(layers)
        with pytest.raises(L.LuminalB200Error, match=what):
            L.models.build_model(device, cfg, "f32", shapes=K.tensor_shapes(cfg))
