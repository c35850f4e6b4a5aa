"""Decoders described layer by layer (latent attention, retention, parallel feed-forward) against the plain restatement in
oracle/gibutar_oracle.py: each mechanism alone, prompts, portions of prompts, decoding, mixed batches, reused slots, generation."""
import json

import numpy as np
import pytest

import gibutar_oracle as G

F32_TOL, BF16_TOL = 2e-5, 3.5e-2          # of the logits' spread; what rounding alone leaves


def latent(heads=3, dim=24, rot_dim=8, vdim=16, kv_rank=40, q_rank=56, base=5000.0, scale=0.2, kv_from=None, ff=80):
    mx = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale,
              rot=dict(base=base, dims=rot_dim))
    if kv_from is not None:
        mx["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=mx, mlp=dict(kind="dense", ff=ff) if ff else None)


def retention(heads=3, dim=20, vdim=28, dims=12, base=300.0, decay=None, ff=80):
    mx = dict(heads=heads, dim=dim, vdim=vdim, rot=dict(base=base, dims=dims), decay=decay or [1.0 - 0.5 ** (1 + 2 * i) for i in range(heads)])
    return dict(type="retention", mixer=mx, mlp=dict(kind="dense", ff=ff) if ff else None)


def config(layers, width=72, vocab=131, eps=3e-5, cap=9.0):
    return dict(architecture="Gibutar", width=width, vocab=vocab, norm=dict(eps=eps), logit_softcap=cap, layers=layers)


CONFIGS = {
    # odd sizes everywhere, a layer that borrows its latents, layers without a feed-forward
    "odd": config([retention(), latent(), latent(heads=5, dim=10, vdim=12, q_rank=33, scale=0.4, kv_from=1, ff=0), retention(heads=1, dim=8, vdim=6, dims=8, decay=[0.9])]),
    # a borrower two layers on, a second cache, decays at both ends, no bound on the logits
    "borrow": config([latent(ff=0, heads=2, dim=32, rot_dim=16, vdim=24, kv_rank=64, q_rank=48), retention(heads=2, dim=16, vdim=32, dims=16, decay=[0.25, 1.0]),
                      latent(kv_from=0, heads=4, dim=16, rot_dim=16, vdim=8, kv_rank=64, q_rank=40), latent(heads=2, base=777.0), latent(kv_from=3, heads=1, base=777.0)],
                     width=96, vocab=200, cap=None),
    # head sizes of larger models: every tensor-core path
    "large": config([latent(heads=4, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=256, scale=0.07, base=10000.0, ff=512),
                     retention(heads=3, dim=128, vdim=256, dims=128, base=10000.0, ff=256, decay=[0.9, 0.97, 0.999]),
                     latent(heads=18, dim=64, rot_dim=64, vdim=64, kv_rank=512, q_rank=192, scale=0.1, kv_from=0, base=10000.0, ff=0),
                     retention(heads=2, dim=256, vdim=128, dims=64, base=10000.0, ff=128, decay=[0.6, 0.99])], width=256, vocab=384),
    "latent_only": config([latent(ff=0)]),
    "retention_only": config([retention(ff=0)]),
}


def rows_rel(got, want):
    d, w = np.asarray(got, np.float64) - want, want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())


def rel(got, want):
    """Root mean square of the difference over that of the (centred) reference, worst row."""
    return float(rows_rel(got, want).max())


def agree(got, want, dtype):
    """float32: every row within rounding.  bf16: a retention output that nearly cancels before its norm magnifies rounding (random
    weights make a few such rows), so one row in twenty-five (or one) may be up to three times over."""
    r = rows_rel(got, want)
    if dtype == "f32":
        return bool(r.max() < F32_TOL)
    return bool(r.max() < 3 * BF16_TOL and (r > BF16_TOL).sum() <= max(1, 0.04 * len(r)))


def ids(seed, n, vocab):
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, n)]


@pytest.fixture(scope="module")
def ctx(device):
    """models and oracle runs, built once per (configuration, dtype)"""
    import luminal_jl_b200 as L

    class Ctx:
        models, refs, weights = {}, {}, {}

        def w(self, name):
            if name not in self.weights:
                self.weights[name] = G.random_weights(CONFIGS[name], seed=11)
            return self.weights[name]

        def model(self, name, dtype):
            if (name, dtype) not in self.models:
                m = L.models.build_model(device, CONFIGS[name], dtype)
                m.set_weights(self.w(name))
                assert m.missing_weights() == []
                self.models[name, dtype] = m
            return self.models[name, dtype]

        def session(self, name, dtype, batch=1, ctx=512):
            return L.Session(self.model(name, dtype), batch, ctx)

        def ref(self, name, tokens):
            key = (name, tuple(tokens))
            if key not in self.refs:
                self.refs[key] = G.forward(CONFIGS[name], self.w(name), tokens)
            return self.refs[key]
    c = Ctx()
    yield c
    for m in c.models.values():
        m.close()


BOTH = pytest.mark.parametrize("dtype", ["f32", "bf16"])
gpu = pytest.mark.gpu


# ---------------------------------------------------------------------------------------------------------------------------
# without a GPU
# ---------------------------------------------------------------------------------------------------------------------------
def test_configuration_reader():
    from luminal_jl_b200 import models
    layers = models.gibutar_layers(CONFIGS["odd"])
    assert [x["mixer"] for x in layers] == ["retention", "latent_attention", "latent_attention", "retention"]
    assert layers[2]["kv_from"] == 1 and layers[1]["kv_from"] is None and layers[2]["ff"] == 0 and layers[0]["ff"] == 80
    assert layers[0]["rot_layout"] == "half" and layers[1]["rot_layout"] == "interleaved"
    with pytest.raises(ValueError, match="not registered"):
        models.architecture(dict(architecture="Unheard"))
    with pytest.raises(ValueError, match="mixer"):
        models.gibutar_layers(dict(layers=[dict(type="convolution", mixer=dict(heads=1, dim=1, vdim=1), mlp=None)]))


def test_oracle_retention_is_the_masked_product():
    """The recurrence equals the sum over earlier tokens with decay to the power of the distance."""
    rng = np.random.default_rng(1)
    T, D, V, g = 9, 6, 5, 0.7
    cfg = retention(heads=1, dim=D, vdim=V, dims=4, decay=[g], ff=0)["mixer"]
    p, W = "l0.mix.", 7
    w = {p + n: rng.standard_normal(s) for n, s in (("q", (D, W)), ("k", (D, W)), ("v", (V, W)), ("g", (V, W)), ("o", (W, V)))}
    h, pos = rng.standard_normal((T, W)), np.arange(T, dtype=float)
    q = G.rotate((h @ w[p + "q"].T)[None], pos, 300.0, 4, False)[0]
    k = G.rotate((h @ w[p + "k"].T)[None], pos, 300.0, 4, False)[0] / np.sqrt(D)
    dist = pos[:, None] - pos[None]
    a = np.where(dist >= 0, g ** np.maximum(dist, 0), 0.0) * (q @ k.T)
    y = (G.rms(a @ (h @ w[p + "v"].T), 1e-6) * G.silu(h @ w[p + "g"].T)) @ w[p + "o"].T
    assert np.allclose(y, G.retention(h, w, p, cfg, 1e-6, pos))


def test_oracle_rotation_depends_on_distance_only():
    rng = np.random.default_rng(2)
    q, k = rng.standard_normal((2, 1, 1, 10))
    for inter in (False, True):
        at = lambda x, p: G.rotate(x, np.array([float(p)]), 50.0, 6, inter)
        assert np.isclose((at(q, 12) * at(k, 7)).sum(), (at(q, 105) * at(k, 100)).sum())
        assert np.array_equal(at(q, 12)[..., 6:], q[..., 6:])


class FakeSession:
    """echoes position, sequence and token so that the pool's bookkeeping shows"""
    def __init__(self, batch):
        self.batch, self.pos = batch, np.zeros(batch, np.int32)

    def extend(self, tokens, want):
        rows = [[b, self.pos[b] + p, tokens[b][p]] for b in range(self.batch) for p in want[b]]
        self.pos += np.array([len(t) for t in tokens], np.int32)
        return np.array(rows, np.float32).reshape(-1, 3)

    def positions(self):
        return self.pos.copy()

    def set_positions(self, p):
        self.pos = np.array(p, np.int32)


def test_request_pool_slots():
    from luminal_jl_b200.requests import RequestPool
    pool = RequestPool(FakeSession(2))
    a = pool.step([("a", [5, 6, 7], [2])])
    assert a[0].tolist() == [[0, 2, 7]]
    b, a = pool.step([("b", [9, 8], [0, 1]), ("a", [4], [0])])
    assert b.tolist() == [[1, 0, 9], [1, 1, 8]] and a.tolist() == [[0, 3, 4]]
    with pytest.raises(RuntimeError, match="slots"):
        pool.step([("c", [1], [])])
    pool.end(["a"])
    assert pool.step([("c", [1], [0])])[0].tolist() == [[0, 0, 1]]
    assert list(pool.session.pos) == [1, 2]


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
        s.reset()
        got = s.extend([toks], [list(range(n))])
        assert agree(got, ctx.ref(name, toks), dtype), (name, n)
    s.close()


@gpu
@BOTH
@pytest.mark.parametrize("name", ["odd", "borrow", "large"])
def test_decoding_equals_prompt(ctx, name, dtype):
    toks = ids(7, 140, CONFIGS[name]["vocab"])
    ref = ctx.ref(name, toks)
    s = ctx.session(name, dtype)
    got = np.concatenate([s.extend([[t]], [[0]]) for t in toks])
    assert agree(got, ref, dtype)
    s.reset()                                     # a prompt, then one by one
    s.extend([toks[:100]])
    got = np.concatenate([s.extend([[t]], [[0]]) for t in toks[100:]])
    assert agree(got, ref[100:], dtype)
    s.close()


@gpu
@BOTH
@pytest.mark.parametrize("name", ["odd", "borrow", "large"])
def test_portions(ctx, name, dtype):
    toks = ids(8, 330, CONFIGS[name]["vocab"])
    ref = ctx.ref(name, toks)
    s = ctx.session(name, dtype)
    for cuts in ([2] * 12 + [3, 5, 1, 1, 40, 64, 65, 63, 64], [64, 64, 64, 64, 74], [1, 329], [128, 2, 127, 2, 71], [15, 16, 17, 18, 264], [200, 128, 2], [63, 2, 65, 200]):
        assert sum(cuts) <= len(toks)
        s.reset()
        at = 0
        for n in cuts:
            got = s.extend([toks[at:at + n]], [list(range(n))])
            assert agree(got, ref[at:at + n], dtype), (name, cuts, at, n)
            at += n
    s.close()


@gpu
@BOTH
def test_layer_outputs(ctx, dtype):
    """the residual stream after every layer, from a prompt, a portion and a decoded token"""
    name, toks = "odd", ids(3, 41, 131)
    _, ref = G.forward(CONFIGS[name], ctx.w(name), toks, return_layers=True)
    s = ctx.session(name, dtype)
    s.set_capture(True)
    for at, n in ((0, 30), (30, 10), (40, 1)):
        s.extend([toks[at:at + n]])
        for l, r in enumerate(ref):
            assert rel(s.layer_output(l), r[at + n - 1:at + n]) < (1e-5 if dtype == "f32" else 3e-2), (at, l)
    s.close()


@gpu
def test_long_decoding(ctx):
    """hundreds of decoded tokens on one state and one cache (bf16 graph replays), checked along the way"""
    name, toks = "borrow", ids(5, 700, 200)
    ref = ctx.ref(name, toks)
    s = ctx.session(name, "bf16", ctx=704)
    s.extend([toks[:40]])
    for t in range(40, 700):
        got = s.extend([[toks[t]]], [[0] if t % 60 == 0 or t > 690 else []])
        if len(got):
            assert rel(got, ref[t:t + 1]) < BF16_TOL, t
    s.close()


# ---------------------------------------------------------------------------------------------------------------------------
# far keys and edges, made visible by weights that single one key out
# ---------------------------------------------------------------------------------------------------------------------------
def needle_weights(cfg, seed):
    """Weights under which latent attention is close to a copy: token 0 asks, token 1 answers, every other key scores low."""
    w = G.random_weights(cfg, seed)
    width, mx = cfg["width"], cfg["layers"][0]["mixer"]
    w["embed"] = G.to_bf16(0.05 * w["embed"])
    w["embed"][0, 0] = w["embed"][1, 1] = 8.0          # both norm to about sqrt(width) on one feature
    w["l0.norm1"] = np.ones(width, np.float32)
    for n, f in (("dq", 0), ("dkv", 1)):                # the asking feature excites query latent 0, the answering one key latent 0
        m = 0.02 * w[f"l0.mix.{n}"]
        m[0, f] = 2.0
        w[f"l0.mix.{n}"] = G.to_bf16(m)
    H, dim, rd = mx["heads"], mx["dim"], mx["rot_dim"]
    uq, uk = 0.05 * w["l0.mix.uq"], 0.05 * w["l0.mix.uk"]
    for h in range(H):
        uq[h * (dim + rd), 0] = 3.0
        uk[h * dim, 0] = 3.0
    w["l0.mix.uq"], w["l0.mix.uk"] = G.to_bf16(uq), G.to_bf16(uk)
    return w


@gpu
@BOTH
@pytest.mark.parametrize("sizes", [dict(), dict(heads=4, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=256)])
def test_one_far_key(device, dtype, sizes):
    """One key far back carries almost all the weight of the asking token, wherever it sits: first and last token, either side of
    multiples of 16, 64 and 128, in a prompt, in a portion and in decoding."""
    import luminal_jl_b200 as L
    cfg = config([latent(ff=0, scale=0.05, **sizes)], width=128, vocab=64)
    w = needle_weights(cfg, 4)
    m = L.models.build_model(device, cfg, dtype)
    m.set_weights(w)
    s = L.Session(m, 1, 640)
    shift = 0.0
    for n, key in ((2, 0), (200, 0), (200, 198), (257, 15), (257, 16), (300, 63), (300, 64), (300, 127), (301, 128), (513, 255), (513, 256), (600, 1), (600, 511)):
        toks = [2 + t % 60 for t in ids(n + key, n, 60)]
        toks[key], toks[-1] = 1, 0
        ref = G.forward(cfg, w, toks)[-1:]
        without = list(toks)
        without[key] = 7
        shift = max(shift, rel(G.forward(cfg, w, without)[-1:], ref))
        for cuts in ([n], [n - 1, 1], [n // 2, n - n // 2], [max(1, n - 3), min(3, n - 1)]):
            s.reset()
            at = 0
            for c in cuts:
                got = s.extend([toks[at:at + c]], [[c - 1]])
                at += c
            assert agree(got, ref, dtype), (n, key, cuts)
    assert shift > 0.3                                  # the key does show
    s.close()
    m.close()


@gpu
@BOTH
@pytest.mark.parametrize("dims", [(20, 28), (128, 128), (64, 192)])
def test_retention_remembers_one_token(device, dtype, dims):
    """With decay 1 and faint other tokens, the state is one outer product written far back; with a fast decay, the neighbours across
    a chunk's edge are all there is."""
    import luminal_jl_b200 as L
    D, V = dims
    for decay, plant in (([1.0, 0.9995], True), ([0.3, 0.55], False)):
        cfg = config([retention(heads=2, dim=D, vdim=V, dims=D // 4 * 2, decay=decay, ff=0)], width=128, vocab=64, cap=None)
        w = G.random_weights(cfg, 9)
        if plant:
            k = 0.05 * w["l0.mix.k"]
            k[:, 1] = w["l0.mix.k"][:, 1] * 6.0          # only feature 1 writes strongly, and only token 1 has it
            w["l0.mix.k"] = G.to_bf16(k)
            w["embed"][:, 1] = 0.0
            w["embed"][1, :] = G.to_bf16(0.1 * w["embed"][1])
            w["embed"][1, 1] = 9.0
            w["l0.mix.q"][:, 2] = k[:, 1]
        else:
            w["l0.mix.q"][:, 2] *= 2.0
            w["l0.mix.k"] = G.to_bf16(w["l0.mix.q"] + 0.3 * w["l0.mix.k"])
        w["embed"][:, 2] = 2.0 if plant else 8.0             # every query has a share along every key: no output is a near-cancellation
        m = L.models.build_model(device, cfg, dtype)
        m.set_weights(w)
        s = L.Session(m, 1, 512)
        for key in (0, 1, 62, 63, 64, 65, 127, 128):
            n = 300
            toks = [2 + t % 60 for t in ids(key, n, 60)]
            toks[key] = 1
            ref = G.forward(cfg, w, toks)
            for cuts in ([n], [64, 64, 172], [63, 2, 235], [129, 1, 1, 169], [5, 2, 2, 291]):
                s.reset()
                at = 0
                for c in cuts:
                    got = s.extend([toks[at:at + c]], [list(range(c))])
                    assert agree(got, ref[at:at + c], dtype), (decay, key, cuts, at)
                    at += c
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
        want = np.concatenate([r[a:a + n] for r, a, n in zip(ref, at, plan)])
        assert agree(got, want, dtype), plan
        at = [a + n for a, n in zip(at, plan)]
    assert list(s.positions()) == at
    s.close()


@gpu
@BOTH
def test_slots_used_again(ctx, dtype):
    import luminal_jl_b200 as L
    name, V = "borrow", 200
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
def test_wide_batch(ctx):
    """more sequences than one weight pass serves"""
    name, V, B = "odd", 131, 40
    toks = [ids(300 + b, 3 + b % 7, V) for b in range(B)]
    s = ctx.session(name, "f32", batch=B, ctx=64)
    got = s.extend(toks, [[len(t) - 1] for t in toks])
    assert rel(got, np.concatenate([ctx.ref(name, t)[-1:] for t in toks])) < F32_TOL
    nxt = [int(t) for t in got.argmax(-1)]
    got = s.extend([[t] for t in nxt], [[0]] * B)
    assert rel(got, np.concatenate([ctx.ref(name, t + [x])[-1:] for t, x in zip(toks, nxt)])) < F32_TOL
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
    assert rel(got, np.stack([ctx.ref("odd", [7, 8])[-1], ctx.ref("odd", [4, 5, 9])[-1]])) < F32_TOL
    with pytest.raises(L.LuminalB200Error, match="max_ctx"):
        s.extend([[1] * 63, []])
    s.close()


# ---------------------------------------------------------------------------------------------------------------------------
# generation through the framework's own entry points
# ---------------------------------------------------------------------------------------------------------------------------
def oracle_greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(np.argmax(G.forward(cfg, w, toks)[-1])))
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
    s.reset()                                                          # stop at a token
    s.prefill(np.array(prompts))
    eot = int(want[0, 5])
    out = s.decode_until(None, 30, eot)
    for b in range(3):
        row = list(want[b, 1:])
        cut = row.index(eot) + 1 if eot in row else len(row)
        assert list(out[:min(cut, len(out)), b]) == row[:min(cut, len(out))]
    s.close()


@gpu
@BOTH
def test_pool_generation(ctx, dtype):
    """continuous batching: five requests over two slots give what each gives alone"""
    import luminal_jl_b200 as L
    name, V = "borrow", 200
    prompts = {i: ids(40 + i, n, V) for i, n in enumerate((20, 3, 50, 1, 9))}
    pool = L.RequestPool(ctx.session(name, dtype, batch=2, ctx=128))
    got = pool.generate(prompts, 8)
    for i, p in prompts.items():
        if dtype == "f32":
            assert got[i] == oracle_greedy(CONFIGS[name], ctx.w(name), p, 8)
        else:                                            # bf16: every chosen token is within rounding of the best
            ref = ctx.ref(name, p + got[i])
            for j, t in enumerate(got[i]):
                row = ref[len(p) - 1 + j]
                assert row.max() - row[t] < 4 * BF16_TOL * row.std()
    pool.session.close()


@gpu
def test_model_folder_and_replay(device, tmp_path):
    """a folder with config.json and bf16 safetensors through load_model and through bin/trace_run"""
    import os
    import subprocess
    import luminal_jl_b200 as L
    cfg = CONFIGS["odd"]
    w = G.random_weights(cfg, 21)
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    L.weights.write_safetensors(str(folder / "model.safetensors"), w, dtype="BF16")
    toks = ids(1, 30, 131)
    ref = G.forward(cfg, w, toks)
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
        assert [x for x in r.stdout.split("\n") if x] == [f"done {i}" for i in range(4)]
        assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32"]
        for n, rows in ((0, [0, 19]), (2, [29]), (3, [2])):
            got = np.fromfile(out / f"{n}.f32", "<f4").reshape(len(rows), -1)
            assert rel(got, ref[rows]) < t
    with open(folder / "config.json", "w") as f:
        json.dump(dict(cfg, width=64), f)
    with pytest.raises(L.LuminalB200Error, match="shape"):
        L.load_model(device, str(folder), "f32")


@gpu
def test_bad_configurations_are_refused(device):
    import luminal_jl_b200 as L
    for layers, what in (([latent(kv_from=0)], "kv_from"), ([latent(), latent(kv_from=0, kv_rank=48)], "latent cache"),
                         ([retention(), latent(kv_from=0)], "latent cache"), ([retention(heads=2, decay=[0.5, 1.5])], "decay"),
                         ([retention(dim=8, dims=12)], "rotated")):
        with pytest.raises(L.LuminalB200Error, match=what):
            L.models.build_model(device, config(layers), "f32")
