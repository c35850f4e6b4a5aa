"""Plain NumPy restatement of the Kevatar decoder: windowed attention with bounded scores, a delta rule with one decay per key channel,
decayed linear attention, sublayers normed on their output, and a token input in every layer.

Slow on purpose and shares nothing with the library: one function per mechanism, whole sequences at once, float64 unless the caller's
arrays say otherwise.  The tests compare the CUDA sessions with it; nothing of the product path imports it.

Notation (one sequence, T positions, row t = position t, rms(x) = x / sqrt(mean(x^2) + eps)):
    x_0 = s embed[token]
    x <- x + rms(mixer(x)) w1;   x <- x + rms(ff(x)) w2;   x <- x + rms(P (gelu(G x) e)) w3     e = the layer's share of the token's row
    attention, head a of H over key head a // (H / G):
        q, k <- rms over the head of the rotated projections
        s_ij = cap tanh(scale q_i . k_j / cap),  0 <= i - j < window;   o_i = sum_j softmax_j(s_ij) v_j
    channel delta, head a:
        q, k, v <- silu(conv(projection));   q <- q / |q| / sqrt(dim),  k <- k / |k|
        g = exp(-exp(A) softplus(Wa2 Wa1 x + b)) per key channel,   beta = sigmoid(Wb x)
        S <- diag(g) S;   S <- S + k (beta (v - S^T k))^T;   o = S^T q
        y = rms(o) w sigmoid(Wg2 Wg1 x)
    lightning, head a:   q, k, v <- silu(projection);   S <- decay S + k v^T;   o = S^T q;   y = rms(all heads' o) w sigmoid(Wg x)
    ff(x) = Wdown (silu(Wgate x) * (Wup x));   logits = embed (rms(x) w)
"""
from __future__ import annotations

import numpy as np


def rms(x, eps, w=None):
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if w is None else y * w


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (x + 0.044715 * x ** 3)))


def softplus(x):
    return np.logaddexp(x, 0.0)


def split_heads(x, heads):
    """[T, heads * d] -> [heads, T, d]"""
    T = x.shape[0]
    return x.reshape(T, heads, -1).transpose(1, 0, 2)


def merge_heads(x):
    return x.transpose(1, 0, 2).reshape(x.shape[1], -1)


def rotation(rot):
    """(frequencies [dims / 2], factor on cosine and sine)"""
    n, base, sc = rot["dims"], float(rot["base"]), rot.get("scaling")
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    if not sc:
        return f, 1.0

    def turns(t):                                     # the feature that turns t times over the original length
        return n * np.log(sc["original"] / (2.0 * np.pi * t)) / (2.0 * np.log(base))
    lo, hi = max(np.floor(turns(sc["fast"])), 0.0), min(np.ceil(turns(sc["slow"])), n - 1.0)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * np.log(sc["factor"]) + 1.0


def rotate(x, pos, rot):
    """Rotates the first rot['dims'] features of x [..., T, D], neighbouring pairs; pos [T]."""
    y = np.array(x, copy=True)
    if not rot:
        return y
    f, m = rotation(rot)
    for i in range(rot["dims"] // 2):
        c, s = (m * np.cos(pos * f[i])).astype(x.dtype), (m * np.sin(pos * f[i])).astype(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * c - v * s
        y[..., 2 * i + 1] = v * c + u * s
    return y


def cached_keys_values(h, w, p, mx, eps, pos):
    G = mx["kv_heads"]
    return rms(rotate(split_heads(h @ w[p + "k"].T, G), pos, mx.get("rot")), eps), split_heads(h @ w[p + "v"].T, G)


def attention(h, w, p, mx, eps, pos, kv):
    """kv = cached_keys_values(...) of this layer or of the layer it borrows from."""
    H, G = mx["heads"], mx["kv_heads"]
    q = rms(rotate(split_heads(h @ w[p + "q"].T, H), pos, mx.get("rot")), eps)
    k, v = (np.repeat(a, H // G, axis=0) for a in kv)
    s = (q @ k.transpose(0, 2, 1)) * mx["scale"]
    if mx.get("softcap"):
        s = mx["softcap"] * np.tanh(s / mx["softcap"])
    dist = pos[:, None] - pos[None]
    seen = dist >= 0
    if mx.get("mask"):
        seen &= dist < mx["mask"]["size"]
    s = np.where(seen, s, -np.inf)
    s = np.exp(s - s.max(-1, keepdims=True))
    return merge_heads((s / s.sum(-1, keepdims=True)) @ v) @ w[p + "o"].T


def short_conv(y, taps):
    """Causal convolution per channel, y [T, C], taps [C, n]: the last tap meets the current row."""
    out = np.zeros_like(y)
    n = taps.shape[1]
    for j in range(n):
        back = n - 1 - j
        out[back:] += y[:len(y) - back] * taps[:, j] if back < len(y) else 0.0
    return out


def channel_delta(h, w, p, mx, eps):
    H, G, dim = mx["heads"], mx["kv_heads"], mx["dim"]
    q, k, v = (silu(short_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv")
    q, k, v = split_heads(q, G), split_heads(k, G), split_heads(v, H)
    q = np.repeat(q / np.sqrt((q * q).sum(-1, keepdims=True) + 1e-6) * dim ** -0.5, H // G, axis=0)
    k = np.repeat(k / np.sqrt((k * k).sum(-1, keepdims=True) + 1e-6), H // G, axis=0)
    beta = sigmoid(h @ w[p + "b"].T).T                                                # [H, T]
    g = np.exp(-np.exp(w[p + "A_log"])[:, None, None] * split_heads(softplus((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]), H))
    S = np.zeros((H, dim, v.shape[-1]), dtype=h.dtype)
    o = np.empty_like(v)
    for t in range(h.shape[0]):
        S = g[:, t, :, None] * S
        u = beta[:, t, None] * (v[:, t] - np.einsum("hdv,hd->hv", S, k[:, t]))
        S = S + k[:, t, :, None] * u[:, None, :]
        o[:, t] = np.einsum("hdv,hd->hv", S, q[:, t])
    y = merge_heads(rms(o, eps, w[p + "norm"])) * sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T)
    return y @ w[p + "o"].T


def lightning(h, w, p, mx, eps):
    H = mx["heads"]
    q, k, v = (split_heads(silu(h @ w[p + n].T), H) for n in "qkv")
    g = np.asarray(mx["decay"], dtype=h.dtype)[:, None, None]
    S = np.zeros((H, q.shape[-1], v.shape[-1]), dtype=h.dtype)
    o = np.empty_like(v)
    for t in range(h.shape[0]):
        S = g * S + k[:, t, :, None] * v[:, t, None, :]
        o[:, t] = np.einsum("hdv,hd->hv", S, q[:, t])
    return (rms(merge_heads(o), eps, w[p + "norm"]) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def feed_forward(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def token_side(x, e, w, p, eps):
    """What a layer adds to the residual from its share e [T, dim] of the tokens' rows."""
    g = gelu_tanh(x @ w[p + "gate"].T) * e
    return rms(g @ w[p + "proj"].T, eps, w[p + "norm"])


def forward(cfg, w, tokens, dtype=np.float64, return_layers=False, rounded=lambda x: x):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer).  `rounded` is applied to what every sublayer and
    the head read: with a rounding it shows how far rounding alone moves the logits."""
    w = {k: np.asarray(v, dtype=dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    tokens = np.asarray(tokens)
    x = w["embed"][tokens] * cfg["embedding"]["scale"]
    pos = np.arange(len(tokens), dtype=np.float64)
    kvs, outs = {}, []
    for i, layer in enumerate(cfg["layers"]):
        mx, p = layer["mixer"], f"l{i}."
        if layer["type"] == "attention":
            src = mx.get("kv_from")
            if src is None:
                kvs[i] = cached_keys_values(rounded(x), w, p + "mix.", mx, eps, pos)
            y = attention(rounded(x), w, p + "mix.", mx, eps, pos, kvs[i if src is None else src])
        elif layer["type"] == "channel_delta":
            y = channel_delta(rounded(x), w, p + "mix.", mx, eps)
        else:
            y = lightning(rounded(x), w, p + "mix.", mx, eps)
        x = x + rms(y, eps, w[p + "norm1"])
        if layer.get("mlp"):
            x = x + rms(feed_forward(rounded(x), w, p + "mlp."), eps, w[p + "norm2"])
        if cfg.get("token_side"):
            n = cfg["token_side"]["dim"]
            x = x + token_side(rounded(x), w["side.embed"][tokens, i * n:(i + 1) * n], w, p + "side.", eps)
        outs.append(x)
    logits = rounded(rms(x, eps, w["final.norm"])) @ w["embed"].T
    return (logits, outs) if return_layers else logits


def tensor_shapes(cfg, decay_rank=None, gate_rank=None):
    """name -> shape of every tensor a model of this configuration has (the two low ranks are free: the file's shapes give them)."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W)}
    n = (cfg.get("token_side") or {}).get("dim", 0)
    if n:
        out["side.embed"] = (V, len(cfg["layers"]) * n)
    for i, layer in enumerate(cfg["layers"]):
        mx, p = layer["mixer"], f"l{i}.mix."
        H, G, dk, dv = mx["heads"], mx.get("kv_heads", mx["heads"]), mx["dim"], mx["vdim"]
        out[f"l{i}.norm1"] = (W,)
        if layer["type"] == "attention":
            out[p + "q"] = (H * dk, W)
            if mx.get("kv_from") is None:
                out[p + "k"], out[p + "v"] = (G * dk, W), (G * dv, W)
        elif layer["type"] == "channel_delta":
            ra, rg = decay_rank or mx.get("_ranks", (12, 20))[0], gate_rank or mx.get("_ranks", (12, 20))[1]
            for t, c in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                out[p + t], out[p + t + ".conv"] = (c, W), (c, mx["conv"])
            out[p + "b"], out[p + "A_log"], out[p + "norm"], out[p + "dt_bias"] = (H, W), (H,), (dv,), (H * dk,)
            out[p + "a1"], out[p + "a2"], out[p + "g1"], out[p + "g2"] = (ra, W), (H * dk, ra), (rg, W), (H * dv, rg)
        else:
            out[p + "q"] = out[p + "k"] = (H * dk, W)
            out[p + "v"] = out[p + "g"] = (H * dv, W)
            out[p + "norm"] = (H * dv,)
        out[p + "o"] = (W, H * dv)
        if layer.get("mlp"):
            out[f"l{i}.norm2"] = (W,)
            out[f"l{i}.mlp.gate"] = out[f"l{i}.mlp.up"] = (layer["mlp"]["ff"], W)
            out[f"l{i}.mlp.down"] = (W, layer["mlp"]["ff"])
        if n:
            out[f"l{i}.side.gate"], out[f"l{i}.side.proj"], out[f"l{i}.side.norm"] = (n, W), (W, n), (W,)
    out["final.norm"] = (W,)
    return out


def random_weights(cfg, seed, gain=1.0):
    """Random weights that keep activations near unit size (gains around 1), rounded to bf16 so both dtypes load the same values."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        a = rng.standard_normal(shape)
        if name.endswith("A_log"):
            a = 0.7 * a - 0.5
        elif name.endswith("dt_bias"):
            a = 1.5 * a - 2.0
        elif name.endswith(".conv"):
            a = a / np.sqrt(shape[1])
        elif len(shape) == 1:
            a = 1.0 + 0.2 * a
        elif name == "embed":
            a = a / cfg["embedding"]["scale"]
        elif name != "side.embed":
            a = a * (gain / np.sqrt(shape[1]))
        w[name] = to_bf16(a)
    return w


def to_bf16(a):
    """float32 array with every value rounded to the nearest bf16."""
    u = np.ascontiguousarray(np.asarray(a, dtype=np.float32)).view(np.uint32).astype(np.uint64)
    return ((((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16) & 0xFFFFFFFF).astype(np.uint32).view(np.float32)
