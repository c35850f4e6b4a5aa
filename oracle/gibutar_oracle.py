"""Plain NumPy restatement of the Gibutar decoder: latent attention and retention layers with a parallel feed-forward.

Slow on purpose and shares nothing with the library: one function per mechanism, whole sequences at once, float64 unless the
caller's arrays say otherwise.  The tests compare the CUDA sessions with it; nothing of the product path imports it.

Notation (one sequence, T positions, row t = position t):
    h = rms(x) w                                 one norm per layer, read by both sublayers
    x <- x + mixer(h) + ff(h)
    latent attention, head a:
        c_q = rms(Wdq h) w_q,  [q_a | r_a] = (Wuq c_q)_a,   [c' | k'] = Wdkv h,  c = rms(c') w_c
        s_ij = scale (q_ai . (Wuk c_j)_a + R_i r_ai . R_j k'_j),   j <= i
        o_ai = sigmoid(Wg h_i)_a sum_j softmax_j(s_ij) (Wuv c_j)_a
    retention, head a with decay g_a:
        S_t = g_a S_{t-1} + (R_t k_t / sqrt(dim)) v_t^T,   o_t = S_t^T R_t q_t
        y_t = rms(o_t) silu(Wg h_t)
    ff(h) = Wdown relu(Wup h)^2
    logits = cap tanh(head rms(x) w / cap)
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


def rotate(x, pos, base, dims, interleaved):
    """Rotates the first `dims` features of x [..., T, D]; pos [T]."""
    y = np.array(x, copy=True)
    for i in range(dims // 2):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        ang = pos * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(ang).astype(x.dtype), np.sin(ang).astype(x.dtype)
        u, v = x[..., a], x[..., b]
        y[..., a] = u * c - v * s
        y[..., b] = v * c + u * s
    return y


def split_heads(x, heads):
    """[T, heads * d] -> [heads, T, d]"""
    T = x.shape[0]
    return x.reshape(T, heads, -1).transpose(1, 0, 2)


def merge_heads(x):
    return x.transpose(1, 0, 2).reshape(x.shape[1], -1)


def latent_of(h, w, p, mx, eps, pos):
    """What a latent-attention layer caches: (latent c [T, kv_rank], rotated shared key part [T, rot_dim])."""
    y = h @ w[p + "dkv"].T
    c = rms(y[:, :mx["kv_rank"]], eps, w[p + "dkv.norm"])
    return c, rotate(y[:, mx["kv_rank"]:], pos, mx["rot"]["base"], mx["rot"]["dims"], True)


def latent_attention(h, w, p, mx, eps, pos, latent):
    """latent = latent_of(...) of this layer or of the layer it borrows from."""
    H, dim = mx["heads"], mx["dim"]
    cq = rms(h @ w[p + "dq"].T, eps, w[p + "dq.norm"])
    q = split_heads(cq @ w[p + "uq"].T, H)                       # [H, T, dim + rot_dim]
    qn, qr = q[..., :dim], rotate(q[..., dim:], pos, mx["rot"]["base"], mx["rot"]["dims"], True)
    c, kr = latent
    k = split_heads(c @ w[p + "uk"].T, H)
    v = split_heads(c @ w[p + "uv"].T, H)
    s = (qn @ k.transpose(0, 2, 1) + qr @ kr.T) * mx["scale"]
    T = h.shape[0]
    s = np.where(np.tril(np.ones((T, T), bool)), s, -np.inf)
    s = np.exp(s - s.max(-1, keepdims=True))
    o = (s / s.sum(-1, keepdims=True)) @ v                       # [H, T, vdim]
    o = o * sigmoid(h @ w[p + "g"].T).T[:, :, None]
    return merge_heads(o) @ w[p + "o"].T


def retention(h, w, p, mx, eps, pos):
    H, dim = mx["heads"], mx["dim"]
    rot = mx.get("rot") or {"base": 1.0, "dims": 0}
    q = rotate(split_heads(h @ w[p + "q"].T, H), pos, rot["base"], rot["dims"], False)
    k = rotate(split_heads(h @ w[p + "k"].T, H), pos, rot["base"], rot["dims"], False) * dim ** -0.5
    v = split_heads(h @ w[p + "v"].T, H)
    g = np.asarray(mx["decay"], dtype=h.dtype)[:, None, None]
    S = np.zeros((H, dim, v.shape[-1]), dtype=h.dtype)
    o = np.empty_like(v)
    for t in range(h.shape[0]):
        S = g * S + k[:, t, :, None] * v[:, t, None, :]
        o[:, t] = np.einsum("hdv,hd->hv", S, q[:, t])
    return (merge_heads(rms(o, eps)) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


def feed_forward(h, w, p):
    return np.maximum(h @ w[p + "up"].T, 0.0) ** 2 @ w[p + "down"].T


def forward(cfg, w, tokens, dtype=np.float64, return_layers=False):
    """Logits [T, vocab] of one sequence (and the residual stream after every layer)."""
    w = {k: np.asarray(v, dtype=dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    pos = np.arange(len(tokens), dtype=np.float64)
    latents, outs = {}, []
    for i, layer in enumerate(cfg["layers"]):
        mx, p = layer["mixer"], f"l{i}.mix."
        h = rms(x, eps, w[f"l{i}.norm1"])
        if layer["type"] == "latent_attention":
            src = mx.get("kv_from")
            if src is None:
                latents[i] = latent_of(h, w, p, mx, eps, pos)
            y = latent_attention(h, w, p, mx, eps, pos, latents[i if src is None else src])
        else:
            y = retention(h, w, p, mx, eps, pos)
        if layer.get("mlp"):
            y = y + feed_forward(h, w, f"l{i}.mlp.")
        x = x + y
        outs.append(x)
    logits = rms(x, eps, w["final.norm"]) @ w["head"].T
    cap = cfg.get("logit_softcap")
    if cap:
        logits = cap * np.tanh(logits / cap)
    return (logits, outs) if return_layers else logits


def tensor_shapes(cfg):
    """name -> shape of every tensor a model of this configuration has."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W)}
    for i, layer in enumerate(cfg["layers"]):
        mx, p = layer["mixer"], f"l{i}.mix."
        H = mx["heads"]
        out[f"l{i}.norm1"] = (W,)
        if layer["type"] == "latent_attention":
            out[p + "dq"] = (mx["q_rank"], W)
            out[p + "dq.norm"] = (mx["q_rank"],)
            out[p + "uq"] = (H * (mx["dim"] + mx["rot_dim"]), mx["q_rank"])
            if mx.get("kv_from") is None:
                out[p + "dkv"] = (mx["kv_rank"] + mx["rot_dim"], W)
                out[p + "dkv.norm"] = (mx["kv_rank"],)
            out[p + "uk"] = (H * mx["dim"], mx["kv_rank"])
            out[p + "uv"] = (H * mx["vdim"], mx["kv_rank"])
            out[p + "g"] = (H, W)
        else:
            out[p + "q"] = out[p + "k"] = (H * mx["dim"], W)
            out[p + "v"] = out[p + "g"] = (H * mx["vdim"], W)
        out[p + "o"] = (W, H * mx["vdim"])
        if layer.get("mlp"):
            out[f"l{i}.mlp.up"] = (layer["mlp"]["ff"], W)
            out[f"l{i}.mlp.down"] = (W, layer["mlp"]["ff"])
    out["final.norm"] = (W,)
    out["head"] = (V, W)
    return out


def random_weights(cfg, seed, gain=1.0):
    """Unit-variance-preserving random weights (gains around 1), rounded to bf16 so both dtypes load the same values."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        a = rng.standard_normal(shape)
        if len(shape) == 1:
            a = 1.0 + 0.2 * a
        elif name != "embed":
            a = a * (gain / np.sqrt(shape[1]))
        w[name] = to_bf16(a)
    return w


def to_bf16(a):
    """float32 array with every value rounded to the nearest bf16."""
    u = np.ascontiguousarray(np.asarray(a, dtype=np.float32)).view(np.uint32).astype(np.uint64)
    return ((((u + 0x7FFF + ((u >> 16) & 1)) >> 16) << 16) & 0xFFFFFFFF).astype(np.uint32).view(np.float32)
