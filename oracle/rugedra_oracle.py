"""CPU restatement of the Rugedra decoder, one function per mechanism, in float64 numpy.

Test infrastructure only: plain loops over positions, no cache, no chunking, nothing shared with the
product code.  ``weights`` maps tensor names to arrays (``l0.mix.q`` ...), ``config`` is the parsed
config.json.

Notation: i, j positions (from 0); n a head; x the residual stream [T, width].
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    """x divided by its root mean square over the last axis (eps inside the root)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, w, eps):
    """Centred, scaled to unit variance, times w; no bias."""
    d = x - x.mean(axis=-1, keepdims=True)
    return rms(d, eps) * w


def embed(tokens, table, positions):
    return table[tokens] + positions[: len(tokens)]


# ------------------------------------------------------------------------------ latent attention
def rotate(x, position, dims, base):
    """The first `dims` elements of x [..., n] as interleaved pairs turned by position * base^(-2i/dims)."""
    out = x.copy()
    for i in range(dims // 2):
        a = position * base ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * np.cos(a) - v * np.sin(a)
        out[..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def causal_softmax(scores):
    """[T, T] -> weights over j <= i."""
    T = scores.shape[0]
    w = np.zeros_like(scores)
    for i in range(T):
        e = np.exp(scores[i, : i + 1] - scores[i, : i + 1].max())
        w[i, : i + 1] = e / e.sum()
    return w


def latent_split(h, W, c, eps):
    """(latent after its norm [T, rank], rotated shared key [T, rot_dim])"""
    both = h @ W["dkv"].T
    lat = rms(both[:, : c["kv_rank"]], eps) * W["dkv.norm"]
    key = np.stack([rotate(both[p, c["kv_rank"]:], p, c["rot"]["dims"], c["rot"]["base"]) for p in range(len(h))])
    return lat, key


def latent_heads(q, lat, key, uk, uv, c):
    """Heads' results [T, heads, vdim]; q [T, heads, dim + rot_dim] before the rotation."""
    T, H, d = len(q), c["heads"], c["dim"]
    uk, uv = uk.reshape(H, d, -1), uv.reshape(H, c["vdim"], -1)
    qr = np.stack([rotate(q[p, :, d:], p, c["rot"]["dims"], c["rot"]["base"]) for p in range(T)])
    out = np.zeros((T, H, c["vdim"]))
    for n in range(H):
        s = (q[:, n, :d] @ (lat @ uk[n].T).T + qr[:, n] @ key.T) * c["scale"]
        out[:, n] = causal_softmax(s) @ (lat @ uv[n].T)
    return out


def latent_attention(h, W, c, eps):
    T, H = h.shape[0], c["heads"]
    lat, key = latent_split(h, W, c, eps)
    q = (h @ W["q"].T).reshape(T, H, c["dim"] + c["rot_dim"])
    out = latent_heads(q, lat, key, W["uk"], W["uv"], c)
    out = out * sigmoid(h @ W["g"].T)[:, :, None]
    return out.reshape(T, -1) @ W["o"].T


# ------------------------------------------------------------------------------ channel delta rule
def short_conv(x, taps):
    """[T, C] with taps [C, K]: y_t = sum_j taps[:, K - 1 - j] x_{t - j}, zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    y = np.zeros_like(x)
    for t in range(T):
        for j in range(min(K, t + 1)):
            y[t] += taps[:, K - 1 - j] * x[t - j]
    return y


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def channel_decay(h, W, heads):
    """[T, heads, dim] in (0, 1)"""
    z = (h @ W["a1"].T) @ W["a2"].T + W["dt_bias"]
    z = softplus(z).reshape(len(h), heads, -1)
    return np.exp(-np.exp(W["A_log"])[None, :, None] * z)


def delta_recurrence(q, k, v, g, beta, state=None):
    """q, k, g [T, H, dk], v [T, H, dv], beta [T, H] -> (o [T, H, dv], final state [H, dk, dv])."""
    T, H, dk = q.shape
    S = np.zeros((H, dk, v.shape[-1])) if state is None else state.copy()
    o = np.zeros((T, H, v.shape[-1]))
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hcd,hc->hd", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hcd,hc->hd", S, q[t])
    return o, S


def channel_delta(h, W, c, eps):
    T, H, G, dk, dv = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (silu(short_conv(h @ W[n].T, W[n + ".conv"])) for n in "qkv")
    q, k = unit(q.reshape(T, G, dk)) * dk ** -0.5, unit(k.reshape(T, G, dk))
    q, k = np.repeat(q, H // G, axis=1), np.repeat(k, H // G, axis=1)
    o, _ = delta_recurrence(q, k, v.reshape(T, H, dv), channel_decay(h, W, H), sigmoid(h @ W["b"].T))
    gate = sigmoid((h @ W["g1"].T) @ W["g2"].T)
    o = (rms(o, eps) * W["norm"]).reshape(T, H * dv) * gate
    return o @ W["o"].T


MIXERS = {"latent_attention": latent_attention, "channel_delta": channel_delta}


# ------------------------------------------------------------------------------ feed-forward
def squared_relu(h, up, down):
    return np.maximum(h @ up.T, 0.0) ** 2 @ down.T


def clamped_glu(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def choose_experts(logits, top, groups, keep):
    """One token's logits [E] -> (experts [top], weights [top])."""
    e = np.exp(logits - logits.max())
    s = e / e.sum()
    size = len(s) // groups
    best = np.argsort(-s.reshape(groups, size).max(axis=1), kind="stable")[:keep]
    allowed = np.isin(np.arange(len(s)) // size, best)
    chosen = np.argsort(-np.where(allowed, s, -1.0), kind="stable")[:top]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20)


def mixture(h, W, c):
    r, limit = c["router"], c["expert"]["limit"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    logits = h @ W["router"].T
    out = np.zeros_like(h)
    for t in range(len(h)):
        for n, w in zip(*choose_experts(logits[t], r["top"], groups["count"], groups["keep"])):
            e = f"e{n}."
            out[t] += w * clamped_glu(h[t: t + 1], W[e + "gate"], W[e + "up"], W[e + "down"], limit)[0]
    return out


def feed_forward(h, W, c):
    return squared_relu(h, W["up"], W["down"]) if c["kind"] == "dense" else mixture(h, W, c)


# ------------------------------------------------------------------------------ model
def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def layer(x, W, c, eps, mult):
    x = x + mult * MIXERS[c["type"]](layer_norm(x, W["norm1"], eps), _sub(W, "mix."), c["mixer"], eps)
    if c.get("mlp") is not None:
        x = x + mult * feed_forward(layer_norm(x, W["norm2"], eps), _sub(W, "mlp."), c["mlp"])
    return x


def forward(weights, config, tokens, want_layers=False):
    """tokens [T] -> logits [T, vocab] (and the residual stream after every layer)."""
    weights = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = embed(np.asarray(tokens), weights["embed"], weights["pos"])
    streams = []
    for n, c in enumerate(config["layers"]):
        x = layer(x, _sub(weights, f"l{n}."), c, eps, config["residual_mult"])
        streams.append(x)
    logits = layer_norm(x, weights["final.norm"], eps) @ weights["head"].T * config["logit_scale"]
    return (logits, np.stack(streams)) if want_layers else logits


def random_weights(config, rank, seed=0):
    """Weights of the right shapes; `rank`: inner width of the two-step projections."""
    rng = np.random.default_rng(seed)
    wd, out = config["width"], {}

    def lin(name, rows, cols, gain=1.0):
        out[name] = rng.standard_normal((rows, cols)) * gain / cols ** 0.5

    def near_one(name, n):
        out[name] = 1.0 + 0.2 * rng.standard_normal(n)

    out["embed"] = rng.standard_normal((config["vocab"], wd))
    out["pos"] = 0.3 * rng.standard_normal((config["max_positions"], wd))
    for i, c in enumerate(config["layers"]):
        m, p = c["mixer"], f"l{i}.mix."
        near_one(f"l{i}.norm1", wd)
        if c["type"] == "latent_attention":
            H, R = m["heads"], m["kv_rank"]
            lin(p + "q", H * (m["dim"] + m["rot_dim"]), wd, 1.5)
            lin(p + "dkv", R + m["rot_dim"], wd, 1.5)
            near_one(p + "dkv.norm", R)
            lin(p + "uk", H * m["dim"], R, 1.5)
            lin(p + "uv", H * m["vdim"], R)
            lin(p + "g", H, wd)
            lin(p + "o", wd, H * m["vdim"])
        else:
            H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, ch in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                lin(p + n, ch, wd)
                out[p + n + ".conv"] = rng.standard_normal((ch, m["conv"])) * 0.6
            lin(p + "b", H, wd)
            out[p + "A_log"] = rng.uniform(-2.0, 1.0, H)
            near_one(p + "norm", dv)
            lin(p + "a1", rank, wd)
            lin(p + "a2", H * dk, rank)
            out[p + "dt_bias"] = rng.uniform(-5.0, 1.0, H * dk)
            lin(p + "g1", rank, wd)
            lin(p + "g2", H * dv, rank)
            lin(p + "o", wd, H * dv)
        mlp, p = c.get("mlp"), f"l{i}.mlp."
        if mlp is None:
            continue
        near_one(f"l{i}.norm2", wd)
        if mlp["kind"] == "dense":
            lin(p + "up", mlp["ff"], wd)
            lin(p + "down", wd, mlp["ff"])
        else:
            for n in range(mlp["router"]["experts"]):
                lin(f"{p}e{n}.gate", mlp["expert"]["ff"], wd)
                lin(f"{p}e{n}.up", mlp["expert"]["ff"], wd)
                lin(f"{p}e{n}.down", wd, mlp["expert"]["ff"])
            lin(p + "router", mlp["router"]["experts"], wd, 2.0)
    near_one("final.norm", wd)
    lin("head", config["vocab"], wd)
    return out
