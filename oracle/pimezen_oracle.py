"""CPU restatement of the Pimezen decoder, one function per mechanism, in float64 numpy.

Test infrastructure only: plain loops over positions and heads, no cache, no chunking, nothing
shared with the product code.  ``weights`` maps tensor names to arrays (``l0.mix.left.q`` ...),
``config`` is the parsed config.json.

Notation: i, j positions (from 0); h, g query heads; x the residual stream [T, width].
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms(x, eps):
    """x divided by its root mean square over the last axis (eps inside the root)."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    """Model norm: the stored weight is an offset from one."""
    return rms(x, eps) * (1.0 + w)


def head_norm(x, w, heads, eps):
    """[T, heads * dim] -> [T, heads, dim], normed per head with one plain weight [dim]."""
    return rms(x.reshape(x.shape[0], heads, -1), eps) * w


def window_visible(i, j, size, keep_first):
    return j <= i and (i - j < size or j < keep_first)


def distance_bias(i, j, r1, r2):
    """Amount taken off a score at distance i - j."""
    return r1 * np.log(1.0 + r2 * (i - j))


def softmax_weights(q, k, scale, r1, r2, size, keep_first):
    """q [T, H, dim], k [T, G, dim] -> weights [H, T, T] (zero where a key is not seen)."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    w = np.zeros((H, T, T))
    for i in range(T):
        seen = np.array([j for j in range(i + 1) if window_visible(i, j, size, keep_first)])
        for h in range(H):
            s = k[seen, h // rep] @ q[i, h] * scale - distance_bias(i, seen, r1[h], r2[h])
            e = np.exp(s - s.max())
            w[h, i, seen] = e / e.sum()
    return w


def mix_heads(w, talk):
    """out_h = sum_g talk[h, g] w_g on [H, T, T]."""
    return np.einsum("hg,gij->hij", talk, w)


def window_attention(h, W, c, eps):
    """Left mixer on [T, width]; W maps 'q', 'k', ... to arrays, c is its part of the config."""
    T, H, G = h.shape[0], c["heads"], c["kv_heads"]
    q = head_norm(h @ W["q"].T, W["q.norm"], H, eps)
    k = head_norm(h @ W["k"].T, W["k.norm"], G, eps)
    v = (h @ W["v"].T).reshape(T, G, c["vdim"])
    w = softmax_weights(q, k, c["scale"], W["r1"], W["r2"], c["mask"]["size"], c["mask"]["keep_first"])
    w = mix_heads(w, W["talk"])
    out = np.stack([w[hh] @ v[:, hh // (H // G)] for hh in range(H)], axis=1)
    return out.reshape(T, -1) @ W["o"].T


def decay(h, W, tau):
    """Per-channel decays in (0, 1), [T, heads * dim]."""
    z = (h @ W["a1"].T) @ W["a2"].T + W["a2.b"]
    return np.exp(-np.log1p(np.exp(-z)) / tau)


def linear_recurrence(q, k, v, alpha, state=None):
    """q, k, alpha [T, H, dk], v [T, H, dv]: S <- diag(alpha) S + k v^T, o = S^T q.
    Returns (o [T, H, dv], final state [H, dk, dv])."""
    T, H, dk = q.shape
    S = np.zeros((H, dk, v.shape[-1])) if state is None else state.copy()
    o = np.zeros((T, H, v.shape[-1]))
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hcd,hc->hd", S, q[t])
    return o, S


def gated_linear_attention(h, W, c, eps):
    """Right mixer on [T, width]."""
    T, H, dk, dv = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q = (h @ W["q"].T).reshape(T, H, dk) * dk ** -0.5
    k = (h @ W["k"].T).reshape(T, H, dk)
    v = (h @ W["v"].T).reshape(T, H, dv)
    o, _ = linear_recurrence(q, k, v, decay(h, W, c["tau"]).reshape(T, H, dk))
    o = (rms(o, eps) * W["norm"]).reshape(T, H * dv)
    gate = h @ W["g"].T
    return (o * gate * sigmoid(gate)) @ W["o"].T


def clamped_glu(h, gate, up, down, limit):
    g = np.minimum(h @ gate.T, limit)
    u = np.clip(h @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def _sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def parallel_mixer(h, W, c, eps):
    left = window_attention(h, _sub(W, "left."), c["left"], eps)
    right = gated_linear_attention(h, _sub(W, "right."), c["right"], eps)
    return c["left_scale"] * left + c["right_scale"] * right


def layer(x, W, c, eps):
    x = x + W["ls1"] * parallel_mixer(norm(x, W["norm1"], eps), _sub(W, "mix."), c["mixer"], eps)
    if c.get("mlp") is not None:
        y = clamped_glu(norm(x, W["norm2"], eps), W["mlp.gate"], W["mlp.up"], W["mlp.down"],
                        c["mlp"]["limit"])
        x = x + W["ls2"] * y
    return x


def forward(weights, config, tokens, want_layers=False):
    """tokens [T] -> logits [T, vocab] (and the residual stream after every layer)."""
    weights = {k: np.asarray(v, dtype=np.float64) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = weights["embed"][np.asarray(tokens)]
    streams = []
    for n, c in enumerate(config["layers"]):
        x = layer(x, _sub(weights, f"l{n}."), c, eps)
        streams.append(x)
    logits = norm(x, weights["final.norm"], eps) @ weights["embed"].T
    return (logits, streams) if want_layers else logits


def random_weights(config, rank, seed=0, gain=1.0):
    """Random weights (float64) of the shapes that `config` implies; `rank` = inner width of the
    decay projection.  Scaled so that every mechanism matters at the output."""
    rng = np.random.default_rng(seed)
    D, V = config["width"], config["vocab"]

    def lin(o, i, s=1.0):
        return rng.standard_normal((o, i)) * s * gain / np.sqrt(i)

    w = {"embed": rng.standard_normal((V, D)) * 0.5, "final.norm": rng.standard_normal(D) * 0.1}
    for n, c in enumerate(config["layers"]):
        p = f"l{n}."
        L, R = c["mixer"]["left"], c["mixer"]["right"]
        H, G = L["heads"], L["kv_heads"]
        w[p + "norm1"] = rng.standard_normal(D) * 0.1
        w[p + "ls1"] = 0.5 + 0.2 * rng.standard_normal(D)
        a = p + "mix.left."
        w[a + "q"], w[a + "k"] = lin(H * L["dim"], D), lin(G * L["dim"], D)
        w[a + "v"], w[a + "o"] = lin(G * L["vdim"], D), lin(D, H * L["vdim"], 1.5)
        w[a + "q.norm"] = 1.0 + 0.2 * rng.standard_normal(L["dim"])
        w[a + "k.norm"] = 1.0 + 0.2 * rng.standard_normal(L["dim"])
        w[a + "r1"], w[a + "r2"] = rng.uniform(0.1, 1.0, H), rng.uniform(0.05, 1.0, H)
        w[a + "talk"] = np.eye(H) + 0.3 * rng.standard_normal((H, H))
        b = p + "mix.right."
        Hr, dk, dv = R["heads"], R["dim"], R["vdim"]
        w[b + "q"], w[b + "k"] = lin(Hr * dk, D), lin(Hr * dk, D)
        w[b + "v"], w[b + "g"], w[b + "o"] = lin(Hr * dv, D), lin(Hr * dv, D), lin(D, Hr * dv, 1.5)
        w[b + "norm"] = 1.0 + 0.2 * rng.standard_normal(dv)
        w[b + "a1"], w[b + "a2"] = lin(rank, D), lin(Hr * dk, rank)
        w[b + "a2.b"] = rng.uniform(-1.0, 4.0, Hr * dk)
        if c.get("mlp") is not None:
            ff = c["mlp"]["ff"]
            w[p + "norm2"] = rng.standard_normal(D) * 0.1
            w[p + "ls2"] = 0.5 + 0.2 * rng.standard_normal(D)
            w[p + "mlp.gate"], w[p + "mlp.up"] = lin(ff, D), lin(ff, D)
            w[p + "mlp.down"] = lin(D, ff)
    return w
