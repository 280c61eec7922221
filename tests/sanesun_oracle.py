"""Plain FP64 restatement of the Sanesun design for the tests: one function per mechanism, whole sequences only, no cache,
no batching. Shares nothing with the library; `weights` maps tensor names to arrays, configurations are the dictionaries
of config.json.

`mistake` names a deliberate error (tests check that their inputs would show it): "window-1", "window+1" (window off by
one), "no-first" (the kept first tokens unseen), "first-1" (one kept token too few), "no-sink", "no-talk", "no-turn-back"
(outputs not rotated back), "no-bias", "lost-state" (recurrent states and convolution taps zeroed at position `portion`),
"lost-taps" (only the taps), "late-read" (the read-out does not see the token's own write), "no-page" (keys at [portion,
portion + 4) unseen), "portion-positions" (positions counted from `portion`)."""
import math

import numpy as np


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def xielu(z, p, q):
    """Quadratic above zero, exponential below, slope 1/2 at zero on both sides."""
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(neg) - neg)) + 0.5 * z


def turned(x, positions, dims, base, sign=1.0):
    """Rotates the first `dims` entries of the last axis: entry i with entry i + dims / 2. x is [tokens, heads, size]."""
    half = dims // 2
    out = np.array(x, np.float64)
    for i in range(half):
        a = sign * positions * base ** (-2.0 * i / dims)
        c, s = np.cos(a)[:, None], np.sin(a)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def window(n, size, keep_first):
    """seen[i, j]: the last `size` positions up to i, and the first `keep_first` ones."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax_with_sink(score, seen, sink):
    """Rows of weights; exp(sink) joins the denominator only (sink None: plain softmax)."""
    score = np.where(seen, score, -np.inf)
    top = score.max(axis=1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    weight = np.exp(score - top)
    return weight / (weight.sum(axis=1, keepdims=True) + (0.0 if sink is None else np.exp(sink - top)))


def attention(h, w, p, m, eps, mistake=None, portion=0):
    n, H, G = len(h), m["heads"], m["kv_heads"]
    bias = 0.0 if mistake == "no-bias" else 1.0
    q = (h @ w[p + "q"].T + bias * w[p + "q.b"]).reshape(n, H, m["dim"])
    k = (h @ w[p + "k"].T + bias * w[p + "k.b"]).reshape(n, G, m["dim"])
    v = (h @ w[p + "v"].T + bias * w[p + "v.b"]).reshape(n, G, m["vdim"])
    pos = np.arange(n, dtype=np.float64)
    if mistake == "portion-positions":
        pos = np.where(pos >= portion, pos - portion, pos)
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    q, k, v = turned(q, pos, dims, base), turned(k, pos, dims, base), turned(v, pos, m["vdim"], base)
    size, keep = m["mask"]["size"], m["mask"]["keep_first"]
    size += {"window-1": -1, "window+1": 1}.get(mistake, 0)
    keep = 0 if mistake == "no-first" else keep - 1 if mistake == "first-1" else keep
    seen = window(n, size, keep)
    if mistake == "no-page":
        j = np.arange(n)[None, :]
        seen &= ~((j >= portion) & (j < portion + 4) & (j != np.arange(n)[:, None]))
    score = np.stack([q[:, a] @ k[:, a // (H // G)].T * m["scale"] for a in range(H)])
    if mistake != "no-talk":
        score = np.einsum("ab,bij->aij", w[p + "talk"], score)
    out = np.zeros((n, H, m["vdim"]))
    for a in range(H):
        out[:, a] = softmax_with_sink(score[a], seen, None if mistake == "no-sink" else w[p + "sink"][a]) @ v[:, a // (H // G)]
    if mistake != "no-turn-back":
        out = turned(out, pos, m["vdim"], base, -1.0)
    return out.reshape(n, -1) @ w[p + "o"].T


def latent_attention(h, w, p, m, eps, mistake=None, portion=0):
    n, H = len(h), m["heads"]
    cq = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    c = rms(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]
    q = (cq @ w[p + "uq"].T).reshape(n, H, m["dim"])
    k = (c @ w[p + "uk"].T).reshape(n, H, m["dim"])
    v = (c @ w[p + "uv"].T).reshape(n, H, m["vdim"])
    seen = np.tril(np.ones((n, n), bool))
    if mistake == "no-page":
        j = np.arange(n)[None, :]
        seen &= ~((j >= portion) & (j < portion + 4) & (j != np.arange(n)[:, None]))
    gate = sigmoid(h @ w[p + "g"].T)
    out = np.zeros((n, H, m["vdim"]))
    for a in range(H):
        out[:, a] = softmax_with_sink(q[:, a] @ k[:, a].T * m["scale"], seen, None) @ v[:, a] * gate[:, a:a + 1]
    return out.reshape(n, -1) @ w[p + "o"].T


def short_conv(x, taps, cut=None):
    """Causal convolution over time per channel, the last tap on the current token; `cut`: nothing before it is known."""
    n, count = len(x), taps.shape[1]
    out = np.zeros_like(x)
    for t in range(n):
        for back in range(count):
            if t - back >= (cut if cut is not None and t >= cut else 0):
                out[t] += taps[:, count - 1 - back] * x[t - back]
    return out


def channel_delta(h, w, p, m, eps, mistake=None, portion=0):
    n, H, G, dk, dv = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    cut = portion if mistake in ("lost-state", "lost-taps") else None
    q, k, v = (silu(short_conv(h @ w[p + x].T, w[p + x + ".conv"], cut)) for x in "qkv")
    unit = lambda x: x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)
    q, k, v = unit(q.reshape(n, G, dk)) * dk ** -0.5, unit(k.reshape(n, G, dk)), v.reshape(n, H, dv)
    beta = sigmoid(h @ w[p + "b"].T)
    step = softplus(h @ w[p + "a1"].T @ w[p + "a2"].T + w[p + "dt_bias"]).reshape(n, H, dk)
    decay = np.exp(-np.exp(w[p + "A_log"])[:, None] * step)
    state, out = np.zeros((H, dk, dv)), np.zeros((n, H, dv))
    for t in range(n):
        if mistake == "lost-state" and t == portion:
            state[:] = 0
        for a in range(H):
            key, query = k[t, a // (H // G)], q[t, a // (H // G)]
            s = decay[t, a][:, None] * state[a]
            u = beta[t, a] * (v[t, a] - s.T @ key)
            out[t, a] = s.T @ query
            state[a] = s + np.outer(key, u)
            if mistake != "late-read":
                out[t, a] = state[a].T @ query
    gate = sigmoid(h @ w[p + "g1"].T @ w[p + "g2"].T).reshape(n, H, dv)
    return (rms(out, eps) * w[p + "norm"] * gate).reshape(n, -1) @ w[p + "o"].T


MIXERS = {"attention": attention, "channel_delta": channel_delta, "latent_attention": latent_attention}


def feed_forward(h, w, p):
    return xielu(h @ w[p + "up"].T, *w[p + "act"]) @ w[p + "down"].T


def forward(cfg, weights, ids, trace=None, **kw):
    """Logits [len(ids), vocab]; `trace` collects the residual stream after every layer."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps, x = cfg["norm"]["eps"], w["embed"][np.asarray(ids)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms(x, eps) * w[p + "norm1"]
        add = MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps, **kw)
        if layer.get("mlp"):
            add = add + feed_forward(h, w, p + "mlp.")
        x = x + add
        if trace is not None:
            trace.append(x)
    return rms(x, eps) * w["final.norm"] @ w["head"].T


# ------------------------------------------------------------------ small random models
def att(heads, kv_heads, dim, vdim, size, keep, dims=None, base=1000.0, scale=None, ff=0):
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size, "keep_first": keep},
                      "rot": {"dims": dim // 4 * 2 if dims is None else dims, "base": base},
                      "scale": dim ** -0.5 if scale is None else scale}}


def delta(heads, kv_heads, dim, vdim, conv, ff=0):
    return {"type": "channel_delta", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def latent(heads, dim, vdim, kv_rank, q_rank, scale=None, ff=0):
    return {"type": "latent_attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "scale": dim ** -0.5 if scale is None else scale}}


def config(vocab, width, layers, eps=1e-5, embed_scale=3.0):
    return {"architecture": "Sanesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "layers": layers}


def shapes(cfg, rank=5):
    """Tensor names and shapes of a configuration; `rank`: inner size of the decay projection, the gate's is one more."""
    W = cfg["width"]
    out = {"embed": (cfg["vocab"], W), "head": (cfg["vocab"], W), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        out[f"l{i}.norm1"] = (W,)
        H = m["heads"]
        if layer["type"] == "attention":
            for n, r in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                out[p + n], out[p + n + ".b"] = (r, W), (r,)
            out.update({p + "talk": (H, H), p + "sink": (H,), p + "o": (W, H * m["vdim"])})
        elif layer["type"] == "latent_attention":
            out.update({p + "dq": (m["q_rank"], W), p + "dq.norm": (m["q_rank"],), p + "uq": (H * m["dim"], m["q_rank"]),
                        p + "dkv": (m["kv_rank"], W), p + "dkv.norm": (m["kv_rank"],), p + "uk": (H * m["dim"], m["kv_rank"]),
                        p + "uv": (H * m["vdim"], m["kv_rank"]), p + "g": (H, W), p + "o": (W, H * m["vdim"])})
        else:
            K, V = m["kv_heads"] * m["dim"], H * m["vdim"]
            for n, r in (("q", K), ("k", K), ("v", V)):
                out[p + n], out[p + n + ".conv"] = (r, W), (r, m["conv"])
            out.update({p + "b": (H, W), p + "A_log": (H,), p + "norm": (m["vdim"],), p + "a1": (rank, W),
                        p + "a2": (H * m["dim"], rank), p + "dt_bias": (H * m["dim"],), p + "g1": (rank + 1, W),
                        p + "g2": (V, rank + 1), p + "o": (W, V)})
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            out.update({f"l{i}.mlp.up": (ff, W), f"l{i}.mlp.down": (W, ff), f"l{i}.mlp.act": (2,)})
    return out


def random_weights(cfg, seed, rank=5):
    """Random weights on the BF16 grid (so that BF16 storage is exact): inputs of products of unit size, norms around 1,
    head mixing around the unit matrix, slow decays so that old tokens still matter."""
    from puppygrad_b200.synthetic import round_bf16
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg, rank).items():
        leaf = name.split(".")[-1]
        a = rng.standard_normal(shape)
        if name == "embed":
            a = a / cfg["embedding"]["scale"]
        elif leaf == "talk":
            a = np.eye(shape[0]) + 0.4 * a / math.sqrt(shape[0])
        elif leaf == "conv":
            a = a / math.sqrt(shape[1])
        elif leaf in ("a2", "g2"):
            a = a * 2 / math.sqrt(shape[1])
        elif len(shape) == 2:
            a = a / math.sqrt(shape[1])
        elif leaf == "b":
            a = 0.4 * a
        elif leaf == "sink":
            a = a + 1.0
        elif leaf == "A_log":
            a = 0.5 * a - 1.0
        elif leaf == "dt_bias":
            a = a - 3.0
        elif leaf == "act":
            a = 0.5 * a
        else:
            a = 1.0 + 0.2 * a
        out[name] = round_bf16(a.astype(np.float32))
    return out
