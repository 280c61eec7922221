"""Plain FP64 restatement of the layered models for the tests: one function per mechanism, whole sequences only, no
cache, no batching, loops over tokens. Shares nothing with the library; `weights` maps tensor names to arrays.

Configurations are the dictionaries of config.json. `mistake` names a deliberate error (tests check that their inputs
would show it): "chunk-1", "chunk+1" (block size off by one), "chunk-from-portion" (blocks counted from position
`portion`), "lost-state" (recurrent states zeroed at position `portion`), "no-page" (keys at [portion, portion + 4)
unseen)."""
import math

import numpy as np

erf = np.vectorize(math.erf, otypes=[np.float64])


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def rms_divided(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, weight, bias, eps):
    centred = x - x.mean(axis=-1, keepdims=True)
    return centred / np.sqrt(np.mean(centred ** 2, axis=-1, keepdims=True) + eps) * weight + bias


def position_vectors(n, width):
    out = np.zeros((n, width))
    for c in range(width):
        angle = np.arange(n) / 10000.0 ** (2 * (c // 2) / width)
        out[:, c] = np.cos(angle) if c % 2 else np.sin(angle)
    return out


def visible(n, size, mistake=None, portion=0):
    """visible[i, j]: position i sees position j."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    if size is None:
        seen = j <= i
    else:
        size = size + {"chunk-1": -1, "chunk+1": 1}.get(mistake, 0)
        shift = portion if mistake == "chunk-from-portion" else 0
        seen = (j <= i) & ((i - shift) // size == (j - shift) // size)
    if mistake == "no-page":
        seen = seen & ~((j >= portion) & (j < portion + 4) & (i != j))
    return seen


def softmax_attention(h, w, p, m, eps, mistake=None, portion=0):
    n, heads, groups = len(h), m["heads"], m["kv_heads"]
    q = rms_divided((h @ w[p + "q"].T).reshape(n, heads, m["dim"]), eps) * w[p + "q.norm"]
    k = rms_divided((h @ w[p + "k"].T).reshape(n, groups, m["dim"]), eps) * w[p + "k.norm"]
    v = rms_divided((h @ w[p + "v"].T).reshape(n, groups, m["vdim"]), eps)
    seen = visible(n, m["mask"]["size"] if m.get("mask") else None, mistake, portion)
    out = np.zeros((n, heads, m["vdim"]))
    for head in range(heads):
        g = head // (heads // groups)
        score = np.where(seen, q[:, head] @ k[:, g].T * m["scale"], -np.inf)
        weight = np.exp(score - score.max(axis=1, keepdims=True))
        out[:, head] = weight / weight.sum(axis=1, keepdims=True) @ v[:, g]
    return out.reshape(n, -1) @ w[p + "o"].T


def gated_linear_attention(h, w, p, m, eps, mistake=None, portion=0):
    n, heads, dk, dv = len(h), m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).reshape(n, heads, dk) / math.sqrt(dk)
    k = (h @ w[p + "k"].T).reshape(n, heads, dk)
    v = (h @ w[p + "v"].T).reshape(n, heads, dv)
    decay = sigmoid(h @ w[p + "a1"].T @ w[p + "a2"].T + w[p + "a2.b"]).reshape(n, heads, dk) ** (1.0 / m["tau"])
    state, out = np.zeros((heads, dk, dv)), np.zeros((n, heads, dv))
    for t in range(n):
        if mistake == "lost-state" and t == portion:
            state[:] = 0
        state = decay[t][:, :, None] * state + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hkv,hk->hv", state, q[t])
    gate = h @ w[p + "g"].T
    return ((rms_divided(out, eps) * w[p + "norm"]).reshape(n, -1) * gate * sigmoid(gate)) @ w[p + "o"].T


def delta_rule(h, w, p, m, eps, mistake=None, portion=0):
    n, heads, d = len(h), m["heads"], m["dim"]
    r, k, v = ((h @ w[p + x].T).reshape(n, heads, d) for x in "rkv")
    decay = np.exp(-math.exp(-0.5) * sigmoid(np.tanh(h @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).reshape(n, heads, d)
    removal = sigmoid(h @ w[p + "a"].T + w[p + "a.b"]).reshape(n, heads, d)
    unit = k / np.sqrt((k * k).sum(axis=-1, keepdims=True) + 1e-6)
    state, out = np.zeros((heads, d, d)), np.zeros((n, heads, d))
    for t in range(n):
        if mistake == "lost-state" and t == portion:
            state[:] = 0
        old = state
        read = np.einsum("hk,hkv->hv", unit[t], old)
        state = decay[t][:, :, None] * old - (removal[t] * unit[t])[:, :, None] * read[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hkv,hk->hv", state, r[t])
    return (rms_divided(out, eps).reshape(n, -1) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, w, p, m, eps, **kw):
    return (m["left_scale"] * softmax_attention(h, w, p + "left.", m["left"], eps, **kw) +
            m["right_scale"] * delta_rule(h, w, p + "right.", m["right"], eps, **kw))


def feed_forward(h, w, p):
    z = h @ w[p + "up"].T
    return 0.5 * z * (1 + erf(z / math.sqrt(2))) @ w[p + "down"].T


def forward(cfg, weights, ids, **kw):
    """Logits [len(ids), vocab]."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps, ids = cfg["norm"]["eps"], np.asarray(ids)
    x = w["embed"][ids] + position_vectors(len(ids), cfg["width"])
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        norm = lambda v, name: layer_norm(v, w[p + name], w[p + name + ".b"], eps)
        mixer = {"gla": gated_linear_attention, "parallel": parallel}[layer["type"]]
        x = x + norm(mixer(norm(x, "norm1"), w, p + "mix.", layer["mixer"], eps, **kw), "norm1b")
        if layer.get("mlp"):
            x = x + norm(feed_forward(norm(x, "norm2"), w, p + "mlp."), "norm2b")
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["embed"].T


# ------------------------------------------------------------------ small random models
def gla(heads, dim, vdim, tau=16.0, ff=0):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def pair(heads, kv_heads, dim, vdim, size, rheads, rdim, scale=None, left_scale=1.0, right_scale=1.0, ff=0):
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
                               "scale": dim ** -0.5 if scale is None else scale},
                      "right": {"heads": rheads, "dim": rdim}, "left_scale": left_scale, "right_scale": right_scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Dirurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def shapes(cfg, rank=5):
    """Tensor names and shapes of a configuration."""
    W, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}

    def norm(name):
        out[name], out[name + ".b"] = (W,), (W,)

    norm("final.norm")
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        norm(p + "norm1")
        norm(p + "norm1b")
        if layer["type"] == "gla":
            K, V, q = m["heads"] * m["dim"], m["heads"] * m["vdim"], p + "mix."
            out.update({q + "q": (K, W), q + "k": (K, W), q + "v": (V, W), q + "g": (V, W), q + "o": (W, V),
                        q + "norm": (m["vdim"],), q + "a1": (rank, W), q + "a2": (K, rank), q + "a2.b": (K,)})
        else:
            a, r, q = m["left"], m["right"], p + "mix.left."
            out.update({q + "q": (a["heads"] * a["dim"], W), q + "k": (a["kv_heads"] * a["dim"], W),
                        q + "v": (a["kv_heads"] * a["vdim"], W), q + "o": (W, a["heads"] * a["vdim"]),
                        q + "q.norm": (a["dim"],), q + "k.norm": (a["dim"],)})
            K, q = r["heads"] * r["dim"], p + "mix.right."
            out.update({q + x: (K, W) for x in "rkvga"})
            out.update({q + "o": (W, K), q + "norm": (K,), q + "a.b": (K,), q + "w1": (rank + 2, W),
                        q + "w2": (K, rank + 2), q + "w0": (K,)})
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            norm(p + "norm2")
            norm(p + "norm2b")
            out.update({p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def random_weights(cfg, seed, rank=5):
    """Random weights on the BF16 grid (so that BF16 storage is exact): inputs of products of unit size, norms around 1,
    biases and decays away from 0, slow decays in the recurrences so that old tokens still matter."""
    from puppygrad_b200.synthetic import round_bf16
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg, rank).items():
        leaf = name.split(".")[-1]
        if len(shape) == 2:
            a = rng.standard_normal(shape) / math.sqrt(shape[1])
            if name == "embed":
                a = rng.standard_normal(shape)
            if leaf in ("a2", "w2"):
                a = a * 2
        elif leaf == "b" and name.endswith("a2.b"):
            a = rng.standard_normal(shape) + 3.0   # decays near 1
        elif leaf == "w0":
            a = rng.standard_normal(shape) - 4.0
        elif name.endswith("a.b"):
            a = rng.standard_normal(shape) - 1.0
        elif leaf == "b":
            a = rng.standard_normal(shape) * 0.2
        else:
            a = 1.0 + 0.2 * rng.standard_normal(shape)
        out[name] = round_bf16(a.astype(np.float32))
    return out
