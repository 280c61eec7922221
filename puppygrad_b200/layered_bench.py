"""Throughput of a layered model beside an older model of equal width, depth, vocabulary and feed-forward size (random
weights): Dirurax beside GPT-2, Sanesun beside Dirurax.

    python bench.py --layered [--layered-design Sanesun] [--layered-widths 1024,2048] [--layered-depth 8]

Decode: `batch` sequences after 512-token prompts, greedy, token fed back on the device. Prefill: several prompts at
once, and (layered only: GPT-2 here ends at 1024 positions) one long prompt. Device time by CUDA events on the
library's stream; weights and states are larger than L2 for the larger sizes, the line says how many bytes a step reads.
"""
from __future__ import annotations

import math
import os
import shutil
import tempfile
from typing import Dict, List

import numpy as np

VOCAB, PROMPT, SPAN = 32000, 512, 512


def dirurax_config(width: int, depth: int) -> dict:
    """Three gated-linear-attention layers to one parallel layer, a feed-forward of four widths in each."""
    ff = {"kind": "dense", "ff": 4 * width}
    gla = {"type": "gla", "mixer": {"heads": width // 128, "dim": 64, "vdim": 128, "tau": 16.0}, "mlp": ff}
    par = {"type": "parallel",
           "mixer": {"left": {"heads": width // 64, "kv_heads": width // 256, "dim": 64, "vdim": 64, "mask": {"size": SPAN},
                              "scale": 0.125},
                     "right": {"heads": width // 64, "dim": 64}, "left_scale": 0.7, "right_scale": 0.7}, "mlp": ff}
    return {"architecture": "Dirurax", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-5},
            "layers": [par if i % 4 == 3 else gla for i in range(depth)]}


def sanesun_config(width: int, depth: int) -> dict:
    """Cycles of attention, channel delta rule, latent attention, channel delta rule; a feed-forward of four widths in each."""
    ff = {"kind": "dense", "ff": 4 * width}
    att = {"type": "attention", "mlp": ff,
           "mixer": {"heads": width // 64, "kv_heads": width // 256, "dim": 64, "vdim": 64, "scale": 0.125, "rot": {"dims": 32, "base": 1e4},
                     "mask": {"size": SPAN, "keep_first": 4}}}
    delta = {"type": "channel_delta", "mlp": ff,
             "mixer": {"heads": width // 128, "kv_heads": width // 128, "dim": 128, "vdim": 128, "conv": 4}}
    latent = {"type": "latent_attention", "mlp": ff,
              "mixer": {"heads": width // 128, "dim": 128, "vdim": 128, "kv_rank": 512, "q_rank": 3 * width // 8, "scale": 128 ** -0.5}}
    return {"architecture": "Sanesun", "vocab": VOCAB, "width": width, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
            "layers": [(att, delta, latent, delta)[i % 4] for i in range(depth)]}


def weight_pool(out: Dict[str, np.ndarray]):
    """Random weights: slices of one block of normal numbers (the values do not matter here)."""
    pool = np.random.default_rng(0).standard_normal(1 << 24, dtype=np.float32)
    at = [0]

    def mat(name, n, k):
        m = n * k
        at[0] = (at[0] + 7919) % 4096
        out[name] = np.resize(pool[at[0]:], m).reshape(n, k) * np.float32(1 / math.sqrt(k))

    def vec(name, n, v):
        out[name] = np.full(n, v, np.float32)

    return mat, vec


def sanesun_tensors(cfg: dict, rank: int = 128) -> Dict[str, np.ndarray]:
    W, out = cfg["width"], {}
    mat, vec = weight_pool(out)
    mat("embed", cfg["vocab"], W)
    mat("head", cfg["vocab"], W)
    vec("final.norm", W, 1.0)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", l["mixer"]
        H, V = m["heads"], m["heads"] * m["vdim"]
        vec(f"l{i}.norm1", W, 1.0)
        if l["type"] == "attention":
            for n, r in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                mat(p + n, r, W)
                vec(p + n + ".b", r, 0.1)
            mat(p + "talk", H, H)
            vec(p + "sink", H, 0.0)
        elif l["type"] == "channel_delta":
            Q = m["kv_heads"] * m["dim"]
            for n, r in (("q", Q), ("k", Q), ("v", V)):
                mat(p + n, r, W)
                mat(p + n + ".conv", r, m["conv"])
            for n, r, k in (("b", H, W), ("a1", rank, W), ("a2", H * m["dim"], rank), ("g1", rank, W), ("g2", V, rank)):
                mat(p + n, r, k)
            vec(p + "A_log", H, -1.0)
            vec(p + "dt_bias", H * m["dim"], -3.0)
            vec(p + "norm", m["vdim"], 1.0)
        else:
            for n, r, k in (("dq", m["q_rank"], W), ("uq", H * m["dim"], m["q_rank"]), ("dkv", m["kv_rank"], W), ("uk", H * m["dim"], m["kv_rank"]),
                            ("uv", V, m["kv_rank"]), ("g", H, W)):
                mat(p + n, r, k)
            vec(p + "dq.norm", m["q_rank"], 1.0)
            vec(p + "dkv.norm", m["kv_rank"], 1.0)
        mat(p + "o", W, V)
        if l["mlp"]:
            mat(f"l{i}.mlp.up", l["mlp"]["ff"], W)
            mat(f"l{i}.mlp.down", W, l["mlp"]["ff"])
            vec(f"l{i}.mlp.act", 2, 0.5)
    return out


def dirurax_tensors(cfg: dict, rank: int = 64) -> Dict[str, np.ndarray]:
    W, out = cfg["width"], {}
    mat, vec = weight_pool(out)

    def norm(name):
        vec(name, W, 1.0)
        vec(name + ".b", W, 0.0)

    mat("embed", cfg["vocab"], W)
    norm("final.norm")
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        norm(p + "norm1")
        norm(p + "norm1b")
        if l["type"] == "gla":
            K, V = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, r in (("q", K), ("k", K), ("v", V), ("g", V), ("a1", rank)):
                mat(p + "mix." + n, r, W)
            mat(p + "mix.a2", K, rank)
            mat(p + "mix.o", W, V)
            vec(p + "mix.a2.b", K, 2.0)
            vec(p + "mix.norm", m["vdim"], 1.0)
        else:
            a, r = m["left"], m["right"]
            q = p + "mix.left."
            mat(q + "q", a["heads"] * a["dim"], W)
            mat(q + "k", a["kv_heads"] * a["dim"], W)
            mat(q + "v", a["kv_heads"] * a["vdim"], W)
            mat(q + "o", W, a["heads"] * a["vdim"])
            vec(q + "q.norm", a["dim"], 1.0)
            vec(q + "k.norm", a["dim"], 1.0)
            q, K = p + "mix.right.", r["heads"] * r["dim"]
            for n in "rkvga":
                mat(q + n, K, W)
            mat(q + "w1", rank, W)
            mat(q + "w2", K, rank)
            mat(q + "o", W, K)
            vec(q + "w0", K, -4.0)
            vec(q + "a.b", K, -1.0)
            vec(q + "norm", K, 1.0)
        if l["mlp"]:
            norm(p + "norm2")
            norm(p + "norm2b")
            mat(p + "mlp.up", l["mlp"]["ff"], W)
            mat(p + "mlp.down", W, l["mlp"]["ff"])
    return out


def gpt2_config(width: int, depth: int) -> dict:
    return dict(vocab_size=VOCAB, n_positions=1024, n_embd=width, n_layer=depth, n_head=width // 64, n_inner=4 * width,
                layer_norm_epsilon=1e-5)


def gpt2_weights(cfg: dict) -> Dict[str, np.ndarray]:
    pool = np.random.default_rng(1).standard_normal(1 << 24, dtype=np.float32) * np.float32(0.02)
    c, f = cfg["n_embd"], cfg["n_inner"]
    shapes = {"wte.weight": (cfg["vocab_size"], c), "wpe.weight": (cfg["n_positions"], c), "ln_f.weight": (c,), "ln_f.bias": (c,)}
    for i in range(cfg["n_layer"]):
        p = f"h.{i}."
        shapes.update({p + "ln_1.weight": (c,), p + "ln_1.bias": (c,), p + "attn.c_attn.weight": (c, 3 * c), p + "attn.c_attn.bias": (3 * c,),
                       p + "attn.c_proj.weight": (c, c), p + "attn.c_proj.bias": (c,), p + "ln_2.weight": (c,), p + "ln_2.bias": (c,),
                       p + "mlp.c_fc.weight": (c, f), p + "mlp.c_fc.bias": (f,), p + "mlp.c_proj.weight": (f, c), p + "mlp.c_proj.bias": (c,)})
    return {n: (np.resize(pool, int(np.prod(s))).reshape(s) if len(s) == 2 else np.full(s, 1.0 if n.endswith("weight") else 0.0, np.float32))
            for n, s in shapes.items()}


def mixer_flops(cfg: dict, l: dict, lens: List[int]) -> float:
    """Multiply-adds (twice) of one mixer; recurrences counted as the scan runs them, attention over the visible pairs."""
    W, rows, m = cfg["width"], sum(lens), l["mixer"]
    if l["type"] == "gla":
        K, V = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        return 2.0 * rows * (W * (2 * K + 2 * V + 64) + V * W + 64 * K) + 2.0 * rows * K * m["vdim"] * 3
    if l["type"] == "parallel":
        a, r = m["left"], m["right"]
        K = r["heads"] * r["dim"]
        total = 2.0 * rows * W * (a["heads"] * (a["dim"] + a["vdim"]) + a["kv_heads"] * (a["dim"] + a["vdim"]) + 6 * K + 64)
        total += 2.0 * rows * r["heads"] * r["dim"] ** 2 * 5
        for n in lens:
            size = a["mask"]["size"]
            pairs = sum(min(size, n - s) * (min(size, n - s) + 1) / 2 for s in range(0, n, size))
            total += 2.0 * pairs * a["heads"] * (a["dim"] + a["vdim"])
        return total
    H, V = m["heads"], m["heads"] * m["vdim"]
    if l["type"] == "channel_delta":
        K, Q = H * m["dim"], m["kv_heads"] * m["dim"]
        return 2.0 * rows * (W * (2 * Q + 2 * V + H + 256) + 128 * (K + V)) + 2.0 * rows * K * m["vdim"] * 4
    if l["type"] == "latent_attention":
        total = 2.0 * rows * (W * (m["q_rank"] + m["kv_rank"] + H + V) + H * m["dim"] * m["q_rank"] + H * (m["dim"] + m["vdim"]) * m["kv_rank"])
        return total + sum(n * (n + 1) for n in lens) * H * (m["dim"] + m["vdim"])
    total = 2.0 * rows * W * (H * m["dim"] + m["kv_heads"] * (m["dim"] + m["vdim"]) + V)
    for n in lens:
        pairs = sum(min(i + 1, m["mask"]["size"] + m["mask"]["keep_first"]) for i in range(n))
        total += 2.0 * pairs * H * (m["dim"] + m["vdim"] + H)
    return total


def prefill_flops(cfg: dict, lens: List[int]) -> float:
    return sum(mixer_flops(cfg, l, lens) + (4.0 * sum(lens) * cfg["width"] * l["mlp"]["ff"] if l["mlp"] else 0.0) for l in cfg["layers"])


def decode_bytes(pg_model, cfg: dict, batch: int, context: int) -> float:
    """Weights once, every sequence's recurrent states read and written, the visible keys and values read."""
    keys = 0.0
    for l in cfg["layers"]:
        m = l["mixer"]
        if l["type"] == "parallel":
            a = m["left"]
            keys += (context % a["mask"]["size"] + 1) * a["kv_heads"] * (a["dim"] + a["vdim"]) * 2
        elif l["type"] == "attention":
            keys += min(context, m["mask"]["size"] + m["mask"]["keep_first"]) * m["kv_heads"] * (m["dim"] + m["vdim"]) * 2
        elif l["type"] == "latent_attention":
            keys += context * m["kv_rank"] * 2
    return pg_model.weight_bytes_per_step() + batch * (2 * pg_model.state_bytes_per_sequence() + keys)


def build(cfg: dict, tensors: Dict[str, np.ndarray], device: int):
    import puppygrad_b200 as pg
    from puppygrad_b200 import synthetic
    tmp = tempfile.mkdtemp()
    try:
        synthetic.write_design_dir(tmp, cfg, tensors)
        return pg.load_model(tmp, pg.CudaConfig(device=device, math_mode="bf16", max_context=16384))
    finally:
        shutil.rmtree(tmp)


DESIGNS = {"Dirurax": (dirurax_config, dirurax_tensors), "Sanesun": (sanesun_config, sanesun_tensors)}


def time_decode(model, batch: int, prompts, steps: int) -> Dict[str, float]:
    cache = model.new_kv_cache(max_batch=batch)
    _, first = model.prefill_batch(prompts[:batch], cache)
    first = model.decode_greedy(first, cache, 4)[-1]
    best, launches = None, 0
    for _ in range(3):
        n0 = cache.kernel_launches()
        cache.time_begin()
        first = model.decode_greedy(first, cache, steps)[-1]
        sec = cache.time_end()
        launches = (cache.kernel_launches() - n0) // steps
        best = sec if best is None else min(best, sec)
    prof: Dict[str, float] = {}
    for _ in range(3):
        for k, v in model.profile_forward_one(first, cache).items():
            prof[k] = min(prof.get(k, 1e9), v[0] * 1e6)
    return {"tokens_per_s": batch * steps / best, "us_per_step": best / steps * 1e6, "launches_per_step": launches,
            "profile_us": {k: round(v, 1) for k, v in prof.items()}}


def time_prefill(model, prompts) -> Dict[str, float]:
    cache = model.new_kv_cache(max_batch=len(prompts))
    best = None
    for i in range(5):
        cache.time_begin()
        model.prefill_batch(prompts, cache)
        sec = cache.time_end()
        if i >= 2:
            best = sec if best is None else min(best, sec)
    rows = sum(len(p) for p in prompts)
    return {"tokens_per_s": rows / best, "ms": best * 1e3}


def measure_layered(name: str, width: int, depth: int, device: int, steps: int, peaks, prompts, wide, long) -> Dict[str, dict]:
    hbm, tflops, _ = peaks
    config, tensors = DESIGNS[name]
    cfg = config(width, depth)
    model = build(cfg, tensors(cfg), device)
    d: Dict[str, dict] = {}
    for batch in (1, 8, 64):
        r = time_decode(model, batch, prompts, steps)
        r["bytes_per_step"] = decode_bytes(model, cfg, batch, PROMPT + 2 * steps)
        r["hbm_frac"] = r["bytes_per_step"] / (r["us_per_step"] * 1e-6) / 1e9 / hbm
        d[f"decode_b{batch}"] = r
    for label, ps in (("prefill_8x1024", wide), ("prefill_1x8192", long)):
        r = time_prefill(model, ps)
        r["tflops"] = prefill_flops(cfg, [len(p) for p in ps]) / (r["ms"] * 1e-3) / 1e12
        r["bf16_frac"] = r["tflops"] / tflops
        cache = model.new_kv_cache(max_batch=len(ps))
        model.prefill_batch(ps, cache)
        r["profile_us"] = {k: round(v[0] * 1e6, 1) for k, v in model.profile_prefill(ps, cache).items()}
        del cache
        d[label] = r
    return d


def measure_gpt2(width: int, depth: int, device: int, steps: int, peaks, prompts, wide) -> Dict[str, dict]:
    import puppygrad_b200 as pg
    hbm, tflops, _ = peaks
    g: Dict[str, dict] = {}
    gcfg = gpt2_config(width, depth)
    model = pg.Gpt2Model(gcfg, gpt2_weights(gcfg), pg.Gpt2CudaConfig(device=device, math_mode="bf16"))
    for batch in (1, 8, 64):
        r = time_decode(model, batch, prompts, steps)
        kv = batch * 2 * depth * (PROMPT + 2 * steps) * width * 4
        r["bytes_per_step"] = (model.weight_bytes_per_step() * (1 if batch <= 8 else 2)) + kv  # above 8 rows: FP32 copies
        r["hbm_frac"] = r["bytes_per_step"] / (r["us_per_step"] * 1e-6) / 1e9 / hbm
        g[f"decode_b{batch}"] = r
    r = time_prefill(model, wide)
    flops = 2.0 * 8 * 1024 * depth * 12 * width ** 2 + 8 * depth * 2.0 * 1024 * 1025 * width
    r["tflops"] = flops / (r["ms"] * 1e-3) / 1e12
    r["bf16_frac"] = r["tflops"] / tflops
    g["prefill_8x1024"] = r
    return g


def run(device: int, widths: List[int], depth: int, steps: int, peaks, compare: bool = True, design: str = "Dirurax") -> dict:
    rng = np.random.default_rng(3)
    prompts = [rng.integers(0, VOCAB, PROMPT) for _ in range(64)]
    wide = [rng.integers(0, VOCAB, 1024) for _ in range(8)]
    long = [rng.integers(0, VOCAB, 8192)]
    out = {"peak_source": peaks[2], "depth": depth, "sizes": {}}
    for width in widths:
        layered = lambda name: measure_layered(name, width, depth, device, steps, peaks, prompts, wide, long)
        entry = {design: layered(design)}
        if compare and design == "Dirurax":
            entry["gpt2"] = measure_gpt2(width, depth, device, steps, peaks, prompts, wide)
        elif compare:
            entry["Dirurax"] = layered("Dirurax")
        out["sizes"][str(width)] = entry
    return out
