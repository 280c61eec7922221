"""CPU checks of the layered models: configuration and tensor errors, registry, trace replay bookkeeping, command line,
and the plain restatement that the GPU tests compare with."""
import copy
import io
import json

import numpy as np
import pytest

import puppygrad_b200 as pg
from puppygrad_b200 import _native as N
from puppygrad_b200 import registry, synthetic, trace
from tests import layered_oracle as lo

SMALL = lo.config(37, 24, [lo.gla(2, 6, 10, tau=8.0), lo.pair(4, 2, 8, 6, 5, 3, 4, ff=28)])


def model_dir(tmp_path, cfg, weights=None, **kw):
    return synthetic.write_design_dir(str(tmp_path), cfg, lo.random_weights(cfg, 1) if weights is None else weights, **kw)


def load_error(path):
    with pytest.raises(pg.DesignError) as e:
        pg.load_model(path, pg.CudaConfig(math_mode="fp32"))
    return e.value


def test_registry_chooses_the_class_by_architecture(tmp_path):
    d = model_dir(tmp_path / "a", SMALL)
    assert registry.model_class(registry.architecture_of(d)) is pg.DiruraxModel
    g = synthetic.write_model_dir(str(tmp_path / "g"), synthetic.preset("tiny"), synthetic.tiny_weights())
    assert registry.model_class(registry.architecture_of(g)) is pg.Gpt2Model
    with pytest.raises(pg.DesignError, match="unknown architecture 'Nobody'"):
        registry.model_class("Nobody")
    assert N.lib.pg_registered_architectures().decode().split(", ") == list(pg.MODELS)


def test_unknown_architecture_is_refused_by_the_library(tmp_path):
    d = model_dir(tmp_path, SMALL)
    cfg = dict(SMALL, architecture="Nobody")
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    with pytest.raises(pg.Gpt2Error, match='unknown architecture "Nobody"') as e:
        pg.Gpt2Model.from_dir(d, pg.CudaConfig())
    assert e.value.kind == "InvalidConfig"


@pytest.mark.parametrize("edit, message", [
    (lambda c: c.pop("vocab"), "missing or invalid integer `vocab`"),
    (lambda c: c.update(width=0), "`width` 0 must be in"),
    (lambda c: c.pop("norm"), "missing `norm`"),
    (lambda c: c["norm"].update(eps=0.0), "eps must be > 0"),
    (lambda c: c.update(layers=[]), "missing `layers`"),
    (lambda c: c["layers"][0].update(type="lstm"), 'unknown type "lstm"'),
    (lambda c: c["layers"][0]["mixer"].pop("tau"), "missing or invalid number `tau`"),
    (lambda c: c["layers"][0]["mixer"].update(dim=1000), "`dim` 1000 must be in"),
    (lambda c: c["layers"][0]["mixer"].update(heads=1.5), "invalid integer `heads`"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "missing `left` or `right`"),
    (lambda c: c["layers"][1]["mixer"].pop("left_scale"), "missing or invalid number `left_scale`"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "must be divisible by kv_heads 3"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0), "`size` 0 must be in"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "unknown kind"),
])
def test_configuration_errors(tmp_path, edit, message):
    cfg = copy.deepcopy(SMALL)
    edit(cfg)
    err = load_error(model_dir(tmp_path, cfg, lo.random_weights(SMALL, 1)))
    assert err.kind == "InvalidConfig" and message in err.message, err.message


def test_tensor_errors(tmp_path):
    w = lo.random_weights(SMALL, 1)
    missing = {k: v for k, v in w.items() if k != "l1.mix.right.w0"}
    err = load_error(model_dir(tmp_path / "m", SMALL, missing))
    assert err.kind == "Asset" and "tensor l1.mix.right.w0 not found" in err.message
    shape = dict(w, **{"l0.mix.v": w["l0.mix.v"][:-1]})
    err = load_error(model_dir(tmp_path / "s", SMALL, shape))
    assert err.kind == "InvalidWeights" and "tensor l0.mix.v shape [19, 24] does not match expected [20, 24]" in err.message
    rank = dict(w, **{"l0.mix.a2": w["l0.mix.a2"][:, :-1].copy()})  # the two halves of the decay projection must agree
    err = load_error(model_dir(tmp_path / "r", SMALL, rank))
    assert err.kind == "InvalidWeights" and "l0.mix.a2" in err.message


def test_modes_that_the_layered_models_do_not_have(tmp_path):
    d = model_dir(tmp_path, SMALL)
    for conf, message in [(pg.CudaConfig(math_mode="tf32x3"), "must be fp32 or bf16"),
                          (pg.CudaConfig(math_mode="fp32", quantized_weights=True), "quantized_weights is not available"),
                          (pg.CudaConfig(math_mode="bf16", page_tokens=24), "page_tokens"),
                          (pg.CudaConfig(math_mode="bf16", max_context=-1), "max_context")]:
        with pytest.raises(pg.DesignError, match=message) as e:
            pg.load_model(d, conf)
        assert e.value.kind == "InvalidConfig"


def test_there_is_no_cpu_fallback(tmp_path):
    if N.lib.pg_device_count() > 0:
        pytest.skip("a GPU is present")
    assert load_error(model_dir(tmp_path, SMALL)).kind == "Cuda"


class FakeCache:
    def __init__(self, max_batch):
        self.max_batch, self.cleared = max_batch, []

    def clear_slot(self, slot):
        self.cleared.append(slot)


class FakeModel:
    """Logits of a row = [slot, tokens the slot holds up to and with the row]."""

    class config:
        vocab_size = 2

    def __init__(self):
        self.held = {}

    def new_kv_cache(self, max_batch):
        self.cache = FakeCache(max_batch)
        return self.cache

    def extend(self, slots, portions, cache, want):
        rows = []
        for s, p in zip(slots, portions):
            for _ in p:
                self.held[s] = self.held.get(s, 0) + 1
                rows.append([s, self.held[s]])
        return np.array([rows[w] for w in want], np.float32).reshape(-1, 2)


def test_trace_replay_keeps_a_slot_per_name_and_gives_it_back():
    model = FakeModel()
    r = trace.TraceReplay(model, 2)
    out = r.step([{"id": "a", "tokens": [1, 2], "want": [1]}, {"id": "b", "tokens": [3], "want": [0]}], [])
    assert out.tolist() == [[0, 2], [1, 1]]
    out = r.step([{"id": "b", "tokens": [4, 5], "want": [1, 0]}], ["a"])
    assert out.tolist() == [[1, 3], [1, 2]] and model.cache.cleared == [0]
    model.held.pop(0)
    assert r.step([{"id": "c", "tokens": [9], "want": []}], ["b", "c"]).shape == (0, 2)
    assert sorted(r.free) == [0, 1] and r.slot_of == {}
    r.step([{"id": "x", "tokens": [1]}, {"id": "y", "tokens": [1]}], [])
    with pytest.raises(pg.Gpt2Error, match="more than 2 sequences"):
        r.step([{"id": "z", "tokens": [1]}], [])


def test_trace_run_writes_files_and_done_lines(tmp_path, monkeypatch):
    model = FakeModel()
    monkeypatch.setattr(trace, "load_model", lambda path, conf: model)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [0, 2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [4], "want": []}], "end": ["a"]}]
    out = io.StringIO()
    rc = trace.main(["--model", "m", "--dtype", "bfloat16", "--out", str(tmp_path), "--max-tokens", "9"],
                    io.StringIO("".join(json.dumps(x) + "\n" for x in lines)), out)
    assert rc == 0 and out.getvalue() == "done 0\ndone 1\n"
    assert np.fromfile(tmp_path / "0.f32", "<f4").tolist() == [0, 1, 0, 3] and not (tmp_path / "1.f32").exists()


# ------------------------------------------------------------------ the restatement itself
def test_restatement_visibility():
    seen = lo.visible(9, 4)
    assert [list(np.nonzero(r)[0]) for r in seen[[0, 3, 4, 7, 8]]] == [[0], [0, 1, 2, 3], [4], [4, 5, 6, 7], [8]]
    assert lo.visible(5, None)[4].all()


def test_restatement_recurrences_by_hand():
    """Two tokens, one head, everything written out."""
    eps, rng = 1e-5, np.random.default_rng(0)
    h = rng.standard_normal((2, 3))
    cfg = lo.config(7, 3, [lo.gla(1, 2, 2, tau=4.0), lo.pair(1, 1, 2, 2, 4, 1, 2)])
    w = {k: np.asarray(v, np.float64) for k, v in lo.random_weights(cfg, 3, rank=2).items()}
    p = "l0.mix."
    a = [1 / (1 + np.exp(-(w[p + "a2"] @ (w[p + "a1"] @ x) + w[p + "a2.b"]))) for x in h]
    k, v = [w[p + "k"] @ x for x in h], [w[p + "v"] @ x for x in h]
    state = np.diag(a[1] ** 0.25) @ np.outer(k[0], v[0]) + np.outer(k[1], v[1])
    o = state.T @ (w[p + "q"] @ h[1]) * 2 ** -0.5
    g = w[p + "g"] @ h[1]
    want = w[p + "o"] @ (o / np.sqrt((o * o).mean() + eps) * w[p + "norm"] * g / (1 + np.exp(-g)))
    np.testing.assert_allclose(lo.gated_linear_attention(h, w, p, cfg["layers"][0]["mixer"], eps)[1], want, rtol=1e-12)
    p = "l1.mix.right."
    k, v = [w[p + "k"] @ x for x in h], [w[p + "v"] @ x for x in h]
    s0 = np.outer(k[0], v[0])
    u = k[1] / np.sqrt(k[1] @ k[1] + 1e-6)
    rate = 1 / (1 + np.exp(-(w[p + "a"] @ h[1] + w[p + "a.b"])))
    dec = np.exp(-np.exp(-0.5) / (1 + np.exp(-(w[p + "w2"] @ np.tanh(w[p + "w1"] @ h[1]) + w[p + "w0"]))))
    s1 = np.diag(dec) @ s0 - np.outer(rate * u, u @ s0) + np.outer(k[1], v[1])
    o = s1.T @ (w[p + "r"] @ h[1])
    want = w[p + "o"] @ (o / np.sqrt((o * o).mean() + eps) * w[p + "norm"] / (1 + np.exp(-(w[p + "g"] @ h[1]))))
    np.testing.assert_allclose(lo.delta_rule(h, w, p, cfg["layers"][1]["mixer"]["right"], eps)[1], want, rtol=1e-12)


def test_restatement_is_causal_and_positions_matter():
    w = lo.random_weights(SMALL, 5)
    ids = np.random.default_rng(1).integers(0, 37, 14)
    full = lo.forward(SMALL, w, ids)
    np.testing.assert_allclose(lo.forward(SMALL, w, ids[:9]), full[:9], rtol=1e-10, atol=1e-10)
    assert np.abs(full[3] - lo.forward(SMALL, w, np.roll(ids, 1))[4]).max() > 1e-2
