"""CPU checks of the Sanesun design: configuration and tensor errors, registry, and the plain restatement that the GPU tests
compare with."""
import copy

import numpy as np
import pytest

import puppygrad_b200 as pg
from puppygrad_b200 import registry, synthetic
from tests import sanesun_oracle as so
from tests.layered_cases import BOUND, row_errors

SMALL = so.config(37, 24, [so.att(4, 2, 8, 6, 5, 2, ff=28), so.delta(4, 2, 6, 10, 3), so.latent(3, 6, 8, 12, 10, ff=20)])


def model_dir(tmp_path, cfg, weights=None, **kw):
    return synthetic.write_design_dir(str(tmp_path), cfg, so.random_weights(cfg, 1) if weights is None else weights, **kw)


def load_error(path):
    with pytest.raises(pg.DesignError) as e:
        pg.load_model(path, pg.CudaConfig(math_mode="fp32"))
    return e.value


def test_registry(tmp_path):
    d = model_dir(tmp_path, SMALL)
    assert registry.model_class(registry.architecture_of(d)) is pg.SanesunModel
    conf = pg.SanesunConfig.from_dict(SMALL, 99)
    assert conf.to_dict() == SMALL and conf.n_layer == 3 and conf.vocab_size == 37 and conf.n_positions == 99


@pytest.mark.parametrize("edit, message", [
    (lambda c: c.pop("embedding"), "missing `embedding`"),
    (lambda c: c["embedding"].pop("scale"), "missing or invalid number `scale`"),
    (lambda c: c["norm"].update(eps=-1), "eps must be > 0"),
    (lambda c: c["layers"][0].update(type="gla"), 'unknown type "gla"'),
    (lambda c: c["layers"][0]["mixer"].pop("rot"), "missing `rot`"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "`dims` 10 must be in 0..8"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3), "must be even"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=0), "base must be > 0"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=7), "must be even"),
    (lambda c: c["layers"][0]["mixer"]["mask"].pop("keep_first"), "invalid integer `keep_first`"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "`size` 0 must be in"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "must be divisible by kv_heads 3"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "must be divisible by kv_heads 3"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "invalid integer `conv`"),
    (lambda c: c["layers"][2]["mixer"].pop("kv_rank"), "invalid integer `kv_rank`"),
    (lambda c: c["layers"][2]["mixer"].update(q_rank=0), "`q_rank` 0 must be in"),
    (lambda c: c["layers"][2]["mlp"].update(kind="moe"), "unknown kind"),
])
def test_configuration_errors(tmp_path, edit, message):
    cfg = copy.deepcopy(SMALL)
    edit(cfg)
    err = load_error(model_dir(tmp_path, cfg, so.random_weights(SMALL, 1)))
    assert err.kind == "InvalidConfig" and message in err.message, err.message


def test_tensor_errors(tmp_path):
    w = so.random_weights(SMALL, 1)
    for i, name in enumerate(("head", "l0.mix.q.b", "l0.mix.talk", "l0.mix.sink", "l1.mix.k.conv", "l1.mix.dt_bias", "l2.mix.uv", "l2.mlp.act", "l1.norm1")):
        err = load_error(model_dir(tmp_path / f"m{i}", SMALL, {k: v for k, v in w.items() if k != name}))
        assert err.kind == "Asset" and f"tensor {name} not found" in err.message
    for i, (name, cut) in enumerate((("l1.mix.a2", np.s_[:, :-1]), ("l1.mix.g2", np.s_[:, :-1]), ("l0.mix.talk", np.s_[:-1]), ("l2.mix.uk", np.s_[:-1]),
                                     ("l1.mix.v.conv", np.s_[:, :-1]))):
        err = load_error(model_dir(tmp_path / f"s{i}", SMALL, dict(w, **{name: w[name][cut].copy()})))
        assert err.kind == "InvalidWeights" and name in err.message


# ------------------------------------------------------------------ the restatement itself
def test_restatement_window():
    seen = so.window(9, 3, 2)
    assert [list(np.nonzero(r)[0]) for r in seen[[0, 1, 3, 4, 8]]] == [[0], [0, 1], [0, 1, 2, 3], [0, 1, 2, 3, 4], [0, 1, 6, 7, 8]]
    assert [list(np.nonzero(r)[0]) for r in so.window(4, 1, 0)] == [[0], [1], [2], [3]]


def test_restatement_rotation():
    """Scores of rotated rows depend on distances only, the entries past `dims` stay, turning back undoes a rotation."""
    rng = np.random.default_rng(0)
    x, y = rng.standard_normal((1, 1, 8)), rng.standard_normal((1, 1, 8))
    at = lambda v, p: so.turned(v, np.array([float(p)]), 6, 50.0)
    np.testing.assert_allclose((at(x, 9) * at(y, 4)).sum(), (at(x, 105) * at(y, 100)).sum(), rtol=1e-12)
    assert (at(x, 9)[..., 6:] == x[..., 6:]).all()
    np.testing.assert_allclose(so.turned(at(x, 9), np.array([9.0]), 6, 50.0, -1.0), x, rtol=1e-12)
    a = 3 * 50.0 ** (-2 / 6)  # pair 1 = entries 1 and 4
    np.testing.assert_allclose(at(x, 3)[0, 0, 4], x[0, 0, 4] * np.cos(a) + x[0, 0, 1] * np.sin(a), rtol=1e-12)


def test_restatement_attention_by_hand():
    """The last of three tokens, two heads over one key head, everything written out."""
    cfg = so.config(7, 5, [so.att(2, 1, 4, 2, 2, 1, dims=2, base=10.0, scale=0.7)])
    w = {k: np.asarray(v, np.float64) for k, v in so.random_weights(cfg, 3).items()}
    h, p, m = np.random.default_rng(1).standard_normal((3, 5)), "l0.mix.", cfg["layers"][0]["mixer"]
    rot = lambda v, a: np.concatenate([[v[0] * np.cos(a) - v[1] * np.sin(a), v[1] * np.cos(a) + v[0] * np.sin(a)], v[2:]])
    keys = [rot(w[p + "k"] @ x + w[p + "k.b"], j) for j, x in enumerate(h)]       # one pair each: angle = position
    vals = [rot(w[p + "v"] @ x + w[p + "v.b"], j) for j, x in enumerate(h)]
    q = w[p + "q"] @ h[2] + w[p + "q.b"]
    raw = np.array([[rot(q[4 * a:4 * a + 4], 2) @ keys[j] * 0.7 for j in range(3)] for a in range(2)])
    mixed = w[p + "talk"] @ raw
    out = []
    for a in range(2):                                                            # token 2 sees 1 and 2, and the kept 0
        e = np.exp(mixed[a])
        o = sum(e[j] * vals[j] for j in range(3)) / (e.sum() + np.exp(w[p + "sink"][a]))
        out.append(rot(o, -2))
    np.testing.assert_allclose(so.attention(h, w, p, m, 1e-5)[2], w[p + "o"] @ np.concatenate(out), rtol=1e-11)


def test_restatement_channel_delta_by_hand():
    """Two tokens, two heads that share a key head, two taps."""
    cfg = so.config(7, 5, [so.delta(2, 1, 2, 3, 2)])
    w = {k: np.asarray(v, np.float64) for k, v in so.random_weights(cfg, 3, rank=2).items()}
    h, p, m, eps = np.random.default_rng(1).standard_normal((2, 5)), "l0.mix.", cfg["layers"][0]["mixer"], 1e-5
    sig = lambda z: 1 / (1 + np.exp(-z))
    rows = {}
    for n in "qkv":
        x, c = [w[p + n] @ t for t in h], w[p + n + ".conv"]
        z = [c[:, 1] * x[0], c[:, 0] * x[0] + c[:, 1] * x[1]]
        rows[n] = [v * sig(v) for v in z]
    unit = lambda v: v / np.sqrt(v @ v + 1e-6)
    out = []
    for a in range(2):
        s = np.zeros((2, 3))
        for t in range(2):
            z = (w[p + "a2"] @ (w[p + "a1"] @ h[t]) + w[p + "dt_bias"])[2 * a:2 * a + 2]
            s = np.exp(-np.exp(w[p + "A_log"][a]) * np.log(1 + np.exp(z)))[:, None] * s
            k, v = unit(rows["k"][t]), rows["v"][t][3 * a:3 * a + 3]
            s = s + np.outer(k, sig(w[p + "b"] @ h[t])[a] * (v - s.T @ k))
        o = s.T @ unit(rows["q"][1]) / np.sqrt(2)
        out.append(o / np.sqrt((o * o).mean() + eps) * w[p + "norm"] * sig(w[p + "g2"] @ (w[p + "g1"] @ h[1]))[3 * a:3 * a + 3])
    np.testing.assert_allclose(so.channel_delta(h, w, p, m, eps)[1], w[p + "o"] @ np.concatenate(out), rtol=1e-11)


def test_restatement_xielu():
    z = np.array([-3.0, -1e-4, 0.0, 1e-4, 2.0])
    got = so.xielu(z, 0.3, -0.4)
    a, b = np.log(1 + np.exp(0.3)), 0.5 + np.log(1 + np.exp(-0.4))
    np.testing.assert_allclose(got[[0, 4]], [b * (np.exp(-3) - 1 + 3) - 1.5, a * 4 + 1], rtol=1e-12)
    np.testing.assert_allclose(got[1:4], z[1:4] / 2, atol=1e-7)


def test_restatement_is_causal_and_positions_matter():
    w = so.random_weights(SMALL, 5)
    ids = np.random.default_rng(1).integers(0, 37, 14)
    full = so.forward(SMALL, w, ids)
    np.testing.assert_allclose(so.forward(SMALL, w, ids[:9]), full[:9], rtol=1e-10, atol=1e-10)
    assert np.abs(full[3] - so.forward(SMALL, w, np.roll(ids, 1))[4]).max() > 1e-2


@pytest.mark.parametrize("mistake", ["window-1", "window+1", "no-first", "first-1", "no-sink", "no-talk", "no-turn-back", "no-bias", "lost-state", "lost-taps",
                                     "late-read", "no-page", "portion-positions"])
def test_planted_mistakes_would_be_seen(mistake):
    """Each deliberate error of the restatement moves the logits of the GPU tests' inputs past the bounds used there."""
    from tests.test_sanesun_gpu import MIXED
    w = so.random_weights(MIXED, 11)
    ids = np.random.default_rng(1000).integers(0, MIXED["vocab"], 130)
    wrong = so.forward(MIXED, w, ids, mistake=mistake, portion=57)
    assert row_errors(wrong, so.forward(MIXED, w, ids)).max() > 1.5 * BOUND["bf16"]
