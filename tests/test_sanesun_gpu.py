"""GPU tests of the Sanesun design against its plain FP64 restatement (sanesun_oracle.py): each mechanism alone, prompts
against decoding, portions, batches, reuse of pages and slots, edges of windows and pages, generation."""
import io

import numpy as np
import pytest

import puppygrad_b200 as pg
from puppygrad_b200 import trace
from tests import layered_cases as cases
from tests import sanesun_oracle as so
from tests.layered_cases import BOUND, MODES, assert_rows, assert_stream, cut, row_errors, run_portions

pytestmark = pytest.mark.gpu


def Case(cfg, seed, **kw):
    return cases.Case(so, cfg, seed, **kw)


MIXED = so.config(97, 72, [so.delta(6, 2, 12, 20, 4, ff=40), so.att(6, 2, 20, 12, 23, 5, ff=88), so.latent(5, 12, 20, 24, 28),
                           so.delta(3, 3, 20, 8, 3), so.att(4, 4, 8, 16, 40, 0, dims=8, base=300.0), so.latent(2, 24, 8, 40, 12, ff=56)])


@pytest.fixture(scope="module")
def mixed():
    return Case(MIXED, 11)


# ------------------------------------------------------------------ each mechanism alone
ALONE = {
    "attention": so.att(6, 2, 16, 24, 21, 3),
    "attention-odd": so.att(9, 3, 7, 10, 13, 4, dims=6, base=77.0, scale=0.3),
    "attention-one-head": so.att(1, 1, 16, 8, 9, 1),
    "attention-one-key-head": so.att(7, 1, 24, 16, 30, 2),
    "attention-own-keys": so.att(5, 5, 24, 8, 17, 6),
    "attention-wide-groups": so.att(18, 2, 8, 8, 25, 3),
    "attention-many-heads": so.att(40, 8, 16, 8, 33, 7),
    "attention-two-groups-of-heads": so.att(64, 16, 16, 64, 150, 5),
    "attention-300-heads": so.att(300, 1, 16, 8, 140, 2),
    "attention-row-of-5120": so.att(40, 40, 128, 8, 21, 3),
    "attention-row-of-320": so.att(5, 5, 64, 64, 40, 3),
    "attention-row-of-544": so.att(4, 4, 136, 72, 50, 2),
    "attention-row-of-1024": so.att(8, 8, 128, 136, 31, 9),
    "attention-256": so.att(2, 2, 256, 256, 37, 5),
    "attention-window-1": so.att(4, 2, 16, 8, 1, 0),
    "attention-window-1-keeps": so.att(4, 2, 16, 8, 1, 2),
    "attention-keeps-none": so.att(4, 2, 16, 8, 20, 0),
    "attention-keeps-more": so.att(4, 2, 16, 8, 6, 40),
    "attention-sees-all": so.att(4, 2, 16, 8, 500, 3),
    "attention-rotates-all": so.att(4, 2, 16, 8, 20, 2, dims=16),
    "attention-rotates-none": so.att(4, 2, 16, 8, 20, 2, dims=0),
    "attention-negative-scale": so.att(4, 2, 16, 8, 20, 2, scale=-0.2),
    "delta": so.delta(6, 2, 16, 24, 4),
    "delta-odd": so.delta(6, 3, 7, 9, 3),
    "delta-one": so.delta(1, 1, 8, 8, 2),
    "delta-no-past-inputs": so.delta(4, 4, 8, 12, 1),
    "delta-six-taps": so.delta(4, 2, 12, 8, 6),
    "delta-one-key-head": so.delta(5, 1, 20, 16, 4),
    "delta-128": so.delta(2, 1, 128, 128, 4),
    "delta-72": so.delta(2, 2, 72, 40, 4),
    "delta-256": so.delta(1, 1, 200, 256, 3),
    "delta-narrow-keys": so.delta(2, 2, 4, 96, 3),
    "latent": so.latent(6, 16, 24, 40, 28),
    "latent-odd": so.latent(3, 7, 9, 13, 11, scale=0.5),
    "latent-one": so.latent(1, 16, 8, 8, 12),
    "latent-many-heads": so.latent(40, 8, 8, 64, 16),
    "latent-512": so.latent(16, 64, 72, 512, 200),
    "latent-two-groups-of-heads": so.latent(130, 8, 8, 500, 16),
    "latent-1000": so.latent(3, 128, 256, 1000, 48),
    "feed-forward": so.delta(1, 1, 4, 4, 2, ff=136),
}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", ALONE)
def test_mechanism_alone(name, mode):
    case = Case(so.config(59, 50 if "odd" in name else 64, [ALONE[name]]), 3, rank=3 if "odd" in name else 16)
    ids = case.ids(173)
    model = case.model(mode)
    assert_rows(model.forward(ids).logits, case.want(ids), mode)
    cache = model.new_kv_cache(1)
    rows = run_portions(model, cache, 0, [ids[:90], ids[90:150]] + [[t] for t in ids[150:]])  # two portions, then decode steps
    assert_rows(rows, case.want(ids), mode)


@pytest.mark.parametrize("mode", MODES)
def test_constants_come_from_the_configuration(mode):
    case = Case(so.config(61, 48, [so.att(2, 1, 8, 8, 9, 2, base=12.5), so.delta(2, 2, 8, 8, 2), so.latent(2, 8, 8, 8, 8, ff=16)], eps=0.3,
                          embed_scale=0.25), 4)
    ids = case.ids(40)
    assert_rows(case.model(mode).forward(ids).logits, case.want(ids), mode)


# ------------------------------------------------------------------ prompts, decoding, portions
@pytest.mark.parametrize("mode", MODES)
def test_token_by_token_equals_prompt(mixed, mode):
    ids = mixed.ids(130)
    model = mixed.model(mode)
    cache = model.new_kv_cache(1)
    assert_rows(run_portions(model, cache, 0, [[t] for t in ids]), mixed.want(ids), mode)
    assert cache.seq_len == 130


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("sizes", [[2], [3, 1], [23], [22, 24, 1], [64], [40, 2, 7, 1, 1, 31], [129], [12, 13, 14, 15, 18, 23, 29, 30, 46]])
def test_portions(mixed, mode, sizes):
    ids = mixed.ids(200, 1)
    model = mixed.model(mode)
    cache = model.new_kv_cache(1)
    assert_rows(run_portions(model, cache, 0, cut(ids, sizes)), mixed.want(ids), mode)


@pytest.mark.parametrize("mode", MODES)
def test_long_prompt_in_segments_and_long_decoding(mixed, mode):
    """Past the length from which a portion's recurrences run in segments, from an empty and from a filled state, then
    far enough in single tokens that every window and every page of one is used again."""
    ids = mixed.ids(1500, 2)
    model = mixed.model(mode)
    cache = model.new_kv_cache(1)
    got = run_portions(model, cache, 0, [ids[:650], ids[650:1280]] + [[t] for t in ids[1280:]])
    assert_rows(got, mixed.want(ids), mode)


@pytest.mark.parametrize("page_tokens", [16, 64])
def test_page_sizes(mixed, page_tokens):
    ids = mixed.ids(120, 3)
    model = mixed.model("fp32", page_tokens=page_tokens)
    cache = model.new_kv_cache(1)
    assert_rows(run_portions(model, cache, 0, [ids[:37]] + [[t] for t in ids[37:]]), mixed.want(ids), "fp32")


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("splits", [1, 2, 5, 16])
def test_split_decode_attention(mixed, mode, splits):
    """The keys of a step cut over several blocks, down to parts without any."""
    ids = mixed.ids(60, 4)
    model = mixed.model(mode, attn_splits=splits)
    cache = model.new_kv_cache(1)
    assert_rows(run_portions(model, cache, 0, [[t] for t in ids]), mixed.want(ids), mode)


def test_launch_paths_agree(mixed):
    """The step as a CUDA graph and kernel by kernel."""
    ids = mixed.ids(40, 4)
    for graphs in (True, False):
        model = mixed.model("bf16", use_graphs=graphs)
        cache = model.new_kv_cache(1)
        assert_rows(run_portions(model, cache, 0, [ids[:20]] + [[t] for t in ids[20:]]), mixed.want(ids), "bf16")


# ------------------------------------------------------------------ batches, slots, pages
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("batch", [2, 3, 8, 13, 70])
def test_batches_of_unequal_prompts(mixed, mode, batch):
    """Prompts of different lengths at once, then steps of all of them, against each sequence alone."""
    steps, model = 4, mixed.model(mode)
    kinds = [mixed.ids(n, 40 + i) for i, n in enumerate((1, 29, 46, 7, 88))]
    seqs = [kinds[i % len(kinds)] for i in range(batch)]
    cache = model.new_kv_cache(batch)
    heads = [s[:max(1, len(s) - steps)] for s in seqs]
    logits, am = model.prefill_batch(heads, cache, want_logits=True)
    assert_rows(logits, np.stack([mixed.want(s)[len(h) - 1] for s, h in zip(seqs, heads)]), mode)
    assert (am == logits.argmax(axis=1)).all()
    feed = [mixed.ids(steps, 60 + i % len(kinds)) for i in range(batch)]
    for t in range(steps):
        got, am, tv, ti = model.forward_one_batch([f[t] for f in feed], cache, want_logits=True, top_k=5)
        want = np.stack([mixed.want(np.concatenate([h, f[:t + 1]]))[-1] for h, f in zip(heads, feed)])
        assert_rows(got, want, mode)
        assert (am == got.argmax(axis=1)).all() and (ti[:, 0] == am).all() and np.allclose(tv[:, 0], got.max(axis=1))


@pytest.mark.parametrize("mode", MODES)
def test_mixed_portions_and_reused_slots(mixed, mode):
    """Sequences that start, grow and end at different times in one cache: portions of several sizes and single tokens in
    the same pass, slots out of order, slots and pages given back and taken again."""
    model = mixed.model(mode)
    rng = np.random.default_rng(9)
    cache = model.new_kv_cache(4)
    free, live, started, checked = [2, 0, 3, 1], {}, 0, 0
    for _ in range(40):
        while free and started < 9:
            live[free.pop()] = (mixed.ids(int(rng.integers(3, 120)), 100 + started), 0)
            started += 1
        if not live:
            break
        slots = [int(s) for s in rng.permutation(list(live))[:int(rng.integers(1, len(live) + 1))]]
        portions = []
        for s in slots:
            ids, at = live[s]
            portions.append(ids[at:at + int(rng.choice([1, 2, 5, 17, 60]))])
        rows = model.extend(slots, portions, cache, range(sum(len(p) for p in portions)))
        base = 0
        for s, p in zip(slots, portions):
            ids, at = live[s]
            assert_rows(rows[base:base + len(p)], mixed.want(ids)[at:at + len(p)], mode)
            base, checked = base + len(p), checked + len(p)
            live[s] = (ids, at + len(p))
            if at + len(p) == len(ids):
                cache.clear_slot(s)
                free.append(s)
                del live[s]
    assert checked > 300 and started == 9


def test_a_full_context(mixed):
    """A cache no longer than the windows, filled to its end."""
    for context in (20, 64):
        model = mixed.model("fp32", max_context=context)
        cache = model.new_kv_cache(1)
        ids = mixed.ids(context, 7)
        assert_rows(run_portions(model, cache, 0, [ids[:context - 9]] + [[t] for t in ids[context - 9:]]), mixed.want(ids), "fp32")
        with pytest.raises(pg.DesignError, match="cache is full|exceeds n_positions"):
            model.forward_one(1, cache)


def test_first_tokens(mixed):
    for mode in MODES:
        model = mixed.model(mode)
        cache = model.new_kv_cache(1)
        for n in (1, 2, 3, 5, 6):
            ids = mixed.ids(n, 70 + n)
            assert_rows(model.forward(ids).logits, mixed.want(ids), mode)
            cache.clear()
            assert_rows(run_portions(model, cache, 0, [[t] for t in ids]), mixed.want(ids), mode)


def test_a_dirty_slot_starts_from_nothing(mixed):
    """States, convolution inputs and pages that earlier sequences left are not read by a new one."""
    model = mixed.model("fp32")
    cache = model.new_kv_cache(2)
    for first_step in (False, True):
        model.prefill_batch([mixed.ids(90, 80), mixed.ids(50, 81)], cache)
        cache.clear_slot(0)
        ids = mixed.ids(30, 82)
        assert_rows(run_portions(model, cache, 0, [[t] for t in ids] if first_step else [ids]), mixed.want(ids), "fp32")
        more = mixed.ids(2, 83)
        got = model.extend([1], [more], cache, [1])  # the neighbour is untouched
        assert_rows(got, mixed.want(np.concatenate([mixed.ids(50, 81), more]))[[-1]], "fp32")
        cache.clear()


# ------------------------------------------------------------------ what random weights would hide
def sharp_case(size, keep):
    """One attention layer whose scores single out one key: the query of token 1 matches the key of token 0 and no other (in
    an entry that is not rotated), with a score far above the rest."""
    cfg = so.config(31, 32, [so.att(2, 1, 16, 16, size, keep, dims=4, scale=0.25)], embed_scale=1.0)

    def edit(w):
        w["embed"][0] = w["embed"][1] = 0
        w["embed"][0, 4], w["embed"][1, 5] = 6, 6
        w["l0.norm1"][:] = w["final.norm"][:] = 1
        p = "l0.mix."
        for n in ("q", "k"):
            w[p + n] *= 0.1
            w[p + n + ".b"] *= 0.1
        w[p + "talk"][:] = np.eye(2)
        w[p + "q"][[8, 24], 5] = 4                          # token 1 asks with entry 8 of both heads ...
        w[p + "k"][8, 4] = 4                                # ... and token 0 answers with it
        w[p + "o"] *= 3
    return Case(cfg, 8, edit=edit)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("size, keep", [(32, 0), (33, 4), (20, 33), (70, 7), (130, 3)])
def test_the_matching_key_at_the_edges(mode, size, keep):
    """The matching key just inside and just outside the window and among the kept first tokens, at page borders and far
    away; asked from a prompt, from a portion that starts between the two, and from a decode step."""
    case = sharp_case(size, keep)
    model = case.model(mode)
    far = 3 * size + 40
    for key, ask in [(60, 60 + size - 1), (60, 60 + size), (60, 60 + size + 1), (31, 31 + size - 1), (32, 32 + size), (0, far), (max(keep - 1, 0), far),
                     (keep, keep + size - 1), (keep, keep + size), (keep, far), (keep + 1, far), (0, 1), (far - 1, far)]:
        ids = 2 + case.ids(max(ask, far) + 3) % 29
        ids[key], ids[ask] = 0, 1
        want = case.want(ids)
        # the inputs tell right from wrong: a key that is seen decides the asking token's logits, another does not touch them
        other = ids.copy()
        other[key] = 2
        moved = row_errors(so.forward(case.cfg, case.w, other), want)[ask]
        assert moved > 0.13 if ask - key < size or key < keep else moved < 1e-9, (key, ask, moved)

        def check(rows):
            assert_rows(rows, want, mode, 2.5 if mode == "bf16" else 1.0)
            assert row_errors(rows, want)[ask] <= BOUND[mode]

        check(model.forward(ids).logits)
        cache = model.new_kv_cache(1)
        first = [ids[:ask - 1]] if ask > 1 else []
        check(run_portions(model, cache, 0, first + [ids[max(ask - 1, 0):ask + 1], ids[ask + 1:]]))
        cache.clear()
        check(run_portions(model, cache, 0, [ids[:ask]] + [[t] for t in ids[ask:]]))


@pytest.mark.parametrize("mode", MODES)
def test_a_far_key_among_hundreds_of_latent_rows(mode):
    """Latent attention that singles out one key, asked from a prompt, a short portion and a decode step."""
    cfg = so.config(31, 32, [so.latent(2, 16, 16, 16, 16, scale=0.25)], embed_scale=1.0)

    def edit(w):
        w["embed"][0] = w["embed"][1] = 0
        w["embed"][0, 4], w["embed"][1, 5] = 6, 6
        p = "l0.mix."
        for n in ("l0.norm1", "final.norm", p + "dq.norm", p + "dkv.norm"):
            w[n][:] = 1
        for n in ("dq", "dkv"):
            w[p + n] *= 0.3
        w[p + "uq"] *= 0.1
        w[p + "uk"] *= 0.1
        w[p + "dq"][:, 5] = w[p + "dkv"][:, 4] = 0
        w[p + "dq"][3, 5] = w[p + "dkv"][7, 4] = 1
        w[p + "uq"][[2, 18], 3] = 4
        w[p + "uk"][[2, 18], 7] = 4
        w[p + "o"] *= 3
    case = Case(cfg, 9, edit=edit)
    model = case.model(mode)
    for key, ask in [(0, 700), (255, 256), (31, 640), (32, 383), (500, 703)]:
        ids = 2 + case.ids(705) % 29
        ids[key], ids[ask] = 0, 1
        want = case.want(ids)
        other = ids.copy()
        other[key] = 2
        assert row_errors(so.forward(case.cfg, case.w, other), want)[ask] > 0.13
        cache = model.new_kv_cache(1)
        for rows in (model.forward(ids).logits, run_portions(model, cache, 0, [ids[:ask - 1], ids[ask - 1:ask + 1], ids[ask + 1:]])):
            assert_rows(rows, want, mode, 2.5 if mode == "bf16" else 1.0)
            assert row_errors(rows, want)[ask] <= BOUND[mode]
        cache.clear()
        rows = run_portions(model, cache, 0, [ids[:ask]] + [[t] for t in ids[ask:]])
        assert row_errors(rows, want)[ask] <= BOUND[mode]


@pytest.mark.parametrize("mode", MODES)
def test_a_large_sink_and_a_large_score(mode):
    """Sinks far above and far below every score, and scores of several hundred."""
    for sink, scale in ((12.0, 0.25), (-30.0, 0.25), (0.0, 30.0), (60.0, -30.0)):
        case = Case(so.config(61, 48, [so.att(4, 2, 16, 8, 21, 3, scale=scale)]), 5,
                    edit=lambda w: w.update({"l0.mix.sink": np.array([sink, 0, sink, 1], np.float32)}))
        ids = case.ids(70)
        factor = 8.0 if abs(scale) > 1 else 1.0  # the rounding of a score grows with it
        model = case.model(mode)
        assert_rows(model.forward(ids).logits, case.want(ids), mode, factor)
        cache = model.new_kv_cache(1)
        assert_rows(run_portions(model, cache, 0, [ids[:40]] + [[t] for t in ids[40:]]), case.want(ids), mode, factor)


# ------------------------------------------------------------------ generation through the usual entry points
@pytest.fixture(scope="module")
def greedy(mixed):
    prompts = [mixed.ids(n, 200 + n) for n in (5, 21, 40)]
    return [(p, *cases.greedy(mixed, p, 30)) for p in prompts]


@pytest.mark.parametrize("mode", MODES)
def test_greedy_generation(mixed, greedy, mode):
    model, bound = mixed.model(mode), BOUND[mode]
    for prompt, want, gaps in greedy:
        n = len(prompt)
        assert_stream(model.stream_greedy_tokens(prompt, 30, lambda t: None), want, gaps, n, bound)
        assert_stream(pg.generate(model, prompt, 30), want, gaps, n, bound)
        out, stats = model.generate_with_config(prompt, pg.TextGenerationConfig(30))
        assert_stream(list(prompt) + out, want, gaps, n, bound)
        assert stats.generated_tokens == 30
        cache = model.new_kv_cache(1)
        _, first = model.prefill_batch([prompt], cache)
        toks = model.decode_greedy(first, cache, 29)
        assert_stream(list(prompt) + [int(first[0])] + [int(t) for t in toks[:, 0]], want, gaps, n, bound)
    batch = model.generate_batch([p for p, _, _ in greedy], pg.TextGenerationConfig(30))
    for out, (prompt, want, gaps) in zip(batch, greedy):
        assert_stream(list(prompt) + out, want, gaps, len(prompt), bound)


def test_command_line_with_token_ids(mixed, greedy):
    from puppygrad_b200 import runtime
    prompt, want, gaps = greedy[1]
    out, err = io.StringIO(), io.StringIO()
    rc = runtime.run_gpt2(["--model-dir", mixed.dir, "--prompt-ids", ",".join(str(t) for t in prompt), "--max-new-tokens", "12",
                           "--math-mode", "fp32", "--stats"], out, err)
    assert rc == 0 and "loading Sanesun" in err.getvalue() and "decode:" in err.getvalue()
    got = [int(t) for t in out.getvalue().split()]
    assert_stream(list(prompt) + got, want[:len(prompt) + 12], gaps, len(prompt), BOUND["fp32"])


def test_trace_replay_on_the_device(mixed):
    replay = trace.TraceReplay(mixed.model("fp32"), 2)
    a, b = mixed.ids(40, 400), mixed.ids(33, 401)
    got = replay.step([{"id": "a", "tokens": a[:20].tolist(), "want": [0, 19]}], [])
    assert_rows(got, mixed.want(a)[[0, 19]], "fp32")
    got = replay.step([{"id": "b", "tokens": b.tolist(), "want": [32]}, {"id": "a", "tokens": a[20:39].tolist(), "want": [18]}], ["b"])
    assert_rows(got, np.stack([mixed.want(b)[32], mixed.want(a)[38]]), "fp32")
    got = replay.step([{"id": "a", "tokens": [int(a[39])], "want": [0]}], ["a"])
    assert_rows(got, mixed.want(a)[[39]], "fp32")


def test_profiles_and_sizes(mixed):
    model = mixed.model("bf16")
    cache = model.new_kv_cache(2)
    prof = model.profile_prefill([mixed.ids(50), mixed.ids(9, 1)], cache)
    assert all(prof[k][0] > 0 for k in ("layer_norm", "qkv_projection", "attention", "attention_projection", "final_logits"))
    n0 = cache.kernel_launches()
    step = model.profile_forward_one([1, 2], cache)
    assert sum(n for _, n in step.values()) == cache.kernel_launches() - n0
    up4 = lambda n: -(-n // 4) * 4
    want = 0
    for l in MIXED["layers"]:
        m = l["mixer"]
        if l["type"] == "channel_delta":
            channels = 2 * up4(m["kv_heads"] * m["dim"]) + up4(m["heads"] * m["vdim"])
            want += 4 * (m["heads"] * m["dim"] * up4(m["vdim"]) + m["conv"] * channels)
    assert model.state_bytes_per_sequence() == want


# ------------------------------------------------------------------ sizes past one tile of every product
@pytest.fixture(scope="module")
def wide():
    return Case(so.config(500, 1100, [so.delta(10, 5, 40, 72, 4, ff=7000), so.att(10, 2, 72, 80, 90, 6, ff=300), so.latent(9, 72, 80, 136, 260, ff=520)]),
                21, rank=33)


@pytest.mark.parametrize("mode", MODES)
def test_wide_layers(wide, mode):
    """Several tiles and k blocks of the products, rows too long for the eight-row kernel's shared memory."""
    model = wide.model(mode)
    ids = wide.ids(300)
    assert_rows(model.forward(ids).logits, wide.want(ids), mode)
    for batch in (1, 3, 8, 40):
        cache = model.new_kv_cache(batch)
        prompts = [ids[:100 + 3 * (i % 4)] for i in range(batch)]
        model.prefill_batch(prompts, cache)
        for t in range(2):
            got, _, _, _ = model.forward_one_batch([ids[len(p) + t] for p in prompts], cache, want_logits=True)
            assert_rows(got, np.stack([wide.want(ids)[len(p) + t] for p in prompts]), mode)
