"""GPU tests of the layered models against the plain FP64 restatement (layered_oracle.py): each mechanism alone, prompts
against decoding, portions, batches, reuse of pages and slots, edges of blocks and pages, generation.

A row of logits is compared by the root mean square of its difference (mean removed) over the spread of the expected
logits: FP32 within 3e-5, BF16 (weights exact, product inputs and cached keys rounded) within 4e-2."""
import io

import numpy as np
import pytest

import puppygrad_b200 as pg
from puppygrad_b200 import trace
from tests import layered_cases as cases
from tests import layered_oracle as lo
from tests.layered_cases import BOUND, MODES, assert_rows, assert_stream, cut, row_errors, run_portions

pytestmark = pytest.mark.gpu


def Case(cfg, seed, **kw):
    return cases.Case(lo, cfg, seed, **kw)


MIXED = lo.config(101, 72, [lo.gla(3, 12, 20, tau=9.0, ff=40), lo.pair(6, 2, 20, 12, 23, 5, 16, left_scale=0.7, right_scale=1.3),
                            lo.gla(2, 32, 16), lo.pair(4, 4, 8, 24, 40, 2, 32, ff=88)])


@pytest.fixture(scope="module")
def mixed():
    return Case(MIXED, 11)


# ------------------------------------------------------------------ each mechanism alone
ALONE = {
    "gla": lo.config(67, 48, [lo.gla(4, 16, 24)]),
    "gla-odd": lo.config(59, 50, [lo.gla(3, 7, 9, tau=2.5)]),
    "gla-128": lo.config(67, 64, [lo.gla(2, 128, 128)]),
    "gla-256": lo.config(67, 64, [lo.gla(1, 200, 256)]),
    "gla-narrow-keys": lo.config(67, 64, [lo.gla(2, 4, 96)]),
    "attention": lo.config(67, 48, [lo.pair(6, 2, 16, 24, 21, 1, 4, right_scale=0.0)]),
    "attention-odd": lo.config(59, 50, [lo.pair(9, 3, 7, 11, 13, 1, 4, right_scale=0.0)]),
    "attention-wide": lo.config(67, 64, [lo.pair(7, 1, 136, 72, 50, 1, 4, right_scale=0.0)]),
    "attention-256": lo.config(67, 64, [lo.pair(2, 2, 256, 256, 37, 1, 4, right_scale=0.0)]),
    "attention-one": lo.config(67, 48, [lo.pair(4, 4, 16, 8, 1, 1, 4, right_scale=0.0)]),
    "delta": lo.config(67, 48, [lo.pair(1, 1, 8, 8, 5, 4, 16, left_scale=0.0)]),
    "delta-odd": lo.config(59, 50, [lo.pair(1, 1, 8, 8, 5, 3, 9, left_scale=0.0)]),
    "delta-128": lo.config(67, 64, [lo.pair(1, 1, 8, 8, 5, 2, 128, left_scale=0.0)]),
    "delta-72": lo.config(67, 64, [lo.pair(1, 1, 8, 8, 5, 2, 72, left_scale=0.0)]),
    "feed-forward": lo.config(67, 48, [lo.gla(1, 4, 4, ff=136)]),
    "eps": lo.config(67, 48, [lo.gla(2, 8, 8), lo.pair(2, 1, 8, 8, 9, 2, 8, ff=16)], eps=0.3),
}


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("name", ALONE)
def test_mechanism_alone(name, mode):
    case = Case(ALONE[name], 3, rank=3 if "odd" in name else 16)
    ids = case.ids(83)
    model = case.model(mode)
    assert_rows(model.forward(ids).logits, case.want(ids), mode)
    cache = model.new_kv_cache(1)
    rows = run_portions(model, cache, 0, [ids[:60]] + [[t] for t in ids[60:]])  # a prompt, then decode steps
    assert_rows(rows, case.want(ids), mode)


def test_full_causal_attention_without_a_mask():
    cfg = lo.config(67, 48, [lo.pair(4, 2, 16, 16, 5, 2, 8)])
    cfg["layers"][0]["mixer"]["left"]["mask"] = None
    case = Case(cfg, 5)
    ids = case.ids(150)
    model = case.model("fp32", max_context=160)
    cache = model.new_kv_cache(1)
    assert_rows(run_portions(model, cache, 0, [ids[:70], ids[70:140]] + [[t] for t in ids[140:]]), case.want(ids), "fp32")


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
    far enough in single tokens that every block of keys and every page is used again."""
    ids = mixed.ids(1500, 2)
    model = mixed.model(mode)
    cache = model.new_kv_cache(1)
    want = mixed.want(ids)
    got = run_portions(model, cache, 0, [ids[:650], ids[650:1280]] + [[t] for t in ids[1280:]])
    assert_rows(got, want, mode)


@pytest.mark.parametrize("page_tokens", [16, 64])
def test_page_sizes(mixed, page_tokens):
    ids = mixed.ids(90, 3)
    model = mixed.model("fp32", page_tokens=page_tokens)
    cache = model.new_kv_cache(1)
    assert_rows(run_portions(model, cache, 0, [ids[:37]] + [[t] for t in ids[37:]]), mixed.want(ids), "fp32")


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("splits", [2, 5])
def test_split_decode_attention(mode, splits):
    case = Case(lo.config(67, 48, [lo.pair(6, 2, 16, 24, 300, 2, 8)]), 4)
    ids = case.ids(330)
    model = case.model(mode, attn_splits=splits)
    cache = model.new_kv_cache(1)
    assert_rows(run_portions(model, cache, 0, [ids[:260]] + [[t] for t in ids[260:]]), case.want(ids), mode)


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
    for step in range(40):
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


def test_wanted_rows_and_bad_requests(mixed):
    model = mixed.model("fp32")
    cache = model.new_kv_cache(2)
    ids = mixed.ids(30, 5)
    got = model.extend([1], [ids], cache, [29, 3, 3])
    assert_rows(got, mixed.want(ids)[[29, 3, 3]], "fp32")
    assert cache.seq_len_of(1) == 30 and cache.seq_len_of(0) == 0
    for call, message in [(lambda: model.extend([0, 0], [[1], [2]], cache), "appears twice"),
                          (lambda: model.extend([5], [[1]], cache), "slot out of range"),
                          (lambda: model.extend([0], [[101]], cache), "exceeds vocab_size 101"),
                          (lambda: model.extend([0], [[1]], cache, [1]), "outside the portion"),
                          (lambda: model.extend([1], [mixed.ids(4090)], cache), "exceeds n_positions")]:
        with pytest.raises(pg.DesignError, match=message):
            call()
    assert_rows(model.extend([1], [mixed.ids(3, 6)], cache, [2]), mixed.want(np.concatenate([ids, mixed.ids(3, 6)]))[[-1]], "fp32")


def test_a_full_context_is_refused(mixed):
    model = mixed.model("fp32", max_context=20)
    cache = model.new_kv_cache(1)
    ids = mixed.ids(20, 7)
    assert model.max_context_len() == 20
    assert_rows(run_portions(model, cache, 0, [ids[:19], ids[19:]]), mixed.want(ids), "fp32")
    with pytest.raises(pg.DesignError, match="cache is full|exceeds n_positions"):
        model.forward_one(1, cache)
    assert len(model.generate_greedy_cached(ids[:15], 50)) == 20


# ------------------------------------------------------------------ what random weights would hide
def sharp_case(size):
    """Attention whose scores single out one key: the query of token 1 matches the key of token 0 and no other, with a
    score far above the rest; token 0's value is large."""
    cfg = lo.config(31, 32, [lo.pair(2, 1, 16, 16, size, 1, 4, scale=2.0, right_scale=0.0)])

    def edit(w):
        w["embed"][0] = w["embed"][1] = 0
        w["embed"][0, 4], w["embed"][1, 5] = 24, 24      # two clean directions, well above the position vector
        w["embed"][2:] *= 0.25
        for n in ("l0.norm1", "l0.norm1b", "final.norm"):
            w[n][:], w[n + ".b"][:] = 1, 0
        w["l0.norm1b"][:] = 16                            # what attention brings outweighs the token itself
        q, k = w["l0.mix.left.q"], w["l0.mix.left.k"]
        q *= 0.1
        k *= 0.1
        q[[0, 16], 5] = 4                                 # token 1 asks with channel 0 of both heads ...
        k[0, 4] = 4                                       # ... and token 0 answers with it
    return Case(cfg, 8, edit=edit)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("size", [32, 33, 48, 70])
def test_the_matching_key_at_the_edges_of_a_block(mode, size):
    """The matching key as the first of the asking token's own block, the last of the block before, at page borders, and
    far away; asked from a prompt, from a portion that starts inside the block, and from a decode step."""
    case = sharp_case(size)
    model = case.model(mode)
    for key, ask in [(size, 2 * size - 1), (size - 1, size), (size - 1, 2 * size - 1), (2 * size, 2 * size + 1), (0, size - 1),
                     (31, 32), (size + 15, size + 16), (2 * size - 1, 2 * size + 2)]:
        ids = 2 + case.ids(2 * size + 6) % 29
        ids[key], ids[ask] = 0, 1
        want = case.want(ids)
        # the inputs tell right from wrong: a block one position off moves some logits here far past the bound
        same = key // size == ask // size
        other = ids.copy()
        other[key] = 2
        moved = row_errors(lo.forward(case.cfg, case.w, other), want)[ask]
        assert moved > 0.13 if same else moved < 1e-9

        def check(rows):
            assert_rows(rows, want, mode, 2.5 if mode == "bf16" else 1.0)  # rows with two keys nearly alike are touchy
            assert row_errors(rows, want)[ask] <= BOUND[mode]

        check(model.forward(ids).logits)
        cache = model.new_kv_cache(1)
        check(run_portions(model, cache, 0, [ids[:ask - 1], ids[ask - 1:ask + 1], ids[ask + 1:]]))
        cache.clear()
        check(run_portions(model, cache, 0, [ids[:ask]] + [[t] for t in ids[ask:]]))


def test_planted_mistakes_would_be_seen(mixed):
    """Each deliberate error of the restatement moves the logits of these inputs past the bounds used here."""
    ids = mixed.ids(130)
    want = mixed.want(ids)
    for mistake in ("chunk-1", "chunk+1", "chunk-from-portion", "lost-state", "no-page"):
        wrong = lo.forward(mixed.cfg, mixed.w, ids, mistake=mistake, portion=57)
        assert row_errors(wrong, want).max() > 2 * BOUND["bf16"], mistake


def test_first_tokens(mixed):
    for mode in MODES:
        model = mixed.model(mode)
        cache = model.new_kv_cache(1)
        for n in (1, 2, 3):
            ids = mixed.ids(n, 70 + n)
            assert_rows(model.forward(ids).logits, mixed.want(ids), mode)
            cache.clear()
            assert_rows(run_portions(model, cache, 0, [[t] for t in ids]), mixed.want(ids), mode)


def test_a_dirty_slot_starts_from_nothing(mixed):
    """States and pages that earlier sequences left are not read by a new one, neither by a prompt nor by a first step."""
    model = mixed.model("fp32")
    cache = model.new_kv_cache(2)
    for first_step in (False, True):
        model.prefill_batch([mixed.ids(90, 80), mixed.ids(50, 81)], cache)
        cache.clear_slot(0)
        ids = mixed.ids(30, 82)
        portions = [[t] for t in ids] if first_step else [ids]
        assert_rows(run_portions(model, cache, 0, portions), mixed.want(ids), "fp32")
        more = mixed.ids(2, 83)
        got = model.extend([1], [more], cache, [1])  # the neighbour is untouched
        assert_rows(got, mixed.want(np.concatenate([mixed.ids(50, 81), more]))[[-1]], "fp32")
        cache.clear()


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
        seen = []
        assert_stream(model.stream_greedy_tokens(prompt, 30, lambda t: seen.append(t)), want, gaps, n, bound)
        assert len(seen) == 30
        assert_stream(pg.generate(model, prompt, 30), want, gaps, n, bound)
        assert_stream(model.generate_greedy(prompt, 30), want, gaps, n, bound)
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


def test_sampled_generation_is_reproducible_and_stops_at_eos(mixed):
    model = mixed.model("bf16")
    conf = pg.TextGenerationConfig(25, temperature=0.9, top_k=12, seed=5)
    prompts = [mixed.ids(9, 300), mixed.ids(17, 301)]
    a, b = model.generate_batch(prompts, conf), model.generate_batch(prompts, conf)
    assert a == b and all(len(x) == 25 for x in a)
    alone, _ = model.generate_with_config(prompts[0], conf)
    assert alone == a[0]
    eos = a[0][7]
    stopped, _ = model.generate_with_config(prompts[0], pg.TextGenerationConfig(25, temperature=0.9, top_k=12, seed=5, eos_token_id=eos))
    assert stopped == a[0][:a[0].index(eos)]


def test_command_line_with_token_ids(mixed, greedy):
    from puppygrad_b200 import runtime
    prompt, want, gaps = greedy[1]
    out, err = io.StringIO(), io.StringIO()
    rc = runtime.run_gpt2(["--model-dir", mixed.dir, "--prompt-ids", ",".join(str(t) for t in prompt), "--max-new-tokens", "12",
                           "--math-mode", "fp32", "--stats"], out, err)
    assert rc == 0 and "loading Dirurax" in err.getvalue() and "decode:" in err.getvalue()
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
    assert all(prof[k][0] > 0 for k in ("layer_norm", "qkv_projection", "attention", "attention_projection", "mlp_fc_projection", "final_logits"))
    n0 = cache.kernel_launches()
    step = model.profile_forward_one([1, 2], cache)
    assert sum(n for _, n in step.values()) == cache.kernel_launches() - n0
    assert cache.seq_len_of(0) == 51 and cache.seq_len_of(1) == 10
    want = sum(l["mixer"]["heads"] * l["mixer"]["dim"] * -(-l["mixer"]["vdim"] // 4) * 16 if l["type"] == "gla" else
               l["mixer"]["right"]["heads"] * l["mixer"]["right"]["dim"] ** 2 * 4 for l in MIXED["layers"])
    assert model.state_bytes_per_sequence() == want
    assert model.weight_bytes_per_step() > 0


# ------------------------------------------------------------------ sizes past one tile of every product
@pytest.fixture(scope="module")
def wide():
    return Case(lo.config(500, 1100, [lo.gla(3, 40, 72, ff=7000), lo.pair(10, 2, 72, 80, 90, 5, 40, ff=300)]), 21, rank=33)


@pytest.mark.parametrize("mode", MODES)
def test_wide_layers(wide, mode):
    """Several tiles and k blocks of the products, a hidden row too long for the eight-row kernel's shared memory."""
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
