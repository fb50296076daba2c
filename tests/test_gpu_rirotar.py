"""Rirotar models on a GPU against the plain implementation: prompts, decoding, portions, mixed batches, pages and slots used
again, keys at window borders, far writes to a state, sinks, long decoding, greedy generation through the scheduler and the
command line tools."""
import json

import numpy as np
import pytest

import plain_rirotar as plain
import rirotar_cases as rc
from test_gpu_vuzunex import run_tool

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


class Loaded:
    def __init__(self, pkg, name, cfg, dtype, seed=5, sharpen=1.0, **runtime):
        self.name, self.cfg, self.dtype = name, cfg, dtype
        self.bits, self.weights = rc.random_weights(name, cfg, seed, sharpen)
        self.store = pkg.WeightStore(0)
        self.builder = rc.builder_of(pkg, name, cfg, dtype, **runtime)
        self.model = pkg.load_model(self.store, self.builder, self.bits)

    def tokens(self, n, seed=0):
        return np.random.default_rng(seed + 77).integers(0, self.cfg["vocab"], size=n).tolist()

    def plain(self, tokens):
        return plain.forward(self.cfg, self.weights, tokens)[0]

    def portions(self, seq, tokens, sizes):
        """Logits of every token, fed in portions of the given sizes (the last one repeated)."""
        out, at, i = [], 0, 0
        while at < len(tokens):
            n = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
            out.append(self.model.run_batch([(seq, tokens[at:at + n], list(range(n)))])[0])
            at, i = at + n, i + 1
        return np.concatenate(out)

    def agree(self, got, want, slack=1.0):
        rc.agree(got, want, self.cfg, self.dtype, slack)

    def close(self):
        self.model.close()
        self.store.close()


@pytest.fixture
def load(pkg):
    made = []

    def make(name, dtype, cfg=None, **kw):
        made.append(Loaded(pkg, name, cfg or rc.cases()[name], dtype, **kw))
        return made[-1]

    yield make
    for m in made:
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(rc.cases()))
def test_prompt_portions_and_decoding_agree_with_the_plain_model(load, dtype, name):
    m = load(name, dtype)
    tokens = m.tokens(150)
    want = m.plain(tokens)
    m.agree(m.portions(0, tokens, [150]), want)
    m.model.reset_sequence(0)
    m.agree(m.portions(0, tokens, [1]), want)
    for seq, sizes in enumerate(([2], [64, 2, 63, 3, 65], [5, 64, 1, 80], [100, 1])):
        if seq == 0:
            m.model.reset_sequence(0)
        m.agree(m.portions(seq, tokens, sizes), want)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mid", "odd", "state_only"])
def test_residual_stream_after_every_layer(pkg, load, dtype, name):
    m = load(name, dtype)
    tokens = m.tokens(90)
    _, after = plain.forward(m.cfg, m.weights, tokens)
    for n in range(1, len(m.cfg["layers"]) + 1):
        part = pkg.rirotar.dataclasses.replace(m.builder.config, layers=m.builder.config.layers[:n])
        model = pkg.InferenceModel(m.store, pkg.RirotarPlanBuilder(part).decode_steps(store_final=True), part.buffers_desc())
        for rows in (90, 3, 1):
            model.run_batch([(0, tokens[:rows], list(range(rows)))])
            got = model.read_buffer_f32(pkg.plan.BUF_RESIDUAL, rows, m.cfg["width"])
            err = np.abs(got - after[n - 1][:rows]).max(axis=1) / np.abs(after[n - 1]).max()
            # (in bf16 an expert with an all but equal score may be another: the bulk of the rows counts)
            assert (err.max() if dtype == "float32" else np.quantile(err, 0.7)) <= (1e-5 if dtype == "float32" else 3e-2)
            model.reset_sequence(0)
        model.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mid", "odd", "wide", "huge"])
def test_mixed_batches_against_each_request_alone(load, dtype, name):
    m = load(name, dtype, max_batch=4, max_seq=256)
    requests = [m.tokens(n, seed=i) for i, n in enumerate((201, 1, 130, 67))]
    cuts = [[70, 1, 1, 64, 65], [1], [1, 1, 66, 1, 61], [2, 3, 60, 1, 1]]
    alone = []
    for r in requests:
        alone.append(m.portions(0, r, [len(r)]))
        m.model.reset_sequence(0)
    got, at = [[] for _ in requests], [0] * 4
    for step in range(5):
        entries = []
        for i in (2, 0, 3, 1):   # not in the order of the slots
            if step < len(cuts[i]) and at[i] < len(requests[i]):
                n = cuts[i][step]
                entries.append((i, requests[i][at[i]:at[i] + n], list(range(n))))
                at[i] += n
        logits, greedy = m.model.run_batch(entries)
        assert greedy.tolist() == np.argmax(logits, axis=1).tolist()
        row = 0
        for i, part, _ in entries:
            got[i].append(logits[row:row + len(part)])
            row += len(part)
    for i, r in enumerate(requests):
        assert at[i] == len(r)
        g = np.concatenate(got[i])
        m.agree(g, m.plain(r))
        m.agree(g, alone[i].astype(np.float64))
    assert m.model.positions.tolist() == [201, 1, 130, 67]


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_slots_and_states_are_used_again(pkg, load, dtype):
    m = load("mid", dtype, max_batch=3, max_seq=256, pool_tokens=5 * 64)
    model = m.model
    assert model.free_pages == 5
    a, b, c = m.tokens(65, 1), m.tokens(130, 2), m.tokens(60, 3)
    wa, wb, wc = m.plain(a), m.plain(b), m.plain(c)
    m.agree(m.portions(0, a, [40, 1]), wa)
    m.agree(m.portions(1, b, [128, 1]), wb)
    assert model.free_pages == 0
    with pytest.raises(pkg.SwlmError):   # no page left: refused, nothing changed
        model.run_batch([(1, b[:1], [0]), (2, c, [0])])
    assert model.free_pages == 0 and model.positions.tolist() == [65, 130, 0]
    # slots whose states and pages other requests have used; a first token alone and a first portion
    model.reset_sequence(0)
    m.agree(m.portions(2, c, [7, 9]), wc)
    m.agree(m.portions(0, c, [1]), wc)
    model.reset_sequence(1)
    model.reset_sequence(2)
    m.agree(m.portions(1, c, [60]), wc)
    model.reset_state()
    for seq in (2, 0):
        m.agree(m.portions(seq, b[:100], [64, 1]), wb[:100])
    # a request that is left out of steps and goes on
    model.reset_state()
    first = m.portions(1, b[:50], [50])
    m.portions(0, a, [30, 1])
    m.agree(np.concatenate([first, m.portions(1, b[50:], [3, 1, 76])]), wb)
    model.reset_state()
    assert model.free_pages == 5
    lg, _ = model.run_batch([(1, a, [64, 0, 64])])
    m.agree(np.repeat(lg, 3, axis=0), np.repeat(wa[[64, 0, 64]], 3, axis=0))


def edge_model(load, dtype, heads, dim, vdim, rank, window):
    """One layer of latent attention with sharpened queries: a row's result hangs on few keys."""
    cfg = rc.config(256, 128, [rc.latent(heads, dim, vdim, rank, window, None)], cap=50.0)
    return load("edge", dtype, cfg=cfg, sharpen=3.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, vdim, rank, window", [(4, 32, 24, 48, 40), (3, 24, 40, 72, 64), (5, 13, 7, 33, 65), (2, 32, 32, 64, 100)])
def test_keys_just_inside_and_just_outside_the_window(load, dtype, heads, dim, vdim, rank, window):
    m = edge_model(load, dtype, heads, dim, vdim, rank, window)
    tokens = m.tokens(200, seed=9)
    want = m.plain(tokens)
    limit = {"float32": 5e-5, "bfloat16": 3e-2}[dtype]
    for sizes in ([200], [64, 65, 1], [1], [127, 2, 1], [window, window - 1, 2]):
        err = rc.row_errors(m.portions(0, tokens, sizes), want)
        assert err.max() <= limit, (sizes, int(err.argmax()))
        m.model.reset_sequence(0)
    # the test itself: a window one token longer or shorter, or a sink that is left out, shows
    for other in (window - 1, window + 1):
        cfg = dict(m.cfg, layers=[rc.latent(heads, dim, vdim, rank, other, None)])
        err = rc.row_errors(plain.forward(cfg, m.weights, tokens)[0], want)
        assert err[:min(window, other)].max() < 1e-12 and (err[min(window, other):] > 2.5 * limit).any()
    without = dict(m.weights, **{"l0.mix.sink": np.full(heads, -1e30)})
    assert (rc.row_errors(plain.forward(m.cfg, without, tokens)[0], want) > 2.5 * limit).mean() > 0.2


def far_write_weights(weights, eps):
    """Token 299 alone writes to the state, token 298 asks for what it wrote, and nothing is forgotten: q of 298 is k of 299
    (opposite embeddings, opposite projections), and a component that all embeddings share keeps everyone else's step size at
    zero."""
    w = {k: v.copy() for k, v in weights.items()}
    w["embed"][:, 0] = 3.0
    w["embed"][298] = -w["embed"][299]
    h = plain.rms_norm(w["embed"], w["l0.norm1"], eps, 1.0)
    w["l0.mix.b"] = np.tile(20.0 * h[299] / (h[299] @ h[299]), (w["l0.mix.b"].shape[0], 1))
    w["l0.mix.b"][:, 0] -= 10.0 / h[:298, 0].mean()
    w["l0.mix.q"] = -w["l0.mix.k"]
    for t in "qk":
        w[f"l0.mix.{t}.conv"][:, -1], w[f"l0.mix.{t}.conv"][:, :-1] = 1.0, 0.0
    w["l0.mix.A_log"][:] = -9.0
    w["l0.mix.norm"] *= 4.0
    bits = {k: rc.to_bf16_bits(v) for k, v in w.items()}
    return bits, {k: rc.from_bf16_bits(v) for k, v in bits.items()}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channel", [True, False])
def test_a_far_write_is_found_again(pkg, load, dtype, channel):
    layer = rc.delta(2, 1, 64, 48, None, conv=2, channel=channel)
    m = load("far", dtype, cfg=rc.config(300, 96, [layer], cap=60.0), max_seq=640)
    m.bits, m.weights = far_write_weights(m.weights, m.cfg["norm"]["eps"])
    pkg.upload_weights(m.store, m.builder, m.bits)
    tokens = np.random.default_rng(3).integers(0, 298, size=500)
    tokens[499] = 298
    for where in (0, 3, 250):
        t = tokens.copy()
        t[where] = 299
        want, absent = m.plain(t), m.plain(tokens)
        assert rc.row_errors(absent[499:], want[499:])[0] > 0.2
        for sizes in ([500], [499, 1], [300, 198, 2], [3, 1]):
            got = m.portions(0, t.tolist(), sizes)
            assert rc.row_errors(got[499:], want[499:])[0] <= (1e-4 if dtype == "float32" else 5e-2), (where, sizes)
            m.model.reset_sequence(0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_of_a_sequence(load, dtype):
    """Convolutions and windows that reach beyond the start."""
    m = load("odd", dtype)
    for n in (1, 2, 3, 5, 6, 7):
        tokens = m.tokens(n, seed=n)
        want = m.plain(tokens)
        for sizes in ([n], [1], [1, 2], [2, 1]):
            got = m.portions(n % 4, tokens, sizes)
            m.model.reset_sequence(n % 4)
            if dtype == "float32":
                m.agree(got, want)
            else:
                assert np.median(rc.row_errors(got, want)) <= 5e-2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch", [1, 3, 9])
def test_long_greedy_decoding_through_the_decode_graph(load, dtype, batch):
    m = load("mid", dtype, max_batch=batch, max_seq=320)
    prompt = np.array([m.tokens(5, seed=i) for i in range(batch)], dtype=np.int32)
    first = m.model.prefill(prompt)
    tokens = np.concatenate([first[None], m.model.decode_n(first, 290)])
    assert m.model.positions.tolist() == [295] * batch
    for b in range(min(batch, 3)):
        seq = prompt[b].tolist() + tokens[:, b].tolist()
        logits = m.plain(seq)[4:-1]
        top = logits.max(axis=1)
        chosen = logits[np.arange(291), tokens[:, b]]
        # the device's choice is the plain model's, or as good within rounding
        worse = (top - chosen) / logits.std()
        if dtype == "float32":
            assert worse.max() <= 1e-3 and (chosen == top).mean() >= 0.99
        else:
            assert np.quantile(worse, 0.95) <= 0.2 and (chosen == top).mean() >= 0.8
    again = m.model.decode(tokens[-1])
    lg = m.model.logits()
    assert again.tolist() == np.argmax(lg, axis=1).tolist()
    if dtype == "float32":
        m.agree(lg[:1], m.plain(prompt[0].tolist() + tokens[:, 0].tolist())[-1:])


def test_prompt_chunks_snapshot_and_reset(load):
    m = load("mid", "float32", max_batch=2, max_seq=256)
    model, tokens = m.model, m.tokens(180)
    want = int(np.argmax(m.plain(tokens)[-1]))
    model.set_prefill_chunk(70)
    assert model.prefill_sequence(1, tokens) == want
    snap = model.prompt_snapshot()
    a = model.run_batch([(1, [want], [0])])[0]
    model.reset_state()
    assert model.free_pages == 8 and model.positions.tolist() == [0, 0]
    model.run_batch([(1, tokens[:100], [])])   # other data on the pages and in the state
    model.restore(snap)
    assert model.positions.tolist() == [0, 180]
    assert np.array_equal(a, model.run_batch([(1, [want], [0])])[0])
    model.free_snapshot(snap)


@pytest.mark.parametrize("name, budget", [("mid", 5), ("mid", 48), ("odd", 512)])
def test_greedy_generation_through_the_scheduler(pkg, load, name, budget):
    m = load(name, "float32", max_batch=3, max_seq=256, pool_tokens=6 * 64)
    sched = pkg.BatchScheduler(m.model, row_budget=budget)
    requests = [pkg.Request(i, m.tokens(n, seed=20 + i), k) for i, (n, k) in enumerate([(3, 6), (100, 4), (64, 5), (1, 8), (30, 3)])]
    for r in requests:
        sched.submit(r)
    sched.run()
    assert m.model.free_pages == 6
    for r in requests:
        tokens, margins = plain.greedy(m.cfg, m.weights, r.prompt, r.max_new_tokens)
        assert min(margins) > 1e-4   # no tie that rounding could turn
        assert r.generated == tokens


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(pkg, tmp_path, dtype):
    cfg = rc.cases()["mid"]
    bits, w = rc.random_weights("mid", cfg, 8)
    rc.write_model(pkg, cfg, bits, str(tmp_path / "model"))
    (tmp_path / "out").mkdir()
    rng = np.random.default_rng(1)
    a, b = (rng.integers(0, cfg["vocab"], size=n).tolist() for n in (90, 70))
    places = list(range(20, 68))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:80], "want": [3, 79]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[80:81], "want": []}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[2:], "want": places}, {"id": "a", "tokens": a[81:], "want": [8]}], "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b, "want": places}], "end": ["c"]}]
    out = run_tool("trace_run", ["--model", str(tmp_path / "model"), "--dtype", dtype, "--out", str(tmp_path / "out"), "--max-tokens", "256"],
                   input="".join(json.dumps(s) + "\n" for s in steps))
    assert [x for x in out.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    pa, pb = plain.forward(cfg, w, a)[0], plain.forward(cfg, w, b)[0]
    for step, want in ((2, np.concatenate([pb[22:70], pa[[89]]])), (3, pb[20:68])):
        got = np.fromfile(tmp_path / "out" / f"{step}.f32", dtype="<f4").reshape(want.shape)
        rc.agree(got, want, cfg, dtype)
    assert not (tmp_path / "out" / "1.f32").exists()


def test_generate_tool(pkg, tmp_path):
    cfg = rc.cases()["state_only"]
    bits, w = rc.random_weights("state_only", cfg, 2)
    rc.write_model(pkg, cfg, bits, str(tmp_path / "model"))
    prompts = [[5, 6, 7], [1], [60, 2]]
    args = ["--model", str(tmp_path / "model"), "--max-new", "6", "--dtype", "float32", "--batch", "2", "--max-seq", "64"]
    out = run_tool("generate", args + [x for p in prompts for x in ("--prompt", ",".join(map(str, p)))])
    assert [[int(t) for t in line.split(",")] for line in out.stdout.splitlines()] == [plain.greedy(cfg, w, p, 6)[0] for p in prompts]
