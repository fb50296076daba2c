"""Vuzunex models on a GPU against the plain implementation: prompts, decoding, portions, mixed batches, pages and slots used
again, far and border keys, long decoding, greedy generation through the scheduler and the command line tools."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import plain_vuzunex as plain
import vuzunex_cases as vc

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


class Loaded:
    def __init__(self, pkg, cfg, dtype, seed=5, sharpen=1.0, **runtime):
        self.cfg, self.dtype = cfg, dtype
        bits, self.weights = vc.random_weights(cfg, seed, sharpen)
        self.store = pkg.WeightStore(0)
        self.builder = vc.builder_of(pkg, cfg, dtype, **runtime)
        self.model = pkg.load_model(self.store, self.builder, bits)

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

    def close(self):
        self.model.close()
        self.store.close()


@pytest.fixture
def load(pkg):
    made = []

    def make(name_or_cfg, dtype, **kw):
        cfg = vc.cases()[name_or_cfg] if isinstance(name_or_cfg, str) else name_or_cfg
        made.append(Loaded(pkg, cfg, dtype, **kw))
        return made[-1]

    yield make
    for m in made:
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(vc.cases()))
def test_prompt_portions_and_decoding_agree_with_the_plain_model(load, dtype, name):
    m = load(name, dtype)
    tokens = m.tokens(150)
    want, limit = m.plain(tokens), vc.TOLERANCE[dtype]
    whole = m.portions(0, tokens, [150])
    assert vc.row_errors(whole, want).max() <= limit
    m.model.reset_sequence(0)
    singles = m.portions(0, tokens, [1])
    assert vc.row_errors(singles, want).max() <= limit
    for seq, sizes in enumerate(([2], [64, 2, 63, 3, 65], [5, 64, 1, 80], [100, 1])):
        if seq == 0:
            m.model.reset_sequence(0)
        assert vc.row_errors(m.portions(seq, tokens, sizes), want).max() <= limit, sizes


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mid", "mixed", "odd"])
def test_residual_stream_after_every_layer(pkg, load, dtype, name):
    m = load(name, dtype)
    tokens = m.tokens(90)
    _, after = plain.forward(m.cfg, m.weights, tokens)
    for n in range(1, len(m.cfg["layers"]) + 1):
        desc = m.builder.config.buffers_desc()
        desc.latent_layers = n
        part = pkg.InferenceModel(m.store, m.builder.decode_steps(layers=n, store_final=True), desc)
        for rows in (90, 3):
            part.run_batch([(0, tokens[:rows], list(range(rows)))])
            got = part.read_buffer_f32(pkg.plan.BUF_RESIDUAL, rows, m.cfg["width"])
            assert np.abs(got - after[n - 1][:rows]).max() <= (1e-5 if dtype == "float32" else 3e-2) * np.abs(after[n - 1]).max()
            part.reset_sequence(0)
        part.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mid", "odd", "wide"])
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
        assert vc.row_errors(g, m.plain(r)).max() <= vc.TOLERANCE[dtype]
        assert vc.row_errors(g, alone[i]).max() <= vc.TOLERANCE[dtype]
    assert m.model.positions.tolist() == [201, 1, 130, 67]


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_slots_are_used_again(pkg, load, dtype):
    m = load("mid", dtype, max_batch=3, max_seq=256, pool_tokens=5 * 64)
    model, limit = m.model, vc.TOLERANCE[dtype]
    assert model.free_pages == 5
    a, b, c = m.tokens(65, 1), m.tokens(130, 2), m.tokens(60, 3)
    wa, wb, wc = m.plain(a), m.plain(b), m.plain(c)
    assert vc.row_errors(m.portions(0, a, [40, 1]), wa).max() <= limit and model.free_pages == 3
    assert vc.row_errors(m.portions(1, b, [128, 1]), wb).max() <= limit and model.free_pages == 0
    # no page left: refused, nothing changed
    with pytest.raises(pkg.SwlmError):
        model.run_batch([(1, b[:1], [0]), (2, c, [0])])
    assert model.free_pages == 0 and model.positions.tolist() == [65, 130, 0]
    # the slot in the middle of the pool's history goes back and other requests take its pages, out of order
    model.reset_sequence(0)
    assert model.free_pages == 2
    assert vc.row_errors(m.portions(2, c, [7, 9]), wc).max() <= limit
    assert vc.row_errors(m.portions(0, c, [60]), wc).max() <= limit and model.free_pages == 0
    model.reset_sequence(1)
    model.reset_sequence(2)
    assert model.free_pages == 4
    model.reset_sequence(0)
    for seq in (2, 0):
        assert vc.row_errors(m.portions(seq, b[:100], [64, 1]), wb[:100]).max() <= limit
    # places are wanted in any order, also twice, or not at all
    model.reset_state()
    assert model.free_pages == 5
    lg, _ = model.run_batch([(1, a, [64, 0, 64])])
    assert vc.row_errors(lg, wa[[64, 0, 64]]).max() <= limit
    assert model.run_batch([(0, a[:20], [])])[1].size == 0
    for bad in ([(0, [m.cfg["vocab"]], [0])], [(0, [1], [1])], [(5, [1], [0])], [(0, [1], [0]), (0, [1], [0])], [(0, [], [])]):
        with pytest.raises(pkg.SwlmError):
            model.run_batch(bad)
    assert model.positions.tolist() == [20, 65, 0]


BORDERS = [0, 1, 2, 62, 63, 64, 65, 126, 127, 128, 129]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mid", "wide", "odd"])
def test_single_keys_at_page_and_tile_borders(pkg, load, dtype, name):
    """Sharpened queries: a row's result hangs on few keys. The plain model without one key (at a border, far away, or the
    row's own) must differ by far more than what is allowed, and the kernels must agree with the plain model at every row."""
    cfg = dict(vc.cases()[name], layers=vc.cases()[name]["layers"][:1])
    m = load(cfg, dtype, sharpen=3.0)
    tokens = m.tokens(192, seed=9)
    want = m.plain(tokens)
    limit = 5e-5 if dtype == "float32" else 3e-2
    for sizes in ([192], [64, 65, 1], [1], [127, 2, 1]):
        err = vc.row_errors(m.portions(0, tokens, sizes), want)
        assert err.max() <= limit, (sizes, int(err.argmax()))
        m.model.reset_sequence(0)
    # the test itself: leaving a key out shows
    real = plain.causal_softmax
    try:
        for key in BORDERS:
            def without(scores, key=key):
                s = scores.copy()
                s[:, key + 1:, key] = -np.inf
                return real(s)

            plain.causal_softmax = without
            err = vc.row_errors(m.plain(tokens), want)
            assert err[key + 1:].max() > 2.5 * limit and err[:key + 1].max() < 1e-12, key

        def without_own(scores):
            s = scores.copy()
            i = np.arange(1, s.shape[1])
            s[:, i, i] = -np.inf
            return real(s)

        plain.causal_softmax = without_own
        assert (vc.row_errors(m.plain(tokens), want)[1:] > 2.5 * limit).sum() > 10
    finally:
        plain.causal_softmax = real


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_far_key_is_found_again(pkg, load, dtype):
    """The last token asks for one token far back: with q = -strength * k of the same input and opposite embeddings its score
    stands out among hundreds of others (the rotated part hardly turns: a huge base)."""
    lay = vc.layer(2, 40, 8, 32, 56, 0, base=1e9)
    m = load(vc.config(300, 64, [lay]), dtype, max_seq=640)
    q, dkv = m.weights["l0.mix.q"], m.weights["l0.mix.dkv"]
    # W_q (per head, plain part) = -strength * W_uk W_dkv
    rank = 56
    bits = {k: vc.to_bf16_bits(v) for k, v in m.weights.items()}
    new_q = q.copy()
    for h in range(2):
        new_q[h * 48:h * 48 + 40] = -2.5 * (m.weights["l0.mix.uk"][h * 40:(h + 1) * 40] @ dkv[:rank])
    bits["l0.mix.q"] = vc.to_bf16_bits(new_q)
    bits["embed"][298] = bits["embed"][299] ^ 0x8000
    m.weights = {k: vc.from_bf16_bits(v) for k, v in bits.items()}
    pkg.upload_weights(m.store, m.builder, bits)
    tokens = np.random.default_rng(3).integers(0, 298, size=600)
    tokens[599] = 298
    for where in (0, 63, 64, 130):
        t = tokens.copy()
        t[where] = 299
        want, absent = m.plain(t), m.plain(tokens)
        assert vc.row_errors(absent[599:], want[599:])[0] > 0.2
        for sizes in ([600], [599, 1], [300, 298, 2]):
            got = m.portions(0, t.tolist(), sizes)
            assert vc.row_errors(got[599:], want[599:])[0] <= (1e-4 if dtype == "float32" else 5e-2)
            m.model.reset_sequence(0)


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
        assert ((top - chosen) / logits.std()).max() <= (1e-3 if dtype == "float32" else 0.15)
        assert (chosen == top).mean() >= (0.99 if dtype == "float32" else 0.9)
    # one more step by the per-token call, and the logits it leaves
    again = m.model.decode(tokens[-1])
    lg = m.model.logits()
    assert again.tolist() == np.argmax(lg, axis=1).tolist()
    assert vc.row_errors(lg[:1], m.plain(prompt[0].tolist() + tokens[:, 0].tolist())[-1:]).max() <= vc.TOLERANCE[dtype]


def test_prompt_chunks_snapshot_and_reset(load):
    m = load("mixed", "bfloat16", max_batch=2, max_seq=256)
    model, tokens = m.model, m.tokens(180)
    want = int(np.argmax(m.plain(tokens)[-1]))
    model.set_prefill_chunk(70)
    assert model.prefill_sequence(1, tokens) == want
    snap = model.prompt_snapshot()
    a = [int(model.run_batch([(1, [want], [0])])[1][0])]
    model.reset_state()
    assert model.free_pages == 8 and model.positions.tolist() == [0, 0]
    model.run_batch([(0, tokens[:100], [])])   # other data on the pages
    model.restore(snap)
    assert model.positions.tolist() == [0, 180]
    b = [int(model.run_batch([(1, [want], [0])])[1][0])]
    assert a == b
    model.free_snapshot(snap)


@pytest.mark.parametrize("budget", [5, 48, 512])
def test_greedy_generation_through_the_scheduler(pkg, load, budget):
    m = load("mid", "float32", max_batch=3, max_seq=256, pool_tokens=6 * 64)
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


def run_tool(name, args, **kw):
    return subprocess.run([os.path.join(ROOT, "bin", name)] + args, check=True, capture_output=True, text=True, timeout=300, **kw)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(pkg, tmp_path, dtype):
    cfg = vc.cases()["mixed"]
    bits, w = vc.random_weights(cfg, 8)
    vc.write_model(pkg, cfg, bits, str(tmp_path / "model"))
    (tmp_path / "out").mkdir()
    rng = np.random.default_rng(1)
    a, b = (rng.integers(0, cfg["vocab"], size=n).tolist() for n in (90, 70))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:80], "want": [3, 79]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[80:81], "want": []}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[2:], "want": [67, 0]}, {"id": "a", "tokens": a[81:], "want": [8]}], "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b, "want": [69]}], "end": ["c"]}]
    out = run_tool("trace_run", ["--model", str(tmp_path / "model"), "--dtype", dtype, "--out", str(tmp_path / "out"), "--max-tokens", "256"],
                   input="".join(json.dumps(s) + "\n" for s in steps))
    assert [x for x in out.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    pa, pb = plain.forward(cfg, w, a)[0], plain.forward(cfg, w, b)[0]
    for step, want in ((0, pa[[3, 79]]), (2, np.stack([pb[69], pb[2], pa[89]])), (3, pb[[69]])):
        got = np.fromfile(tmp_path / "out" / f"{step}.f32", dtype="<f4").reshape(want.shape)
        assert vc.row_errors(got, want).max() <= vc.TOLERANCE[dtype]
    assert not (tmp_path / "out" / "1.f32").exists()


def test_generate_tool(pkg, tmp_path):
    cfg = vc.cases()["tiny"]
    bits, w = vc.random_weights(cfg, 2)
    vc.write_model(pkg, cfg, bits, str(tmp_path / "model"))
    prompts = [[5, 6, 7], [1], [60, 2]]
    args = ["--model", str(tmp_path / "model"), "--max-new", "6", "--dtype", "float32", "--batch", "2", "--max-seq", "64"]
    out = run_tool("generate", args + [x for p in prompts for x in ("--prompt", ",".join(map(str, p)))])
    assert [[int(t) for t in line.split(",")] for line in out.stdout.splitlines()] == [plain.greedy(cfg, w, p, 6)[0] for p in prompts]
    sampled = [run_tool("generate", args + ["--prompt", "5,6", "--temperature", "1.5", "--seed", s]).stdout for s in ("1", "1", "2")]
    assert sampled[0] == sampled[1] and sampled[0].count(",") == 5
