"""Vuzunex without a GPU: the plain implementation against closed forms, config.json decoding, tensor inventory, step list,
checkpoint checks, and the batching logic over a stand-in model."""
import copy
import math
import types

import numpy as np
import pytest

import plain_vuzunex as plain
import vuzunex_cases as vc


# ---- the plain implementation --------------------------------------------------------------------------------------
def test_plain_norm_and_activation_values():
    x = np.array([[3.0, 4.0]])
    assert np.allclose(plain.rms_norm(x, np.array([0.5, -0.5]), 0.0, 1.0), x / math.sqrt(12.5) * [1.5, 0.5])
    assert np.allclose(plain.rms_norm(x, np.ones(2), 12.5, 0.0), x / 5.0)   # eps inside the root
    assert plain.gelu_tanh(np.array(0.0)) == 0.0
    assert abs(float(plain.gelu_tanh(np.array(1.0))) - 0.841192) < 1e-6


def test_plain_rotation_is_relative_and_partial():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 6)), rng.standard_normal((1, 6))
    turn = dict(dims=4, base=50.0, scaling=None)
    dots = [float((plain.rotate(q, [p + 3], **turn) @ plain.rotate(k, [p], **turn).T)[0, 0]) for p in (0, 5, 40)]
    assert np.allclose(dots, dots[0])
    assert np.allclose(plain.rotate(q, [7], **turn)[:, 4:], q[:, 4:])
    u, v = q[0, 0], q[0, 2]
    assert np.allclose(plain.rotate(q, [1], **turn)[0, [0, 2]], [u * math.cos(1) - v * math.sin(1), v * math.cos(1) + u * math.sin(1)])


def test_plain_interpolated_frequencies():
    plain_f, one = plain.rotary_frequencies(16, 10000.0, None)
    f, magnitude = plain.rotary_frequencies(16, 10000.0, dict(factor=4.0, original=1000, fast=32.0, slow=1.0))
    assert one == 1.0 and abs(magnitude - (0.1 * math.log(4.0) + 1.0)) < 1e-15
    assert f[0] == plain_f[0] and np.allclose(f[-1], plain_f[-1] / 4.0)   # fastest pair kept, slowest divided
    assert np.all(f <= plain_f) and np.all(f >= plain_f / 4.0 - 1e-18)
    # bounds that fall together: a step instead of a ramp
    g, _ = plain.rotary_frequencies(4, 10000.0, dict(factor=2.0, original=2.0, fast=8.0, slow=8.0))
    assert np.allclose(g, plain.rotary_frequencies(4, 10000.0, None)[0] * [1.0, 0.5])


def test_plain_attention_sees_only_the_past():
    cfg = vc.cases()["mid"]
    _, w = vc.random_weights(cfg, 1)
    tokens = np.random.default_rng(2).integers(0, cfg["vocab"], size=12)
    changed = tokens.copy()
    changed[8] = (changed[8] + 1) % cfg["vocab"]
    a, b = plain.forward(cfg, w, tokens)[0], plain.forward(cfg, w, changed)[0]
    assert np.array_equal(a[:8], b[:8]) and np.abs(a[8:] - b[8:]).max() > 1e-3


# ---- configuration and plan ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(vc.cases()))
def test_tensor_inventory_follows_the_configuration(pkg, name):
    cfg = vc.cases()[name]
    builder = vc.builder_of(pkg, cfg, "bfloat16")
    assert {n: tuple(s) for n, _k, s, _ in builder.tensors()} == {k: tuple(v) for k, v in plain.tensor_shapes(cfg).items()}
    used = set()
    for st in builder.decode_steps():
        used |= {x.decode() for x in (st.weight, st.weight2, st.weight3) if x}
    assert used == set(plain.tensor_shapes(cfg))


def test_steps_of_unequal_and_borrowed_layers(pkg):
    P = pkg.plan
    cfg = vc.cases()["mixed"]
    builder = vc.builder_of(pkg, cfg, "float32", max_seq=128, max_batch=3, pool_tokens=200)
    steps = builder.decode_steps()
    attn = [s for s in steps if s.kind == P.STEP_LATENT_ATTN]
    assert [s.layer for s in attn] == [0, 1, 2, 3, 4]                       # a cache of its own per layer
    assert [s.weight2.decode() for s in attn] == ["l0.mix.uk", "l1.mix.uk", "l0.mix.uk", "l1.mix.uk", "l0.mix.uk"]
    assert [s.heads for s in attn] == [2, 4, 2, 4, 2] and [s.n for s in attn] == [88, 120, 88, 120, 88]
    assert attn[0].rope_factor == 0.0 and attn[1].rope_factor == 2.0 and attn[1].rope_original == 64.0
    assert sum(s.kind == P.STEP_GEGLU for s in steps) == 3                  # layers 1 and 3 have no feed-forward
    # a layer without feed-forward: its mixer's norm is the one in front of the next layer's
    kinds = [(s.weight.decode(), s.weight2.decode()) for s in steps if s.kind == P.STEP_POSTNORM_RESADD_COPY_RMSNORM]
    assert ("l1.norm1b", "l0.norm1") in kinds and ("l0.norm2b", "l1.norm1") in kinds
    assert steps[1].kind == P.STEP_COPY_RMSNORM and steps[-3].kind == P.STEP_POSTNORM_RESADD_RMSNORM
    assert (steps[-3].weight.decode(), steps[-3].weight2.decode()) == ("l0.norm2b", "final.norm")
    d = builder.config.buffers_desc()
    assert (d.stream_dtype, d.latent_layers, d.max_seq, d.max_batch, d.kv_pool_tokens) == (P.STREAM_ALL_F32, 5, 128, 3, 200)


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][0].update(type="other"), "mixer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="routed"), "feed-forward kind"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "rotated entries"),
    (lambda c: c["layers"][0].update(weights_of=0), "weights_of"),
    (lambda c: c.update(architecture="Other"), "architecture"),
])
def test_configurations_outside_the_recipe_are_refused(pkg, change, text):
    cfg = copy.deepcopy(vc.cases()["mid"])
    change(cfg)
    with pytest.raises(ValueError, match=text):
        pkg.vuzunex.decode_config(cfg)


def test_checkpoint_is_checked_against_its_configuration(pkg, tmp_path):
    cfg = vc.cases()["tiny"]
    bits, _ = vc.random_weights(cfg, 3)
    vc.write_model(pkg, cfg, bits, str(tmp_path / "ok"))
    builder, weights = pkg.prepare_dense_bundle(str(tmp_path / "ok"), dtype="float32", max_seq=64, max_batch=1)
    assert builder.config.dtype == "float32" and all(np.array_equal(weights[k], bits[k]) for k in bits)
    broken = dict(bits)
    broken["l0.mix.o"] = bits["l0.mix.o"][:-1]
    vc.write_model(pkg, cfg, broken, str(tmp_path / "shape"))
    with pytest.raises(pkg.bundle.BundleError, match="l0.mix.o"):
        pkg.prepare_dense_bundle(str(tmp_path / "shape"))
    del broken["l0.mix.o"]
    vc.write_model(pkg, cfg, broken, str(tmp_path / "missing"))
    with pytest.raises(pkg.bundle.BundleError, match="missing"):
        pkg.prepare_dense_bundle(str(tmp_path / "missing"))


# ---- batching over a stand-in model --------------------------------------------------------------------------------
class FakeModel:
    """Counts pages as the runtime does; the next token is a function of everything the sequence has seen."""

    def __init__(self, batch, pool_pages, max_seq=512):
        self.batch, self.pool, self.desc = batch, pool_pages, types.SimpleNamespace(max_seq=max_seq)
        self.seen = [[] for _ in range(batch)]
        self.batches = []

    @property
    def free_pages(self):
        return self.pool - sum(-(-len(s) // 64) for s in self.seen)

    def reset_sequence(self, slot):
        self.seen[slot] = []

    @staticmethod
    def next_token(seen):
        return (sum((i + 1) * t for i, t in enumerate(seen)) * 31 + len(seen)) % 97

    def run_batch(self, entries, logits=True):
        self.batches.append([(s, len(t)) for s, t, _ in entries])
        assert len({s for s, _, _ in entries}) == len(entries)
        greedy = []
        for slot, tokens, want in entries:
            before = list(self.seen[slot])
            greedy += [self.next_token(before + list(tokens[:p + 1])) for p in want]
            self.seen[slot] += list(tokens)
        assert self.free_pages >= 0
        out = np.zeros((len(greedy), 97), dtype=np.float32)
        out[np.arange(len(greedy)), greedy] = 1.0
        return (out if logits else None), np.array(greedy, dtype=np.int32)


def expected_tokens(prompt, n):
    seen = list(prompt)
    for _ in range(n):
        seen.append(FakeModel.next_token(seen))
    return seen[len(prompt):]


@pytest.mark.parametrize("budget", [4, 7, 64])
@pytest.mark.parametrize("sampled", [False, True])
def test_scheduler_serves_every_request_whatever_the_budget(pkg, budget, sampled):
    model = FakeModel(batch=3, pool_pages=5)
    sched = pkg.BatchScheduler(model, row_budget=budget, sampler=(lambda row: int(np.argmax(row))) if sampled else None)
    rng = np.random.default_rng(budget)
    requests = [pkg.Request(i, rng.integers(0, 97, size=n).tolist(), m) for i, (n, m) in enumerate([(1, 3), (70, 5), (9, 80), (64, 1), (2, 2), (130, 9)])]
    for r in requests:
        sched.submit(r)
    sched.run()
    assert all(r.generated == expected_tokens(r.prompt, r.max_new_tokens) for r in requests)
    assert model.free_pages == 5 and len(sched.slots.free) == 3
    assert all(sum(n for _, n in b) <= budget for b in model.batches)
    assert any(len(b) > 1 and max(n for _, n in b) > 1 and min(n for _, n in b) == 1 for b in model.batches) or budget == 4


def test_scheduler_refuses_what_can_never_run_and_stops_early(pkg):
    model = FakeModel(batch=2, pool_pages=2, max_seq=100)
    sched = pkg.BatchScheduler(model, row_budget=16)
    with pytest.raises(ValueError):
        sched.submit(pkg.Request("long", list(range(90)), 20))
    with pytest.raises(ValueError):
        sched.submit(pkg.Request("empty", [], 2))
    tokens = expected_tokens([5, 6], 10)
    sched.submit(pkg.Request("a", [5, 6], 10, stop_tokens=[tokens[3]]))
    with pytest.raises(ValueError):
        sched.submit(pkg.Request("a", [1], 1))
    sched.run()
    slots = pkg.SequenceSlots(model)
    assert [slots.of("x"), slots.of("y"), slots.of("x")] == [0, 1, 0]
    with pytest.raises(RuntimeError):
        slots.of("z")
    slots.release("x")
    assert slots.of("z") == 0


def test_entry_points_refuse_null_and_foreign_arguments(pkg, lib):
    assert lib.swlm_run_batch(None, 0, None, None, None, None, None, None, None) == -1
    assert lib.swlm_pool_free_pages(None) == -1
    assert lib.swlm_weights_add_matrix_bf16(None, b"w", 1, 1, None) == -1
