"""Rirotar without a GPU: the plain implementation against closed forms, config.json decoding, tensor inventory, step list,
checkpoint checks."""
import copy
import math

import numpy as np
import pytest

import plain_rirotar as plain
import rirotar_cases as rc


# ---- the plain implementation --------------------------------------------------------------------------------------
def test_plain_clamped_gate_values():
    g = plain.clamped_gate(np.array([0.5, 9.0, -9.0, 0.5]), np.array([0.25, 5.0, -5.0, -7.0]), 2.0)
    s = lambda z: 1.0 / (1.0 + math.exp(-1.702 * z))   # noqa: E731
    # the gate has no lower limit
    assert np.allclose(g, [0.5 * s(0.5) * 1.25, 2.0 * s(2.0) * 3.0, -9.0 * s(-9.0) * -1.0, 0.5 * s(0.5) * -1.0])


def test_plain_convolution_is_causal_and_starts_from_zeros():
    x, taps = np.array([[1.0], [10.0], [100.0], [1000.0]]), np.array([[2.0, 3.0, 5.0]])
    assert plain.short_conv(x, taps)[:, 0].tolist() == [5.0, 53.0, 532.0, 5320.0]


def test_plain_delta_reads_its_own_write():
    q = k = np.array([[[1.0, 0.0]]])
    o = plain.delta_scan(q, k, np.array([[[3.0, -2.0]]]), np.full((1, 1, 2), 0.5), np.array([[0.25]]))
    assert np.allclose(o, [[[0.75, -0.5]]])
    # a second write along the same key moves what is stored towards the new value, decayed first
    k2 = np.repeat(k, 2, axis=0)
    o = plain.delta_scan(k2, k2, np.array([[[4.0]], [[8.0]]]), np.full((2, 1, 2), 0.5), np.array([[1.0], [0.5]]))
    assert np.allclose(o[:, 0, 0], [4.0, 2.0 + 0.5 * (8.0 - 2.0)])
    # decay acts on the rows of the key's own channels
    g = np.array([[[1.0, 1.0]], [[0.0, 1.0]]])
    o = plain.delta_scan(np.array([[[0.0, 0.0]], [[1.0, 1.0]]]), np.array([[[0.6, 0.8]], [[0.0, 0.0]]]), np.array([[[1.0]], [[0.0]]]), g, np.ones((2, 1)))
    assert np.allclose(o[1, 0, 0], 0.8)


def test_plain_window_and_sink():
    seen = plain.window_mask(4, 2)
    assert seen.tolist() == [[True, False, False, False], [True, True, False, False], [False, True, True, False], [False, False, True, True]]
    w = plain.sink_softmax(np.zeros((1, 4, 4)), seen, np.array([math.log(2.0)]))
    assert np.allclose(w[0, 0, 0], 1.0 / 3.0) and np.allclose(w[0, 3], [0.0, 0.0, 0.25, 0.25])


def test_plain_routing():
    def logit(p):
        return np.log(p) - np.log1p(-np.asarray(p))

    s = np.array([[0.9, 0.1, 0.6, 0.55, 0.5, 0.2]])
    w = plain.route(logit(s), {"experts": 6, "top": 2, "scale": 2.0, "groups": {"count": 3, "keep": 1}})
    # the pairs sum to 1.0, 1.15 and 0.7: the second group wins although the best expert is in the first
    assert np.allclose(w, [[0, 0, 2 * 0.6 / 1.15, 2 * 0.55 / 1.15, 0, 0]])
    w = plain.route(logit(s), {"experts": 6, "top": 2, "scale": 1.0})
    assert np.allclose(w, [[0.9 / 1.5, 0, 0.6 / 1.5, 0, 0, 0]])
    w = plain.route(logit(s), {"experts": 6, "top": 3, "scale": 1.0, "groups": {"count": 6, "keep": 4}})   # groups of one
    assert np.nonzero(w[0])[0].tolist() == [0, 2, 3]


def test_plain_model_sees_only_the_past_and_nothing_behind_a_window():
    cfg = rc.cases()["windows"]
    short = dict(cfg, layers=[rc.latent(2, 24, 24, 40, 5, rc.dense(48))])
    _, w = rc.random_weights("windows", cfg, 1)
    tokens = np.random.default_rng(2).integers(0, cfg["vocab"], size=20)
    changed = tokens.copy()
    changed[8] = (changed[8] + 1) % cfg["vocab"]
    a, b = plain.forward(short, w, tokens)[0], plain.forward(short, w, changed)[0]
    differs = np.abs(a - b).max(axis=1) > 1e-9
    assert differs.tolist() == [8 <= i < 13 for i in range(20)]


# ---- configuration and plan ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(rc.cases()))
def test_tensor_inventory_follows_the_configuration(pkg, name):
    cfg = rc.cases()[name]
    builder = rc.builder_of(pkg, name, cfg, "bfloat16")
    shapes = rc.shapes_of(name, cfg)
    assert {n: tuple(s) for n, _k, s, _ in builder.tensors()} == {k: tuple(v) for k, v in shapes.items()}
    used = set()
    for st in builder.decode_steps():
        names = [x.decode() for x in (st.weight, st.weight2, st.weight3, st.weight4, st.weight5, st.weight6) if x]
        if st.kind == pkg.plan.STEP_ROUTED_MLP:
            names = [f"{names[0]}{e}{s}" for e in range(st.experts) for s in names[1:]]
        used |= set(names)
    assert used == set(shapes)


def test_steps_carry_every_size_and_constant(pkg):
    P, cfg = pkg.plan, rc.cases()["mid"]
    builder = rc.builder_of(pkg, "mid", cfg, "float32", max_seq=128, max_batch=3, pool_tokens=200)
    steps = builder.decode_steps()
    d = [s for s in steps if s.kind == P.STEP_GATED_DELTA]
    assert [(s.layer, s.heads, s.groups, s.key_dim, s.value_dim, s.conv_kernel, s.k, s.gate_act) for s in d] == \
        [(0, 4, 2, 48, 40, 4, 48, P.GATE_SIGMOID), (1, 6, 3, 32, 72, 3, 1, P.GATE_SILU), (2, 2, 2, 64, 24, 2, 64, P.GATE_SIGMOID)]
    assert all(abs(s.scale - s.key_dim ** -0.5) < 1e-7 and abs(s.eps2 - 1e-6) < 1e-12 and abs(s.eps - 1e-5) < 1e-11 for s in d)
    a = [s for s in steps if s.kind == P.STEP_LATENT_ATTN]
    assert [(s.layer, s.window_left, s.n, s.heads, s.key_dim) for s in a] == [(0, 50, 72, 4, 0), (1, 7, 48, 3, 0)]
    r = [s for s in steps if s.kind == P.STEP_ROUTED_MLP]
    assert [(s.experts, s.top, s.groups, s.groups_keep, s.k, s.n) for s in r] == [(12, 4, 3, 2, 72, 160), (8, 2, 4, 2, 96, 160)]
    assert np.allclose([(s.scale, s.limit) for s in r], [(1.6, 0.9), (0.7, 1.4)])
    g = [s for s in steps if s.kind == P.STEP_CLAMPED_GLU]
    assert np.allclose([(s.scale, s.limit) for s in g], [(1.702, 1.2), (1.702, 0.5)])
    assert steps[1].kind == P.STEP_COPY_RMSNORM and steps[-4].kind == P.STEP_RESADD_RMSNORM and all(s.weight_bias == 1.0 for s in (steps[1], steps[-4]))
    assert steps[-2].kind == P.STEP_SOFTCAP and steps[-2].scale == 9.0
    b = builder.config.buffers_desc()
    assert (b.stream_dtype, b.latent_layers, b.delta_layers, b.max_seq, b.max_batch, b.kv_pool_tokens) == (P.STREAM_ALL_F32, 2, 3, 128, 3, 200)
    uncapped = dict(cfg)
    del uncapped["logit_softcap"]
    assert all(s.kind != P.STEP_SOFTCAP for s in rc.builder_of(pkg, "mid", uncapped, "bfloat16").decode_steps())


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][0].update(type="other"), "mixer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="mixed"), "feed-forward kind"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "4 heads over 3"),
    (lambda c: c["layers"][2]["mixer"].update(rot_dim=8), "rotated part"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "window of 0"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "9 of 12 experts"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=5), "groups"),
    (lambda c: c.update(architecture="Other"), "architecture"),
])
def test_configurations_outside_the_recipe_are_refused(pkg, change, text):
    cfg = copy.deepcopy(rc.cases()["mid"])
    shapes = rc.shapes_of("mid", cfg)
    change(cfg)
    with pytest.raises(ValueError, match=text):
        pkg.rirotar.decode_config(cfg, shapes)


def test_checkpoint_is_checked_against_its_configuration(pkg, tmp_path):
    cfg = rc.cases()["tiny"]
    bits, _ = rc.random_weights("tiny", cfg, 3)
    rc.write_model(pkg, cfg, bits, str(tmp_path / "ok"))
    builder, weights = pkg.prepare_dense_bundle(str(tmp_path / "ok"), dtype="float32", max_seq=64, max_batch=1)
    assert builder.config.layers[0].mixer.decay_rank == 3   # stands in the tensors alone
    assert builder.config.dtype == "float32" and all(np.array_equal(weights[k], bits[k]) for k in bits)
    broken = dict(bits)
    broken["l0.mix.a2"] = np.zeros((8, 4), dtype=np.uint16)
    rc.write_model(pkg, cfg, broken, str(tmp_path / "shape"))
    with pytest.raises(pkg.bundle.BundleError, match="l0.mix.a2"):
        pkg.prepare_dense_bundle(str(tmp_path / "shape"))
    del broken["l0.mix.a1"]
    rc.write_model(pkg, cfg, broken, str(tmp_path / "missing"))
    with pytest.raises(pkg.bundle.BundleError, match="l0.mix.a1"):
        pkg.prepare_dense_bundle(str(tmp_path / "missing"))
