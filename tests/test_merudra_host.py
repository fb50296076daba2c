"""Merudra without a GPU: the plain implementation against closed forms, config.json decoding, tensor inventory, step list,
checkpoint checks."""
import copy
import math

import numpy as np
import pytest

import merudra_cases as mc
import plain_merudra as plain


# ---- the plain implementation --------------------------------------------------------------------------------------
def test_plain_convolution_looks_back_and_starts_from_zeros():
    x = np.arange(1.0, 6.0)[:, None] * np.array([[1.0, 10.0]])
    taps = np.array([[0.5, 2.0, 1.0], [0.0, 0.0, 1.0]])
    y = plain.short_conv(x, taps)
    assert np.allclose(y[:, 1], x[:, 1]) and np.allclose(y[:, 0], [1, 2 + 2, 3 + 4 + 0.5, 4 + 6 + 1, 5 + 8 + 1.5])


def test_plain_query_temperature_steps_up_at_whole_periods():
    t = plain.query_temperature(9, 0.5, 3)
    assert np.allclose(t[:2], 1.0) and np.allclose(t[2:5], 1 + 0.5 * math.log(2)) and np.allclose(t[5:8], 1 + 0.5 * math.log(3)) and np.allclose(t[8], 1 + 0.5 * math.log(4))


def test_plain_attention_returns_keys_as_they_were_projected():
    """A single token sees itself: the result is its projected key, bias included and not normed, times the gate."""
    m = {"heads": 2, "kv_heads": 1, "dim": 3, "scale": 1.0, "q_temp": {"coef": 0.0, "every": 5}}
    rng = np.random.default_rng(1)
    w = {"q": rng.standard_normal((6, 4)), "q.b": rng.standard_normal(6), "k": rng.standard_normal((3, 4)), "k.b": rng.standard_normal(3),
         "g": np.zeros((6, 4)), "o": np.eye(6)}
    h = rng.standard_normal((1, 4))
    k = w["k"] @ h[0] + w["k.b"]
    assert np.allclose(plain.attention(h, w, "", m, 1e-6), 0.5 * np.concatenate([k, k]))


def test_plain_delta_rule_stores_and_replaces():
    """A unit key written twice with a step size of one holds the last value; a decay forgets."""
    k = np.zeros((3, 1, 4))
    k[:, 0, 1] = 1.0
    v = np.array([[[2.0, 3.0]], [[5.0, 7.0]], [[0.0, 0.0]]])
    out = plain.delta_scan(k, k, v, np.ones((3, 1)), np.array([[1.0], [1.0], [0.0]]))
    assert np.allclose(out[:, 0], [[2, 3], [5, 7], [5, 7]])
    out = plain.delta_scan(k, k, v, np.array([[1.0], [1.0], [0.25]]), np.array([[1.0], [0.5], [0.0]]))
    assert np.allclose(out[:, 0], [[2, 3], [3.5, 5], [0.875, 1.25]])


def test_plain_routing_chooses_by_corrected_scores_and_weighs_by_plain_ones():
    s = np.array([[0.40, 0.30, 0.05, 0.25]])
    w = plain.route(np.log(s), np.array([0.0, -0.2, 0.3, 0.0]), 2)
    assert np.allclose(w, [[0.40, 0, 0, 0]] + np.array([[0, 0, 0.05, 0]]))
    mlp = {"router": {"experts": 1, "identity": 3, "top": 2}, "expert": {"ff": 2}}
    h = np.array([[1.0, -2.0]])
    tensors = {"router": np.log(s).T @ h / (h @ h.T), "correction": np.array([-1.0, 0, 0, 0]), "e0.gate": np.ones((2, 2)), "e0.up": np.ones((2, 2)), "e0.down": np.ones((2, 2))}
    assert np.allclose(plain.routed_mlp(h, tensors, "", mlp), 0.55 * h)   # two identity experts


def test_plain_depth_average_and_token_input():
    """With results of zero everything but the averages and the embedding disappears."""
    cfg = mc.config(12, 6, [mc.delta(1, 1, 4, 4, None), mc.delta(1, 1, 4, 4, None)], taps=2, side=2)
    _, w = mc.random_weights(cfg, 1)
    for i in range(2):
        w[f"l{i}.norm1"][:] = w[f"l{i}.side.norm"][:] = 0.0
    w["l0.dwa"][:], w["l1.dwa"][:] = [2.0, 3.0], [0.5, -1.0, 4.0]
    tokens = [3, 7]
    _, after = plain.forward(cfg, w, tokens)
    x = w["embed"][tokens]
    assert np.allclose(after[0], 5 * x) and np.allclose(after[1], 0.5 * x - x + 4 * 5 * x)
    w["l0.side.norm"][:] = 1.0
    w["l0.side.gate"][:] = 0.0
    w["side.embed"][:] = 1.0
    assert np.allclose(plain.token_input(x, w, "l0.", w["side.embed"][tokens, :2], 1e-5), x)   # gelu(0) = 0 closes the gate
    assert np.allclose(plain.gelu_tanh(np.array([1.0, -2.0])), [0.841192, -0.045402], atol=1e-6)


def test_plain_model_sees_the_past_and_not_the_future():
    for layer in (mc.attention(2, 1, 8, None), mc.delta(2, 1, 8, 8, mc.routed(2, 1, 2, 8))):
        cfg = mc.config(40, 24, [layer])
        _, w = mc.random_weights(cfg, 1)
        tokens = np.random.default_rng(2).integers(0, 40, size=17)
        changed = tokens.copy()
        changed[6] = (changed[6] + 1) % 40
        differs = np.abs(plain.forward(cfg, w, tokens)[0] - plain.forward(cfg, w, changed)[0]).max(axis=1) > 1e-12
        assert differs.tolist() == [i >= 6 for i in range(17)]


# ---- configuration and plan ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(mc.cases()))
def test_tensor_inventory_follows_the_configuration(pkg, name):
    cfg = mc.cases()[name]
    builder = mc.builder_of(pkg, cfg, "bfloat16")
    shapes = plain.tensor_shapes(cfg)
    assert {n: tuple(s) for n, _k, s, _ in builder.tensors()} == {k: tuple(v) for k, v in shapes.items()}
    used = set()
    for st in builder.decode_steps():
        names = [x.decode() for x in (st.weight, st.weight2, st.weight3, st.weight4, st.weight5, st.weight6, st.weight7) if x]
        if st.kind == pkg.plan.STEP_ROUTED_MLP:
            names = [f"{names[0]}{e}{s}" for e in range(st.experts) for s in names[1:4]] + names[4:]
        used |= set(names)
    assert used == set(shapes)
    elems = sum(int(np.prod(s)) for n, kind, s, _ in builder.tensors() if kind == "matrix" and ".mlp.e" not in n)
    assert builder.config.product_elems() == elems


def test_steps_carry_every_size_and_constant(pkg):
    P, cfg = pkg.plan, mc.cases()["mid"]
    builder = mc.builder_of(pkg, cfg, "float32", max_seq=128, max_batch=3, pool_tokens=200)
    steps = builder.decode_steps()
    a = [s for s in steps if s.kind == P.STEP_GROUPED_ATTN]
    assert [(s.layer, s.heads, s.kv_heads, s.head_dim, s.value_dim, s.temp_every) for s in a] == [(0, 6, 2, 40, 40, 10 + 14), (1, 4, 4, 32, 32, 7), (2, 8, 1, 48, 48, 50)]
    assert np.allclose([(s.scale, s.temp_coef) for s in a], [(40 ** -0.5, 0.4), (1.7 * 32 ** -0.5, 1.5), (48 ** -0.5, -0.2)])
    assert all((s.value_is_key, s.head_norm, s.sink_one, s.rope_dim, s.chunk, s.window_left, s.in3_buf, s.in4_buf) == (1, 1, 0, 0, 0, 0, -1, P.BUF_S2) and s.in4_off % 8 == 0 for s in a)
    d = [s for s in steps if s.kind == P.STEP_GATED_DELTA]
    assert [(s.layer, s.heads, s.groups, s.key_dim, s.value_dim, s.conv_kernel, s.k) for s in d] == [(0, 4, 2, 48, 40, 3, 1), (1, 3, 3, 32, 64, 4, 1)]
    assert np.allclose([(s.scale, s.eps2) for s in d], [(48 ** -0.5, 1e-6), (32 ** -0.5, 1e-6)])
    m = [s for s in steps if s.kind == P.STEP_ROUTED_MLP]
    assert [(s.experts, s.identity, s.top, s.k) for s in m] == [(6, 3, 4, 56), (9, 1, 3, 72), (4, 4, 2, 40)]
    assert all((s.score_act, s.raw_weights, s.expert_act, s.scale, s.groups) == (P.SCORE_SOFTMAX, 1, P.EXPERT_SILU, 1.0, 1) for s in m)
    c = [s for s in steps if s.kind == P.STEP_STREAM_CONV]
    assert [(s.layer, s.conv_kernel, s.weight) for s in c] == [(i, 4, n) for i, n in enumerate((b"l0.canon1", b"l0.canon2", b"l1.canon1", b"l1.canon2", b"l2.canon1", b"l3.canon1", b"l4.canon1", b"l4.canon2"))]
    t = [s for s in steps if s.kind == P.STEP_TOKEN_GATE]
    assert [(s.n, s.in2_off) for s in t] == [(24, 24 * i) for i in range(5)]
    avg = [s for s in steps if s.kind == P.STEP_DEPTH_AVG]
    assert [(s.k, s.weight) for s in avg] == [(i + 2, f"l{i}.dwa".encode()) for i in range(5)]
    added = [s for s in steps if s.kind == P.STEP_GATED_POSTNORM_ADD]
    assert [s.in3_buf != -1 for s in added] == [True, True, False, True, True, False, True, False, True, False, True, True, False]
    assert all(np.isclose(s.eps, 1e-5) for s in a + d + added)
    biased = {s.weight3 for s in steps if s.kind == P.STEP_PRODUCT and s.weight3}
    assert biased == {f"l{i}.mix.{t}.b".encode() for i in (0, 2, 4) for t in "qk"} | {f"l{i}.rg{j}.b".encode() for i in range(5) for j in (1, 2) if j == 1 or i in (0, 1, 4)}
    b = builder.config.buffers_desc()
    assert (b.stream_dtype, b.latent_layers, b.grouped_layers, b.delta_layers, b.max_seq, b.max_batch, b.kv_pool_tokens, b.stream_convs, b.depth_results) == \
        (P.STREAM_ALL_F32, 0, 3, 2, 128, 3, 200, 8, 6)
    b = builder.config.buffers_desc(2)
    assert (b.grouped_layers, b.delta_layers, b.stream_convs, b.depth_results) == (1, 1, 4, 3)


def test_absent_options_are_off(pkg):
    cfg = mc.cases()["mid"]
    del cfg["layers"][0]["mlp"]["router"]["identity"], cfg["layers"][0]["mixer"]["q_temp"]
    c = pkg.merudra.decode_config(cfg)
    assert c.layers[0].mlp.identity == 0 and c.layers[0].mixer.temp_every == 0 and c.layers[1].mlp.identity == 1


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][0].update(type="other"), "mixer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="mixed"), "feed-forward kind"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "6 heads over 4"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=32), "values of 32"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0), "temperature"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=2.5), "temperature"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "4 heads over 3"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=10), "10 of 6"),
    (lambda c: c["canon"].update(taps=0), "0 taps"),
    (lambda c: c["token_side"].update(dim=0), "0 entries"),
    (lambda c: c.update(architecture="Other"), "architecture"),
])
def test_configurations_outside_the_recipe_are_refused(pkg, change, text):
    cfg = copy.deepcopy(mc.cases()["mid"])
    change(cfg)
    with pytest.raises(ValueError, match=text):
        pkg.merudra.decode_config(cfg)


def test_checkpoint_is_checked_against_its_configuration(pkg, tmp_path):
    cfg = mc.cases()["tiny"]
    bits, _ = mc.random_weights(cfg, 3)
    mc.write_model(pkg, cfg, bits, str(tmp_path / "ok"))
    builder, weights = pkg.prepare_dense_bundle(str(tmp_path / "ok"), dtype="float32", max_seq=64, max_batch=1)
    assert isinstance(builder, pkg.MerudraPlanBuilder) and builder.config.dtype == "float32" and all(np.array_equal(weights[k], bits[k]) for k in bits)
    broken = dict(bits)
    broken["l1.mix.g"] = np.zeros((8, 4), dtype=np.uint16)
    mc.write_model(pkg, cfg, broken, str(tmp_path / "shape"))
    with pytest.raises(pkg.bundle.BundleError, match="l1.mix.g"):
        pkg.prepare_dense_bundle(str(tmp_path / "shape"))
    del broken["l1.mix.g"]
    mc.write_model(pkg, cfg, broken, str(tmp_path / "missing"))
    with pytest.raises(pkg.bundle.BundleError, match="l1.mix.g"):
        pkg.prepare_dense_bundle(str(tmp_path / "missing"))
