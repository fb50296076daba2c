"""Kalevik without a GPU: the plain implementation against closed forms, config.json decoding, tensor inventory, step list,
checkpoint checks."""
import copy
import math

import numpy as np
import pytest

import kalevik_cases as kc
import plain_kalevik as plain


# ---- the plain implementation --------------------------------------------------------------------------------------
def test_plain_rotations_pair_the_right_entries():
    x = np.zeros((3, 1, 6))
    x[:, 0, 0] = 1.0
    a = 2 * 1.0
    assert np.allclose(plain.rotate_neighbours(x, 4, 100.0)[2, 0], [math.cos(a), math.sin(a), 0, 0, 0, 0])
    assert np.allclose(plain.rotate_halves(x, 4, 100.0)[2, 0], [math.cos(a), 0, math.sin(a), 0, 0, 0])
    assert np.allclose(plain.rotate_halves(x, 4, 100.0, 4.0)[2, 0], [math.cos(a / 4), 0, math.sin(a / 4), 0, 0, 0])
    y = np.zeros((3, 1, 6))
    y[:, 0, 3], y[:, 0, 5] = 1.0, 7.0   # the second pair turns with base^(-1/2), the last entry stays
    s = 2 * 100.0 ** -0.5
    assert np.allclose(plain.rotate_neighbours(y, 4, 100.0)[2, 0], [0, 0, -math.sin(s), math.cos(s), 0, 7.0])
    assert np.allclose(plain.rotate_halves(y, 4, 100.0)[2, 0], [0, -math.sin(s), 0, math.cos(s), 0, 7.0])


def test_plain_rotation_makes_scores_relative():
    rng = np.random.default_rng(1)
    for turn in (plain.rotate_neighbours, plain.rotate_halves):
        q, k = (turn(np.tile(rng.standard_normal((1, 1, 8)), (9, 1, 1)), 8, 50.0)[:, 0] for _ in range(2))
        s = q @ k.T
        assert np.allclose(s[5, 2], s[8, 5]) and not np.allclose(s[5, 2], s[5, 3])


def test_plain_chunk_mask_and_sink():
    seen = plain.chunk_mask(7, 3)
    assert seen.sum(axis=1).tolist() == [1, 2, 3, 1, 2, 3, 1] and seen[4].tolist() == [False, False, False, True, True, False, False]
    w = plain.softmax_plus_one(np.zeros((1, 7, 7)), seen)
    assert np.allclose(w[0, 5], [0, 0, 0, 0.25, 0.25, 0.25, 0]) and np.allclose(w[0, 6, 6], 0.5)
    big = plain.softmax_plus_one(np.full((1, 1, 1), -800.0), np.ones((1, 1), dtype=bool))
    assert big[0, 0, 0] == 0.0


def test_plain_retention_is_the_sum_over_the_past():
    rng = np.random.default_rng(2)
    q, k, v = (rng.standard_normal((6, 2, n)) for n in (4, 4, 3))
    decay = np.array([0.5, 1.0])
    o = plain.retention_scan(q, k, v, decay)
    want = sum(decay ** (5 - s) * np.einsum("hd,hd->h", q[5], k[s]) * v[s].T for s in range(6)).T
    assert np.allclose(o[5], want)


def test_plain_routing():
    s = np.array([[0.30, 0.05, 0.25, 0.20, 0.15, 0.05]])
    w = plain.route(np.log(s), {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 2}})
    assert np.allclose(w, [[0.30, 0, 0.25, 0, 0, 0]])   # the chosen scores as they are
    w = plain.route(np.log(s), {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}})
    assert np.allclose(w, [[0.30, 0, 0.25, 0.20, 0, 0]])
    w = plain.route(np.log(s), {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}})
    assert np.allclose(w, [[0.30, 0.05, 0, 0, 0, 0]])   # a group's best counts, not its sum
    assert np.allclose(plain.gelu_erf(np.array([1.0, -2.0])), [0.841344746, -0.045500264])


def test_plain_loop_order():
    cfg = kc.config(8, 8, [None] * 4, (1, 3, 3))
    assert plain.runs(cfg) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert plain.runs(kc.config(8, 8, [None] * 2)) == [(0, False), (1, False)]


def test_plain_model_sees_the_past_and_only_its_chunk():
    a, r = kc.left(2, 1, 8, 8, 5, 4), kc.right(1, 8, 8)
    tokens = np.random.default_rng(2).integers(0, 40, size=17)
    changed = tokens.copy()
    changed[6] = (changed[6] + 1) % 40
    for scales, reach in (((1.0, 0.0), range(6, 10)), ((0.0, 1.0), range(6, 17))):
        cfg = kc.config(40, 24, [kc.parallel(a, r, None, scales)])
        _, w = kc.random_weights(cfg, 1)
        differs = np.abs(plain.forward(cfg, w, tokens)[0] - plain.forward(cfg, w, changed)[0]).max(axis=1) > 1e-12
        assert differs.tolist() == [i in reach for i in range(17)]


# ---- configuration and plan ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", sorted(kc.cases()))
def test_tensor_inventory_follows_the_configuration(pkg, name):
    cfg = kc.cases()[name]
    builder = kc.builder_of(pkg, cfg, "bfloat16")
    shapes = plain.tensor_shapes(cfg)
    assert {n: tuple(s) for n, _k, s, _ in builder.tensors()} == {k: tuple(v) for k, v in shapes.items()}
    used = set()
    for st in builder.decode_steps():
        names = [x.decode() for x in (st.weight, st.weight2, st.weight3, st.weight4, st.weight5, st.weight6) if x]
        if st.kind == pkg.plan.STEP_ROUTED_MLP:
            names = [f"{names[0]}{e}{s}" for e in range(st.experts) for s in names[1:3]] + names[3:]
        used |= set(names)
    constants = builder.constants()
    assert used == set(shapes) | set(constants)
    assert set(constants) == {f"l{i}.mix.right.decay" for i, layer in enumerate(cfg["layers"]) if layer["type"] == "parallel"}
    assert builder.config.runs() == plain.runs(cfg)
    elems = sum(int(np.prod(s)) for n, _k, s, _ in builder.tensors() if _k == "matrix" and ".e" not in n and "shared.up" not in n and "shared.down" not in n
                and not n.endswith((".uk", ".uv")))
    if max(layers for layers, _ in builder.config.runs()) + 1 == len(builder.config.runs()):   # nothing runs twice
        assert builder.config.product_elems() == elems


def test_steps_carry_every_size_and_constant(pkg):
    P, cfg = pkg.plan, kc.cases()["mid"]
    builder = kc.builder_of(pkg, cfg, "float32", max_seq=128, max_batch=3, pool_tokens=200)
    steps = builder.decode_steps()
    g = [s for s in steps if s.kind == P.STEP_GROUPED_ATTN]
    assert [(s.layer, s.heads, s.kv_heads, s.head_dim, s.value_dim, s.chunk, s.rope_dim, s.rope_pairs, s.sink_one) for s in g] == \
        [(0, 6, 2, 40, 24, 50, 24, P.ROPE_HALVES, 1)] + [(i, 4, 4, 32, 48, 100, 32, P.ROPE_HALVES, 1) for i in (1, 2, 3)]
    assert np.allclose([(s.rope_divisor, s.rope_base, s.out_scale) for s in g], [(2.5, 1e4, 0.8)] + 3 * [(1.0, 500.0, 1.3)])
    r = [s for s in steps if s.kind == P.STEP_RETENTION]
    assert [(s.layer, s.heads, s.key_dim, s.value_dim, s.in4_off % 8, s.out_off % 8) for s in r] == [(0, 3, 48, 40, 0, 0)] + [(i, 2, 24, 72, 0, 0) for i in (1, 2, 3)]
    assert np.allclose([(s.scale, s.out_scale) for s in r], [(48 ** -0.5, 0.5)] + 3 * [(24 ** -0.5, 0.4)])
    a = [s for s in steps if s.kind == P.STEP_LATENT_ATTN]
    assert [(s.layer, s.heads, s.n, s.head_dim, s.key_dim, s.rope_dim, s.rope_pairs) for s in a] == \
        [(i, 3, 72, 24, 8, 8, 1) if i % 2 == 0 else (i, 5, 56, 16, 24, 24, 1) for i in range(6)] + [(6, 2, 40, 32, 16, 16, 1)]
    m = [s for s in steps if s.kind == P.STEP_ROUTED_MLP]
    assert [(s.experts, s.top, s.groups, s.groups_keep, s.k, s.k2, bool(s.weight5)) for s in m] == [(12, 3, 3, 2, 56, 72, True)] + 3 * [(8, 2, 4, 3, 40, 0, False)]
    assert all((s.score_act, s.group_best, s.raw_weights, s.scale) == (P.SCORE_SOFTMAX, 1, 1, 1.0) for s in m)
    joins = [s for s in steps if s.kind == P.STEP_POSTNORM_RESADD_COPY_RMSNORM and s.weight3]
    assert [(s.weight, s.weight2, s.weight3) for s in joins] == 2 * [(b"l3.norm2b", b"l1.norm1", b"embed")] and np.allclose([s.scale for s in joins], 0.7)
    assert steps[-3].kind == P.STEP_POSTNORM_RESADD_RMSNORM and steps[-3].weight == b"l4.norm1b"   # the last layer has no feed-forward
    b = builder.config.buffers_desc()
    assert (b.stream_dtype, b.latent_layers, b.grouped_layers, b.delta_layers, b.max_seq, b.max_batch, b.kv_pool_tokens) == (P.STREAM_ALL_F32, 7, 4, 4, 128, 3, 200)


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][0].update(type="other"), "mixer type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="mixed"), "feed-forward kind"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "6 heads over 4"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "chunks of 0"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=42), "42 rotated entries of 40"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "7 rotated entries of 8"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5]), "1 decays for 3"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "9 of 12 experts"),
    (lambda c: c["loop"].update(stop=6), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c.update(architecture="Other"), "architecture"),
])
def test_configurations_outside_the_recipe_are_refused(pkg, change, text):
    cfg = copy.deepcopy(kc.cases()["mid"])
    change(cfg)
    with pytest.raises(ValueError, match=text):
        pkg.kalevik.decode_config(cfg)


def test_checkpoint_is_checked_against_its_configuration(pkg, tmp_path):
    cfg = kc.cases()["tiny"]
    bits, _ = kc.random_weights(cfg, 3)
    kc.write_model(pkg, cfg, bits, str(tmp_path / "ok"))
    builder, weights = pkg.prepare_dense_bundle(str(tmp_path / "ok"), dtype="float32", max_seq=64, max_batch=1)
    assert isinstance(builder, pkg.KalevikPlanBuilder) and builder.config.dtype == "float32" and all(np.array_equal(weights[k], bits[k]) for k in bits)
    broken = dict(bits)
    broken["l0.mix.right.g"] = np.zeros((8, 4), dtype=np.uint16)
    kc.write_model(pkg, cfg, broken, str(tmp_path / "shape"))
    with pytest.raises(pkg.bundle.BundleError, match="l0.mix.right.g"):
        pkg.prepare_dense_bundle(str(tmp_path / "shape"))
    del broken["l0.mix.right.g"]
    kc.write_model(pkg, cfg, broken, str(tmp_path / "missing"))
    with pytest.raises(pkg.bundle.BundleError, match="l0.mix.right.g"):
        pkg.prepare_dense_bundle(str(tmp_path / "missing"))
