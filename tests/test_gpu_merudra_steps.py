"""The step kinds of the Merudra recipe alone, on a GPU, against the plain implementation."""
import numpy as np
import pytest

import merudra_cases as mc
import plain_merudra as plain
from test_gpu_kalevik_steps import weights
from test_gpu_vuzunex_steps import DTYPES, act, close, model_of

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def store(pkg):
    s = pkg.WeightStore(0)
    yield s
    s.close()


# ---- products with biases and of two inputs ------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 2, 4, 5, 40, 130])
@pytest.mark.parametrize("k, first, second", [(64, (24, 8), (40,)), (133, (37, 13, 5), (21, 8)), (520, (300, 4), (520, 3)), (72, (6,), (72,)), (136, (256,), (72, 13)), (200, (500, 12), (264,))])
def test_products_of_two_inputs_with_biases(pkg, store, dtype, rows, k, first, second):
    """Results of both inputs side by side in one buffer, every other one with a bias; the second input starts at rows that are a
    multiple of four, and at others."""
    P, rng, p = pkg.plan, np.random.default_rng(k + rows), f"two{k}."
    steps, parts, at = [], [], 0
    for i, n in enumerate(first + second):
        w = weights(store, p, **{f"m{i}": rng.standard_normal((n, k)) / np.sqrt(k), f"b{i}": rng.standard_normal(n)})
        src = P.BUF_S0 if i < len(first) else P.BUF_S1
        steps.append(P._step(P.STEP_PRODUCT, in_buf=src, out_buf=P.BUF_S2 if i % 2 else P.BUF_S4, out_off=at, n=n, k=k, weight=f"{p}m{i}", weight3=f"{p}b{i}" if i % 2 else ""))
        parts.append((at, n, src, w[f"m{i}"], w[f"b{i}"] if i % 2 else 0.0, i % 2))
        at += -(-n // 8) * 8
    steps.insert(0, P._step(P.STEP_EMBED, out_buf=P.BUF_RESIDUAL, n=k, weight=p + "e"))
    steps[1:1] = [P._step(P.STEP_STREAM_CONV, layer=0, out_buf=P.BUF_S1, n=k, conv_kernel=1, weight=p + "c"), P._step(P.STEP_STREAM_COPY, out_buf=P.BUF_S0, n=k)]
    table = mc.to_bf16_bits(rng.standard_normal((11, k)))
    taps = mc.to_bf16_bits(rng.standard_normal((k, 1)))
    store.add_dense(p + "e", table)
    store.add_dense(p + "c", taps)
    m = model_of(pkg, store, steps, dtype, k, vocab=11, batch=1, max_seq=rows, stream_convs=1)
    assert m.describe().count("\n") == 2   # one launch over the stream, one product
    tokens = (3 * np.arange(rows) + 2) % 11
    m.run_batch([(0, tokens.tolist(), [])])
    x = mc.from_bf16_bits(table)[tokens]
    inputs = {P.BUF_S0: act(x, dtype), P.BUF_S1: act(x + x * mc.from_bf16_bits(taps)[:, 0], dtype)}
    assert np.allclose(m.read_buffer_f32(P.BUF_S1, rows, k), inputs[P.BUF_S1], rtol=1e-2 if dtype == "bfloat16" else 1e-6, atol=1e-6)
    inputs[P.BUF_S1] = m.read_buffer_f32(P.BUF_S1, rows, k).astype(np.float64)
    for at, n, src, w, b, narrow in parts:
        got = m.read_buffer_f32(P.BUF_S2 if narrow else P.BUF_S4, rows, at + n)[:, at:]
        close(got, plain.linear(inputs[src], w, b), dtype if narrow else "float32", slack=4.0)
    m.close()


# ---- the stream ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 3, 9])
@pytest.mark.parametrize("width", [24, 133, 1000, 2184, 5000])
@pytest.mark.parametrize("gated", [True, False])
def test_gated_norm_is_added_to_the_stream(pkg, store, dtype, rows, width, gated):
    P, rng, eps, p = pkg.plan, np.random.default_rng(width + rows), 0.03, f"gn{width}."
    w = weights(store, p, a=0.3 * rng.standard_normal(width))
    st = P._step(P.STEP_GATED_POSTNORM_ADD, in_buf=P.BUF_HIDDEN, in3_buf=P.BUF_S3 if gated else -1, n=width, eps=eps, weight_bias=1.0, weight=p + "a")
    m = model_of(pkg, store, [st], dtype, width, batch=rows)
    x, z, res = (s * rng.standard_normal((rows, width)).astype(np.float32) for s in (1, 2, 3))
    m.write_buffer_f32(P.BUF_HIDDEN, x)
    m.write_buffer_f32(P.BUF_RESIDUAL, res)
    if gated:
        m.write_buffer_f32(P.BUF_S3, z)
    m.run_step(st)
    t = x.astype(np.float64) * (plain.sigmoid(z.astype(np.float64)) if gated else 1.0)
    close(m.read_buffer_f32(P.BUF_RESIDUAL, rows, width), res + plain.rms_norm(t, 1.0 + w["a"], eps), "float32")
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [24, 133, 600, 2184])
def test_depth_average_over_many_results(pkg, store, dtype, width):
    """Seven rounds of: the stream times a matrix, normed and added, averaged with everything before. Single rows and portions."""
    P, rng, eps, p, rounds = pkg.plan, np.random.default_rng(width), 0.01, f"da{width}.", 7
    table = mc.to_bf16_bits(rng.standard_normal((11, width)))
    store.add_dense(p + "e", table)
    steps, w = [P._step(P.STEP_EMBED, out_buf=P.BUF_RESIDUAL, n=width, scale=1.5, weight=p + "e")], {}
    for i in range(rounds):
        w.update(weights(store, p, **{f"m{i}": rng.standard_normal((width, width)) / np.sqrt(width), f"n{i}": 1 + 0.2 * rng.standard_normal(width),
                                      f"a{i}": 0.5 * rng.standard_normal(i + 2)}))
        steps += [P._step(P.STEP_STREAM_COPY, out_buf=P.BUF_S0, n=width), P._step(P.STEP_PRODUCT, in_buf=P.BUF_S0, out_buf=P.BUF_HIDDEN, n=width, k=width, weight=f"{p}m{i}"),
                  P._step(P.STEP_GATED_POSTNORM_ADD, in_buf=P.BUF_HIDDEN, n=width, eps=eps, weight=f"{p}n{i}"), P._step(P.STEP_DEPTH_AVG, n=width, k=i + 2, weight=f"{p}a{i}")]
    m = model_of(pkg, store, steps, dtype, width, vocab=11, batch=2, max_seq=64, depth_results=rounds + 1)
    tokens = (7 * np.arange(40) + 2) % 11
    x = 1.5 * mc.from_bf16_bits(table)[tokens]
    results = [x]
    for i in range(rounds):
        results.append(x + plain.rms_norm(plain.linear(x, w[f"m{i}"]), w[f"n{i}"], eps))
        x = sum(c * r for c, r in zip(w[f"a{i}"], results))
    for rows in (40, 5, 1):
        m.run_batch([(1, tokens[:rows].tolist(), [])])
        close(m.read_buffer_f32(P.BUF_RESIDUAL, rows, width), x[:rows], dtype, slack=3.0)
        m.reset_sequence(1)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width, taps", [(24, 1), (24, 4), (133, 3), (600, 2), (96, 17), (2184, 4), (4100, 3)])
def test_convolution_over_the_stream_alone(pkg, store, dtype, width, taps):
    """Two sequences in portions of all lengths, down to one token, together and alone; the last step of the plan is the convolution,
    so its inputs go to the state by a launch of their own."""
    P, rng, p = pkg.plan, np.random.default_rng(width + taps), f"sc{width}.{taps}."
    table, kernel = mc.to_bf16_bits(rng.standard_normal((31, width))), mc.to_bf16_bits(rng.standard_normal((width, taps)))
    store.add_dense(p + "e", table)
    store.add_dense(p + "c", kernel)
    steps = [P._step(P.STEP_EMBED, out_buf=P.BUF_RESIDUAL, n=width, weight=p + "e"), P._step(P.STEP_STREAM_CONV, layer=0, out_buf=P.BUF_S1, n=width, conv_kernel=taps, weight=p + "c")]
    m = model_of(pkg, store, steps, dtype, width, vocab=31, batch=3, max_seq=200, stream_convs=1)
    tokens = {s: rng.integers(0, 31, size=150) for s in (0, 2)}
    want = {}
    for s, t in tokens.items():
        x = mc.from_bf16_bits(table)[t]
        want[s] = x + plain.short_conv(x, mc.from_bf16_bits(kernel))
    at = {0: 0, 2: 0}
    for cut in ((1, 3), (1, 1), (2, 1), (3, 40), (1, 1), (1, 2), (30, 1), (0, 5), (64, 64), (5, 0), (7, 7), (2, 2)):
        entries = [(s, tokens[s][at[s]:at[s] + n].tolist(), []) for s, n in ((2, cut[1]), (0, cut[0])) if n]
        m.run_batch(entries)
        got = m.read_buffer_f32(P.BUF_S1, sum(len(e[1]) for e in entries), width)
        close(got, np.concatenate([want[s][at[s]:at[s] + len(t)] for s, t, _ in entries]), dtype)
        for s, t, _ in entries:
            at[s] += len(t)
    m.reset_sequence(0)   # whatever the slot holds, a sequence starts from zeros
    m.run_batch([(0, tokens[0][:2].tolist(), [])])
    close(m.read_buffer_f32(P.BUF_S1, 2, width), want[0][:2], dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 3, 64])
@pytest.mark.parametrize("side", [1, 13, 256])
def test_token_gate(pkg, store, dtype, rows, side):
    P, rng, p = pkg.plan, np.random.default_rng(side + rows), f"tg{side}."
    table = mc.to_bf16_bits(rng.standard_normal((9, 3 * side)))
    store.add_dense(p + "t", table)
    st = P._step(P.STEP_TOKEN_GATE, in_buf=P.BUF_S1, out_buf=P.BUF_S1, n=side, in2_off=side, weight=p + "t")
    m = model_of(pkg, store, [st], dtype, 8, vocab=9, batch=rows)
    x = act(3 * rng.standard_normal((rows, side)), dtype)
    tokens = (5 * np.arange(rows) + 3) % 9
    m.write_buffer_f32(P.BUF_S1, x)
    m.run_step(st, token_in=tokens)
    # (far below zero the function is the small rest of a sum that cancels: the error counts against the input)
    want = plain.gelu_tanh(x) * mc.from_bf16_bits(table)[tokens, side:2 * side]
    assert np.abs(m.read_buffer_f32(P.BUF_S1, rows, side) - want).max() <= (3e-6 if dtype == "float32" else 6e-3) * np.abs(x).max() * np.abs(mc.from_bf16_bits(table)).max()
    m.close()


# ---- attention whose values are its keys ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window, every", [(0, 0), (0, 1), (0, 64), (50, 7)])
@pytest.mark.parametrize("heads, kv, dim", [(4, 2, 24), (20, 1, 128), (3, 3, 64), (3, 3, 11), (2, 1, 200), (2, 1, 264)])
def test_attention_over_shared_rows_alone(pkg, store, dtype, window, every, heads, kv, dim):
    """Decode rows at places around page borders, over rows that were appended before them; the gates of the entries come and go."""
    P, n, eps, rng = pkg.plan, 150, 1e-3, np.random.default_rng(window + every + heads)
    gated, scale, coef = heads != 2, 2.0 * dim ** -0.5, 0.8
    gate_at = -(-(heads + kv) * dim // 8) * 8
    st = P._step(P.STEP_GROUPED_ATTN, layer=0, in_buf=P.BUF_S2, in4_buf=P.BUF_S2 if gated else -1, in4_off=gate_at if gated else 0, out_buf=P.BUF_S0, heads=heads, kv_heads=kv,
                 head_dim=dim, value_dim=dim, value_is_key=1, head_norm=1, scale=scale, eps=eps, window_left=window, out_scale=1.0, rope_base=1.0, temp_every=every, temp_coef=coef)
    m = model_of(pkg, store, [st], dtype, 8, batch=1, max_seq=n, grouped_layers=1)
    x, z = 2 * rng.standard_normal((n, (heads + kv) * dim)), rng.standard_normal((n, heads * dim))
    y, z = act(x, dtype), act(z, dtype)
    q = plain.over_rms(y[:, :heads * dim].reshape(n, heads, dim), eps)
    if every:
        q = q * plain.query_temperature(n, coef, every)[:, None, None]
    v = np.repeat(y[:, heads * dim:].reshape(n, kv, dim), heads // kv, axis=1)
    scores = np.einsum("qhd,khd->hqk", act(q, dtype), plain.over_rms(v, eps)) * scale
    i = np.arange(n)
    if window:
        scores = np.where(i[:, None] - i[None, :] < window, scores, -1e30)
    want = np.einsum("hqk,khv->qhv", plain.causal_softmax(scores), v).reshape(n, heads * dim)
    if gated:
        want = want * plain.sigmoid(z)
    got = {}
    for t in range(n):
        m.set_positions([t])
        row = np.zeros((1, gate_at + heads * dim))
        row[0, :(heads + kv) * dim], row[0, gate_at:] = x[t], z[t]
        m.write_buffer_f32(P.BUF_S2, row if gated else row[:, :gate_at])
        m.run_step(st)
        if t in {0, 1, 2, 62, 63, 64, 65, 127, 128, 129, 149, window - 1, window, window + 1, every - 2, every - 1, every}:
            got[t] = m.read_buffer_f32(P.BUF_S0, 1, heads * dim)[0]
    rows = sorted(got)
    close(np.array([got[t] for t in rows]), want[rows], dtype, slack=4.0)
    m.close()


# ---- gated delta rule out of shared buffers ------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, kv, dim, vdim", [(4, 2, 48, 40), (3, 1, 13, 7), (2, 2, 128, 128)])
def test_gated_delta_reads_its_columns(pkg, store, dtype, heads, kv, dim, vdim):
    """q | k | v | gate in one buffer, step sizes and decay inputs in another."""
    P, n, eps, p, taps = pkg.plan, 30, 1e-3, f"gd{heads}.{dim}.", 3
    rng = np.random.default_rng(dim)
    gk, hv = kv * dim, heads * vdim
    w = weights(store, p, q=rng.standard_normal((gk, taps)), k=rng.standard_normal((gk, taps)), v=rng.standard_normal((hv, taps)), n=1 + 0.2 * rng.standard_normal(vdim),
                A_log=rng.standard_normal(heads) - 2, dt=rng.standard_normal(heads))
    for t in "qkv":   # (taps are small tensors, not operands of a product)
        store.add_dense(f"{p}{t}c", mc.to_bf16_bits(w[t]))
    gate_at, decay_at = -(-(2 * gk + hv) // 8) * 8, -(-heads // 8) * 8
    st = P._step(P.STEP_GATED_DELTA, layer=0, in_buf=P.BUF_S2, in2_buf=P.BUF_S4, in3_buf=P.BUF_S4, in3_off=decay_at, in4_buf=P.BUF_S2, in4_off=gate_at, out_buf=P.BUF_S0, k=1,
                 heads=heads, groups=kv, key_dim=dim, value_dim=vdim, conv_kernel=taps, eps=eps, eps2=1e-6, scale=dim ** -0.5, gate_act=P.GATE_SILU, weight=p + "qc",
                 weight2=p + "kc", weight3=p + "vc", weight4=p + "n", weight5=p + "A_log", weight6=p + "dt")
    m = model_of(pkg, store, [st], dtype, 8, batch=1, max_seq=n, delta_layers=1)
    x, b, a = act(rng.standard_normal((n, gate_at + hv)), dtype), rng.standard_normal((n, heads)), rng.standard_normal((n, heads))
    q, k, v = (plain.silu(plain.short_conv(x[:, lo:lo + c], w[t])) for t, lo, c in (("q", 0, gk), ("k", gk, gk), ("v", 2 * gk, hv)))
    q = np.repeat(plain.unit(q.reshape(n, kv, dim)) * dim ** -0.5, heads // kv, axis=1)
    k = np.repeat(plain.unit(k.reshape(n, kv, dim)), heads // kv, axis=1)
    g = np.exp(-np.exp(w["A_log"]) * plain.softplus(a + w["dt"]))
    o = plain.rms_norm(plain.delta_scan(q, k, v.reshape(n, heads, vdim), g, plain.sigmoid(b)), w["n"], eps).reshape(n, hv)
    want = o * plain.silu(x[:, gate_at:])
    got = np.zeros_like(want)
    scalars = np.zeros((n, decay_at + heads))
    scalars[:, :heads], scalars[:, decay_at:] = b, a
    for t in range(n):
        m.set_positions([t])
        m.write_buffer_f32(P.BUF_S2, x[t:t + 1])
        m.write_buffer_f32(P.BUF_S4, scalars[t:t + 1])
        m.run_step(st)
        got[t] = m.read_buffer_f32(P.BUF_S0, 1, hv)[0]
    close(got, want, dtype, slack=4.0)
    m.close()


# ---- routed feed-forward -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 3, 4, 5, 17, 64])
@pytest.mark.parametrize("experts, identity, top, n, k", [(6, 3, 4, 160, 72), (7, 0, 3, 133, 33), (64, 8, 8, 264, 136), (3, 5, 8, 40, 8), (1, 1, 1, 72, 300), (2, 70, 40, 48, 16)])
def test_routed_feed_forward_with_identity_experts(pkg, store, dtype, rows, experts, identity, top, n, k):
    P, rng, p = pkg.plan, np.random.default_rng(experts + rows), f"id.{experts}.{identity}."
    w = {}
    for e in range(experts):
        for part, shape in (("gate", (k, n)), ("up", (k, n)), ("down", (n, k))):
            b = mc.to_bf16_bits(rng.standard_normal(shape) / np.sqrt(shape[1]))
            store.add_matrix(f"{p}e{e}.{part}", b)
            w[f"e{e}.{part}"] = mc.from_bf16_bits(b)
    scored = experts + identity
    w.update(weights(store, p, correction=0.5 * rng.standard_normal(scored) / np.sqrt(scored)))
    st = P._step(P.STEP_ROUTED_MLP, in_buf=P.BUF_S0, in2_buf=P.BUF_S3, out_buf=P.BUF_HIDDEN, n=n, k=k, experts=experts, identity=identity, top=top, groups=1, groups_keep=1,
                 scale=1.0, score_act=P.SCORE_SOFTMAX, group_best=1, raw_weights=1, expert_act=P.EXPERT_SILU, weight=p + "e", weight2=".gate", weight3=".up", weight4=".down",
                 weight7=p + "correction")
    m = model_of(pkg, store, [st], dtype, n, batch=rows)
    x, z = act(rng.standard_normal((rows, n)), dtype), 2 * rng.standard_normal((rows, scored)).astype(np.float32).astype(np.float64)
    if rows > 4:
        z[:5] = z[0]                      # several rows meet at the same experts
        z[5:8, experts:] += 9.0           # and some hand their input through at all places they can
    m.write_buffer_f32(P.BUF_S0, x)
    m.write_buffer_f32(P.BUF_S3, z)
    weight = plain.route(z, w["correction"], top)
    want = weight[:, experts:].sum(axis=1)[:, None] * x
    for e in range(experts):
        want = want + weight[:, e:e + 1] * plain.linear(plain.silu(plain.linear(x, w[f"e{e}.gate"])) * plain.linear(x, w[f"e{e}.up"]), w[f"e{e}.down"])
    for _ in range(2):   # (the second run finds what the first left in the counters)
        m.run_step(st)
        close(m.read_buffer_f32(P.BUF_HIDDEN, rows, n), want, dtype, slack=2.0)
    m.close()


def test_equal_corrected_scores_go_to_the_lower_index(pkg, store):
    P, n, rng = pkg.plan, 16, np.random.default_rng(4)
    for e in range(3):
        for part in ("gate", "up", "down"):
            store.add_matrix(f"eq.e{e}.{part}", mc.to_bf16_bits(rng.standard_normal((n, n)) / 4))
    store.add_dense("eq.c", mc.to_bf16_bits(np.array([-8.0, -8.0, -8.0, 0.0, 0.0, 0.0])))   # choice scores below zero rank like all others
    st = P._step(P.STEP_ROUTED_MLP, in_buf=P.BUF_S0, in2_buf=P.BUF_S3, out_buf=P.BUF_HIDDEN, n=n, k=n, experts=3, identity=3, top=2, groups=1, groups_keep=1,
                 scale=1.0, score_act=P.SCORE_SOFTMAX, group_best=1, raw_weights=1, expert_act=P.EXPERT_SILU, weight="eq.e", weight2=".gate", weight3=".up", weight4=".down", weight7="eq.c")
    for rows in (2, 7):
        m = model_of(pkg, store, [st], "float32", n, batch=rows)
        z, x = np.zeros((rows, 6)), rng.standard_normal((rows, n)).astype(np.float32)
        z[1] = [50.0, -500.0, 0.0, 1.0, 1.0, 2.0]
        m.write_buffer_f32(P.BUF_S0, x)
        m.write_buffer_f32(P.BUF_S3, z)
        m.run_step(st)
        got = m.read_buffer_f32(P.BUF_HIDDEN, rows, n)
        close(got[0], x[0] / 3, "float32")   # two identity experts with scores of a sixth
        assert np.abs(got[1]).max() < 1e-9 * np.abs(x).max() and np.isfinite(got).all()
        m.close()
