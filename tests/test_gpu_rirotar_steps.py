"""The step kinds of the Rirotar recipe alone, on a GPU, against the plain implementation."""
import numpy as np
import pytest

import plain_rirotar as plain
import rirotar_cases as rc
from test_gpu_vuzunex_steps import DTYPES, act, close, model_of

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def store(pkg):
    s = pkg.WeightStore(0)
    yield s
    s.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 2, 4, 6, 40])
@pytest.mark.parametrize("n, k", [(37, 52), (400, 264)])
def test_clamped_gate_in_a_product_and_alone(pkg, store, dtype, rows, n, k):
    P, rng, limit, alpha = pkg.plan, np.random.default_rng(n + rows), 0.8, 1.702
    g, u = (rc.to_bf16_bits(2 * rng.standard_normal((n, k)) / np.sqrt(k)) for _ in range(2))
    table, nw = rc.to_bf16_bits(rng.standard_normal((16, k))), rc.to_bf16_bits(0.2 * rng.standard_normal(k))
    for name, v in ((f"c.g{n}", g), (f"c.u{n}", u)):
        store.add_matrix(name, v)
    store.add_dense(f"c.e{n}", table)
    store.add_dense(f"c.n{n}", nw)
    glu = P._step(P.STEP_CLAMPED_GLU, in_buf=P.BUF_S1, in2_buf=P.BUF_S2, out_buf=P.BUF_S1, n=n, scale=alpha, limit=limit)
    steps = [P._step(P.STEP_EMBED, out_buf=P.BUF_HIDDEN, n=k, weight=f"c.e{n}"),
             P._step(P.STEP_COPY_RMSNORM, in_buf=P.BUF_HIDDEN, out_buf=P.BUF_S0, n=k, eps=1e-5, weight_bias=1.0, weight=f"c.n{n}"),
             P._step(P.STEP_PRODUCT, in_buf=P.BUF_S0, out_buf=P.BUF_S1, n=n, k=k, weight=f"c.g{n}"),
             P._step(P.STEP_PRODUCT, in_buf=P.BUF_S0, out_buf=P.BUF_S2, n=n, k=k, weight=f"c.u{n}"), glu]
    m = model_of(pkg, store, steps, dtype, k, vocab=16, batch=rows)
    assert "product+gate" in m.describe()
    m.decode(np.arange(rows) % 16)
    h = plain.rms_norm(rc.from_bf16_bits(table)[np.arange(rows) % 16], rc.from_bf16_bits(nw), 1e-5, 1.0)
    want = plain.clamped_gate(plain.linear(h, rc.from_bf16_bits(g)), plain.linear(h, rc.from_bf16_bits(u)), limit)
    close(m.read_buffer_f32(P.BUF_S1, rows, n), want, dtype, slack=4.0)
    m.close()
    m = model_of(pkg, store, [glu], dtype, k, batch=rows)
    x, y = act(2 * rng.standard_normal((rows, n)), dtype), act(2 * rng.standard_normal((rows, n)), dtype)
    m.write_buffer_f32(P.BUF_S1, x)
    m.write_buffer_f32(P.BUF_S2, y)
    m.run_step(glu)
    close(m.read_buffer_f32(P.BUF_S1, rows, n), plain.clamped_gate(x, y, limit), dtype, slack=1.5)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 3, 5, 40])
def test_several_products_share_a_buffer(pkg, store, dtype, rows):
    """Column offsets of inputs and results; one launch for the products of one input."""
    P, rng, k = pkg.plan, np.random.default_rng(rows), 72
    sizes, offsets = (13, 20, 40), (0, 13, 40)
    table = rc.to_bf16_bits(rng.standard_normal((9, k)))
    store.add_dense("o.e", table)
    store.add_dense("o.n", rc.to_bf16_bits(np.zeros(k)))
    w = [rc.to_bf16_bits(rng.standard_normal((n, k)) / np.sqrt(k)) for n in sizes]
    last = rc.to_bf16_bits(rng.standard_normal((11, 40)) / 6)
    for i, v in enumerate(w):
        store.add_matrix(f"o.w{i}", v)
    store.add_matrix("o.last", last)
    steps = [P._step(P.STEP_EMBED, out_buf=P.BUF_HIDDEN, n=k, weight="o.e"),
             P._step(P.STEP_COPY_RMSNORM, in_buf=P.BUF_HIDDEN, out_buf=P.BUF_S0, n=k, eps=1e-5, weight_bias=1.0, weight="o.n")]
    steps += [P._step(P.STEP_PRODUCT, in_buf=P.BUF_S0, out_buf=P.BUF_S1, n=n, k=k, out_off=o, weight=f"o.w{i}") for i, (n, o) in enumerate(zip(sizes, offsets))]
    steps += [P._step(P.STEP_PRODUCT, in_buf=P.BUF_S1, out_buf=P.BUF_S3, n=11, k=40, in_off=40, out_off=5, weight="o.last")]
    m = model_of(pkg, store, steps, dtype, k, vocab=9, batch=rows)
    assert m.describe().count("\n") == 3
    m.decode(np.arange(rows) % 9)
    h = plain.rms_norm(rc.from_bf16_bits(table)[np.arange(rows) % 9], 0.0, 1e-5, 1.0)
    parts = [plain.linear(h, rc.from_bf16_bits(v)) for v in w]
    got = m.read_buffer_f32(P.BUF_S1, rows, 80)
    for part, n, o in zip(parts, sizes, offsets):
        close(got[:, o:o + n], part, dtype, slack=2.0)
    close(m.read_buffer_f32(P.BUF_S3, rows, 16)[:, 5:], plain.linear(parts[2], rc.from_bf16_bits(last)), dtype, slack=2.0)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_soft_cap(pkg, store, dtype):
    P, rng = pkg.plan, np.random.default_rng(3)
    st = P._step(P.STEP_SOFTCAP, in_buf=P.BUF_LOGITS, n=301, scale=2.5)
    m = model_of(pkg, store, [st], dtype, 8, vocab=301, batch=5)
    x = (6 * rng.standard_normal((5, 301))).astype(np.float32)
    m.write_buffer_f32(P.BUF_LOGITS, x)
    m.run_step(st)
    close(m.read_buffer_f32(P.BUF_LOGITS, 5, 301), plain.soft_cap(x.astype(np.float64), 2.5), "float32")
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [1, 2, 40, 63, 64, 65, 200, 0])
@pytest.mark.parametrize("with_sink", [True, False])
@pytest.mark.parametrize("heads, dim, vdim, rank", [(3, 24, 40, 72), (18, 128, 128, 512), (2, 11, 7, 33)])
def test_windowed_latent_attention_alone(pkg, store, dtype, window, with_sink, heads, dim, vdim, rank):
    """Decode rows at places around page and window borders, over rows that were appended before them."""
    P, n, eps, rng = pkg.plan, 150, 1e-5, np.random.default_rng(window + heads)
    nw, sink = rc.to_bf16_bits(1 + 0.3 * rng.standard_normal(rank)), rc.to_bf16_bits(2 * rng.standard_normal(heads))
    uk, uv = rc.to_bf16_bits(rng.standard_normal((heads * dim, rank)) / np.sqrt(rank)), rc.to_bf16_bits(rng.standard_normal((heads * vdim, rank)) / np.sqrt(rank))
    for name, v in (("cn", nw), ("sink", sink)):
        store.add_dense(f"w.{name}{heads}", v)
    store.add_matrix(f"w.uk{heads}", uk)
    store.add_matrix(f"w.uv{heads}", uv)
    st = P._step(P.STEP_LATENT_ATTN, layer=0, in_buf=P.BUF_S1, in2_buf=P.BUF_S3, out_buf=P.BUF_S0, n=rank, heads=heads, head_dim=dim, value_dim=vdim,
                 scale=2.0 * dim ** -0.5, eps=eps, window_left=window, weight=f"w.cn{heads}", weight2=f"w.uk{heads}", weight3=f"w.uv{heads}",
                 weight4=f"w.sink{heads}" if with_sink else "")
    m = model_of(pkg, store, [st], dtype, 8, batch=1, max_seq=n, latent_layers=1)
    q, kv = rng.standard_normal((n, heads * dim)), rng.standard_normal((n, rank))
    latent = plain.rms_norm(kv, rc.from_bf16_bits(nw), eps, 0.0)
    k, v = plain.linear(latent, rc.from_bf16_bits(uk)).reshape(n, heads, dim), plain.linear(latent, rc.from_bf16_bits(uv)).reshape(n, heads, vdim)
    scores = np.einsum("qhd,khd->hqk", act(q, dtype).reshape(n, heads, dim), k) * 2.0 * dim ** -0.5
    weights = plain.sink_softmax(scores, plain.window_mask(n, window or n), rc.from_bf16_bits(sink) if with_sink else np.full(heads, -1e30))
    want = np.einsum("hqk,khv->qhv", weights, v).reshape(n, heads * vdim)
    looked = {0, 1, 2, 62, 63, 64, 65, 127, 128, 129, 149} | {p for b in (0, 64, 128) for p in (b + window - 2, b + window - 1, b + window, b + window + 1)}
    got = {}
    for t in range(n):
        m.set_positions([t])
        m.write_buffer_f32(P.BUF_S1, q[t:t + 1])
        m.write_buffer_f32(P.BUF_S3, kv[t:t + 1])
        m.run_step(st)
        if t in looked:
            got[t] = m.read_buffer_f32(P.BUF_S0, 1, heads * vdim)[0]
    rows = sorted(got)
    close(np.array([got[t] for t in rows]), want[rows], dtype, slack=4.0)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channel", [True, False])
@pytest.mark.parametrize("heads, groups, dim, vdim, taps", [(4, 2, 48, 40, 4), (3, 1, 13, 7, 2), (2, 2, 128, 128, 4), (1, 1, 200, 136, 3), (2, 1, 272, 264, 6), (1, 1, 8, 8, 1)])
def test_gated_delta_token_by_token(pkg, store, dtype, channel, heads, groups, dim, vdim, taps):
    """Convolutions, unit norms, decays, state and gate over 40 tokens of two sequences that are one token apart."""
    P, n, eps, tag = pkg.plan, 40, 1e-5, f"d.{heads}.{dim}.{int(channel)}."
    rng = np.random.default_rng(dim)
    inputs, gk, hv = dim if channel else 1, groups * dim, heads * vdim
    w = {"conv_q": rng.standard_normal((gk, taps)), "conv_k": rng.standard_normal((gk, taps)), "conv_v": rng.standard_normal((hv, taps)),
         "norm": 1 + 0.3 * rng.standard_normal(vdim), "A_log": rng.uniform(-3, 1, heads), "dt": rng.uniform(-3, 1, heads * inputs)}
    bits = {k: rc.to_bf16_bits(v) for k, v in w.items()}
    for k, v in bits.items():
        store.add_dense(tag + k, v)
    w = {k: rc.from_bf16_bits(v) for k, v in bits.items()}
    st = P._step(P.STEP_GATED_DELTA, layer=0, in_buf=P.BUF_S1, in2_buf=P.BUF_S3, in3_buf=P.BUF_S4, in4_buf=P.BUF_S0, out_buf=P.BUF_S0, k=inputs, heads=heads, groups=groups,
                 key_dim=dim, value_dim=vdim, conv_kernel=taps, eps=eps, eps2=1e-6, scale=dim ** -0.5, gate_act=P.GATE_SIGMOID if channel else P.GATE_SILU,
                 weight=tag + "conv_q", weight2=tag + "conv_k", weight3=tag + "conv_v", weight4=tag + "norm", weight5=tag + "A_log", weight6=tag + "dt")
    m = model_of(pkg, store, [st], dtype, 8, batch=2, max_seq=64, delta_layers=1)
    qkv, beta, dec, gate = rng.standard_normal((n, 2 * gk + hv)), rng.standard_normal((n, heads)), rng.standard_normal((n, heads * inputs)), rng.standard_normal((n, hv))
    got = np.zeros((2, n, hv))
    for t in range(n + 1):   # sequence 1 is one token behind
        at = [min(t, n - 1), max(t - 1, 0)]
        if t == n:
            at[0] = 0        # (sequence 0 starts again: whatever its slot holds, position 0 begins from zeros)
        m.set_positions(at)
        for buf, x in ((P.BUF_S1, qkv), (P.BUF_S3, beta), (P.BUF_S4, dec), (P.BUF_S0, gate)):
            m.write_buffer_f32(buf, x[at])
        m.run_step(st)
        out = m.read_buffer_f32(P.BUF_S0, 2, hv)
        if t < n:
            got[0, t] = out[0]
        else:
            again = out[0]
        got[1, max(t - 1, 0)] = out[1]
    x, g8 = act(qkv, dtype), act(gate, dtype)
    q, k, v = (plain.silu(plain.short_conv(x[:, a:b], w["conv_" + c])) for c, a, b in (("q", 0, gk), ("k", gk, 2 * gk), ("v", 2 * gk, 2 * gk + hv)))
    q, k = (np.repeat(plain.unit(y.reshape(n, groups, dim)), heads // groups, axis=1) for y in (q, k))
    rate = np.exp(w["A_log"])
    decay = np.exp(-rate[:, None] * plain.softplus(dec + w["dt"]).reshape(n, heads, inputs))
    o = plain.delta_scan(q * dim ** -0.5, k, v.reshape(n, heads, vdim), np.broadcast_to(decay, (n, heads, dim)), plain.sigmoid(beta))
    want = plain.rms_norm(o, w["norm"], eps, 0.0).reshape(n, hv) * (plain.sigmoid(g8) if channel else plain.silu(g8))
    # (at the first token of a sequence sequence 1 ran twice from zeros: the same)
    close(got[0], want, dtype, slack=4.0)
    close(got[1], want, dtype, slack=4.0)
    close(again, want[0], dtype, slack=4.0)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 3, 4, 5, 17, 64])
@pytest.mark.parametrize("experts, top, groups, keep, n, k", [(12, 4, 3, 2, 160, 72), (7, 3, 1, 1, 133, 33), (64, 8, 8, 4, 264, 136), (3, 1, 3, 1, 40, 8), (5, 5, 1, 1, 96, 300), (1, 1, 1, 1, 72, 40)])
def test_routed_feed_forward_alone(pkg, store, dtype, rows, experts, top, groups, keep, n, k):
    P, rng, tag = pkg.plan, np.random.default_rng(experts + rows), f"r.{experts}.{top}.e"
    w = {}
    for e in range(experts):
        for part, shape in (("gate", (k, n)), ("up", (k, n)), ("down", (n, k))):
            b = rc.to_bf16_bits(rng.standard_normal(shape) / np.sqrt(shape[1]))
            store.add_matrix(f"{tag}{e}.{part}", b)
            w[f"e{e}.{part}"] = rc.from_bf16_bits(b)
    st = P._step(P.STEP_ROUTED_MLP, in_buf=P.BUF_S0, in2_buf=P.BUF_S3, out_buf=P.BUF_HIDDEN, n=n, k=k, experts=experts, top=top, groups=groups, groups_keep=keep,
                 scale=1.7, limit=0.8, glu_alpha=1.702, weight=tag, weight2=".gate", weight3=".up", weight4=".down")
    m = model_of(pkg, store, [st], dtype, n, batch=rows)
    x, z = act(rng.standard_normal((rows, n)), dtype), 2 * rng.standard_normal((rows, experts)).astype(np.float32).astype(np.float64)
    if rows > 4:
        z[:5] = z[0]   # several rows meet at the same experts
    m.write_buffer_f32(P.BUF_S0, x)
    m.write_buffer_f32(P.BUF_S3, z)
    for _ in range(2):   # (the second run finds what the first left in the counters)
        m.run_step(st)
        weights = plain.route(z, {"experts": experts, "top": top, "scale": 1.7, "groups": {"count": groups, "keep": keep}})
        want = sum(weights[:, e:e + 1] * plain.clamped_mlp(x, w, f"e{e}.", 0.8) for e in range(experts))
        close(m.read_buffer_f32(P.BUF_HIDDEN, rows, n), want, dtype, slack=2.0)
    m.close()


def test_equal_scores_go_to_the_lower_index(pkg, store):
    P, experts, n = pkg.plan, 6, 16
    rng = np.random.default_rng(1)
    w = {}
    for e in range(experts):
        for part in ("gate", "up", "down"):
            b = rc.to_bf16_bits(rng.standard_normal((n, n)) / 4)
            store.add_matrix(f"t.e{e}.{part}", b)
            w[f"e{e}.{part}"] = rc.from_bf16_bits(b)
    st = P._step(P.STEP_ROUTED_MLP, in_buf=P.BUF_S0, in2_buf=P.BUF_S3, out_buf=P.BUF_HIDDEN, n=n, k=n, experts=experts, top=2, groups=3, groups_keep=2,
                 scale=1.0, limit=2.0, glu_alpha=1.702, weight="t.e", weight2=".gate", weight3=".up", weight4=".down")
    for rows in (2, 6):
        m = model_of(pkg, store, [st], "float32" if rows == 2 else "bfloat16", n, batch=rows)
        z, x = np.zeros((rows, experts)), act(rng.standard_normal((rows, n)), "bfloat16")
        z[1] = [0, 0, 1, 0, 1, 0]
        m.write_buffer_f32(P.BUF_S0, x)
        m.write_buffer_f32(P.BUF_S3, z)
        m.run_step(st)
        chosen = [(0, 1)] + [(2, 4)] + [(0, 1)] * (rows - 2)
        want = np.stack([sum(0.5 * plain.clamped_mlp(x[r:r + 1], w, f"e{e}.", 2.0)[0] for e in c) for r, c in enumerate(chosen)])
        close(m.read_buffer_f32(P.BUF_HIDDEN, rows, n), want, "bfloat16", slack=2.0)
        m.close()
