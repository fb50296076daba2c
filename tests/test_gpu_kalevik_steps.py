"""The step kinds of the Kalevik recipe alone, on a GPU, against the plain implementation."""
import numpy as np
import pytest

import kalevik_cases as kc
import plain_kalevik as plain
from test_gpu_vuzunex_steps import DTYPES, act, close, model_of

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def store(pkg):
    s = pkg.WeightStore(0)
    yield s
    s.close()


def weights(store, prefix, **arrays):
    """Tensors into the store under prefix + name, matrices and vectors; their bf16 values back."""
    out = {}
    for name, x in arrays.items():
        bits = kc.to_bf16_bits(x)
        (store.add_matrix if bits.ndim == 2 else store.add_dense)(prefix + name, bits)
        out[name] = kc.from_bf16_bits(bits)
    return out


# ---- the embedding row that joins a norm ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 2, 3, 9])
@pytest.mark.parametrize("width", [24, 133, 1000])
def test_embedding_joins_in_front_of_a_norm(pkg, store, dtype, rows, width):
    """Alone, and in the prologue of the product behind it."""
    P, rng, eps, scale, n = pkg.plan, np.random.default_rng(width + rows), 0.03, 1.75, 20
    p = f"j{width}."
    table = kc.to_bf16_bits(rng.standard_normal((11, width)))
    store.add_dense(p + "e", table)
    w = weights(store, p, a=1 + 0.3 * rng.standard_normal(width), b=1 + 0.3 * rng.standard_normal(width), m=rng.standard_normal((n, width)) / np.sqrt(width))
    norm = P._step(P.STEP_POSTNORM_RESADD_COPY_RMSNORM, in_buf=P.BUF_HIDDEN, out_buf=P.BUF_S0, n=width, eps=eps, scale=scale, weight=p + "a", weight2=p + "b", weight3=p + "e")
    steps = [P._step(P.STEP_EMBED, out_buf=P.BUF_HIDDEN, n=width, scale=scale, weight=p + "e"),
             P._step(P.STEP_COPY_RMSNORM, in_buf=P.BUF_HIDDEN, out_buf=P.BUF_S0, n=width, eps=eps, weight=p + "b"), norm,
             P._step(P.STEP_PRODUCT, in_buf=P.BUF_S0, out_buf=P.BUF_S1, n=n, k=width, weight=p + "m")]
    m = model_of(pkg, store, steps, dtype, width, vocab=11, batch=rows)
    assert "postnorm+rmsnorm" in m.describe() and m.describe().count("\n") == 3
    tokens = (3 * np.arange(rows) + 2) % 11
    m.decode(tokens)
    start = kc.from_bf16_bits(table)[tokens] * scale
    stream = start + plain.rms_norm(start, w["a"], eps) + start   # (the hidden buffer still holds the embedding)
    want = plain.linear(plain.rms_norm(stream, w["b"], eps), w["m"])
    close(m.read_buffer_f32(P.BUF_S1, rows, n), want, dtype, slack=3.0)
    close(m.read_buffer_f32(P.BUF_RESIDUAL, rows, width), stream, "float32")
    m.close()
    m = model_of(pkg, store, [norm], dtype, width, vocab=11, batch=rows)
    x, res = rng.standard_normal((rows, width)).astype(np.float32), (3 * rng.standard_normal((rows, width))).astype(np.float32)
    m.write_buffer_f32(P.BUF_HIDDEN, x)
    m.write_buffer_f32(P.BUF_RESIDUAL, res)
    m.run_step(norm, token_in=tokens)
    stream = res + plain.rms_norm(x.astype(np.float64), w["a"], eps) + start
    close(m.read_buffer_f32(P.BUF_S0, rows, width), plain.rms_norm(stream, w["b"], eps), dtype)
    m.close()


# ---- two matrices side by side -------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 4, 5, 40])
@pytest.mark.parametrize("n, k, k2", [(37, 13, 21), (132, 200, 64), (40, 8, 8), (300, 512, 1000)])
def test_product_over_two_matrices(pkg, store, dtype, rows, n, k, k2):
    P, rng, p = pkg.plan, np.random.default_rng(n + rows), f"two{n}."
    w = weights(store, p, a=rng.standard_normal((n, k)) / np.sqrt(k), b=rng.standard_normal((n, k2)) / np.sqrt(k2))
    at = -(-k // 8) * 8
    st = P._step(P.STEP_PRODUCT, in_buf=P.BUF_S0, out_buf=P.BUF_HIDDEN, n=n, k=k, k2=k2, weight=p + "a", weight2=p + "b")
    m = model_of(pkg, store, [st], dtype, n, batch=rows)
    x = act(rng.standard_normal((rows, at + k2)), dtype)
    m.write_buffer_f32(P.BUF_S0, x)
    m.run_step(st)
    close(m.read_buffer_f32(P.BUF_HIDDEN, rows, n), plain.linear(x[:, :k], w["a"]) + plain.linear(x[:, at:], w["b"]), dtype)
    # new values in the old places
    w = weights(store, p, a=rng.standard_normal((n, k)) / np.sqrt(k), b=rng.standard_normal((n, k2)) / np.sqrt(k2))
    m.run_step(st)
    close(m.read_buffer_f32(P.BUF_HIDDEN, rows, n), plain.linear(x[:, :k], w["a"]) + plain.linear(x[:, at:], w["b"]), dtype)
    m.close()


# ---- latent attention with neighbouring pairs ----------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("pairs", [0, 1])
@pytest.mark.parametrize("heads, dim, rot, vdim, rank, turned", [(3, 24, 8, 40, 72, 8), (18, 128, 64, 128, 512, 64), (2, 11, 6, 7, 33, 4)])
def test_rotations_of_latent_attention(pkg, store, dtype, pairs, heads, dim, rot, vdim, rank, turned):
    P, n, eps, rng, p, base, divisor = pkg.plan, 70, 1e-5, np.random.default_rng(heads), f"la{heads}.", 300.0, 1.5
    w = weights(store, p, cn=1 + 0.3 * rng.standard_normal(rank), uk=rng.standard_normal((heads * dim, rank)) / np.sqrt(rank), uv=rng.standard_normal((heads * vdim, rank)) / np.sqrt(rank))
    scale = 2.0 * (dim + rot) ** -0.5
    st = P._step(P.STEP_LATENT_ATTN, layer=0, in_buf=P.BUF_S1, in2_buf=P.BUF_S3, out_buf=P.BUF_S0, n=rank, heads=heads, head_dim=dim, key_dim=rot, value_dim=vdim,
                 rope_dim=turned, rope_base=base, rope_pairs=pairs, rope_divisor=divisor, scale=scale, eps=eps, weight=p + "cn", weight2=p + "uk", weight3=p + "uv")
    m = model_of(pkg, store, [st], dtype, 8, batch=1, max_seq=n, latent_layers=1)
    q, kv = rng.standard_normal((n, heads * (dim + rot))), rng.standard_normal((n, rank + rot))

    def turn(x):
        if pairs == 0:
            return plain.rotate_halves(x, turned, base, divisor)
        a = plain.angles(n, turned, base, divisor)[:, None, :]
        out = x.copy()
        u, v = x[..., 0:turned:2], x[..., 1:turned:2]
        out[..., 0:turned:2], out[..., 1:turned:2] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
        return out

    qr = act(q, dtype).reshape(n, heads, dim + rot)
    c = plain.rms_norm(kv[:, :rank], w["cn"], eps)
    k, v = plain.linear(c, w["uk"]).reshape(n, heads, dim), plain.linear(c, w["uv"]).reshape(n, heads, vdim)
    scores = np.einsum("qhd,khd->hqk", qr[:, :, :dim], k) + np.einsum("qhd,kd->hqk", turn(qr[:, :, dim:]), turn(kv[:, None, rank:])[:, 0])
    want = np.einsum("hqk,khv->qhv", plain.masked_softmax(scores * scale, plain.causal_mask(n)), v).reshape(n, heads * vdim)
    got = np.zeros_like(want)
    for t in range(n):
        m.set_positions([t])
        m.write_buffer_f32(P.BUF_S1, q[t:t + 1])
        m.write_buffer_f32(P.BUF_S3, kv[t:t + 1])
        m.run_step(st)
        got[t] = m.read_buffer_f32(P.BUF_S0, 1, heads * vdim)[0]
    close(got, want, dtype, slack=4.0)
    m.close()


# ---- grouped attention ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("chunk, window", [(1, 0), (2, 0), (40, 0), (63, 0), (64, 0), (65, 0), (200, 0), (0, 0), (0, 50), (60, 33)])
@pytest.mark.parametrize("heads, kv, dim, vdim, turned", [(4, 2, 24, 40, 16), (20, 1, 128, 128, 128), (3, 3, 11, 7, 6), (2, 1, 200, 136, 48), (2, 1, 264, 272, 0)])
def test_grouped_attention_alone(pkg, store, dtype, chunk, window, heads, kv, dim, vdim, turned):
    """Decode rows at places around page, chunk and window borders, over rows that were appended before them. Norms, sink, gate,
    columns and the scaling of the result come and go with the sizes."""
    P, n, eps, rng, p = pkg.plan, 150, 1e-3, np.random.default_rng(chunk + heads), f"ga{heads}.{dim}."
    normed, sink, gated, at_in, at_out = dim != 11, dim != 128, heads != 2, 8 * (heads % 3), 16 * (kv % 2)
    w = weights(store, p, qn=1 + 0.3 * rng.standard_normal(dim), kn=1 + 0.3 * rng.standard_normal(dim))
    base, divisor, scale, out_scale = 200.0, 2.5, 2.0 * dim ** -0.5, -0.7
    st = P._step(P.STEP_GROUPED_ATTN, layer=0, in_buf=P.BUF_S1, in_off=at_in, in3_buf=P.BUF_S4 if gated else -1, out_buf=P.BUF_S0, out_off=at_out, heads=heads, kv_heads=kv,
                 head_dim=dim, value_dim=vdim, rope_dim=turned, rope_base=base, rope_divisor=divisor, scale=scale, eps=eps, chunk=chunk, window_left=window,
                 sink_one=int(sink), out_scale=out_scale, weight=p + "qn" if normed else "", weight2=p + "kn" if normed else "")
    m = model_of(pkg, store, [st], dtype, 8, batch=1, max_seq=n, grouped_layers=1)
    x = rng.standard_normal((n, (heads + kv) * dim + kv * vdim))
    z = rng.standard_normal((n, heads))
    y = act(x, dtype)
    q, k, v = y[:, :heads * dim].reshape(n, heads, dim), y[:, heads * dim:(heads + kv) * dim].reshape(n, kv, dim), y[:, (heads + kv) * dim:].reshape(n, kv, vdim)
    if normed:
        q, k = plain.rms_norm(q, w["qn"], eps), plain.rms_norm(k, w["kn"], eps)
    if turned:
        q, k = (plain.rotate_halves(a, turned, base, divisor) for a in (q, k))
    q, k, v = act(q, dtype), np.repeat(act(k, dtype), heads // kv, axis=1), np.repeat(v, heads // kv, axis=1)
    i = np.arange(n)
    seen = plain.chunk_mask(n, chunk) if chunk else plain.causal_mask(n)
    if window:
        seen = seen & (i[:, None] - i[None, :] < window)
    weight = (plain.softmax_plus_one if sink else plain.masked_softmax)(np.einsum("qhd,khd->hqk", q, k) * scale, seen)
    want = np.einsum("hqk,khv->qhv", weight, v) * out_scale
    if gated:
        want = want * plain.sigmoid(z)[:, :, None]
    want = want.reshape(n, heads * vdim)
    step = max(chunk, window, 1)
    looked = {0, 1, 2, 62, 63, 64, 65, 127, 128, 129, 149} | {b + d for b in (0, 64, 128) + tuple(range(0, n, step))[:5] for d in (step - 2, step - 1, step, step + 1)}
    got = {}
    for t in range(n):
        m.set_positions([t])
        m.write_buffer_f32(P.BUF_S1, np.concatenate([np.zeros((1, at_in)), x[t:t + 1]], axis=1))
        if gated:
            m.write_buffer_f32(P.BUF_S4, z[t:t + 1])
        m.run_step(st)
        if t in looked:
            got[t] = m.read_buffer_f32(P.BUF_S0, 1, at_out + heads * vdim)[0, at_out:]
    rows = sorted(got)
    close(np.array([got[t] for t in rows]), want[rows], dtype, slack=4.0)
    m.close()


# ---- retention -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dim, vdim", [(4, 48, 40), (3, 13, 7), (2, 128, 128), (1, 200, 136), (2, 264, 40), (1, 40, 296), (1, 8, 8)])
def test_retention_token_by_token(pkg, store, dtype, heads, dim, vdim):
    """State, read-out, norm and gate over 40 tokens of two sequences that are one token apart."""
    P, n, eps, p = pkg.plan, 40, 1e-3, f"rt{heads}.{dim}."
    rng = np.random.default_rng(dim)
    decay = np.array([0.999, 0.5, 0.0, 0.9])[:heads].astype(np.float32)
    store.add_dense_f32(p + "decay", decay)
    qk, hv, gate_at, out_at, out_scale = heads * dim, heads * vdim, 8, 16, 1.3
    st = P._step(P.STEP_RETENTION, layer=0, in_buf=P.BUF_S2, in_off=8, in4_buf=P.BUF_S1, in4_off=gate_at, out_buf=P.BUF_S0, out_off=out_at, heads=heads, key_dim=dim, value_dim=vdim,
                 scale=dim ** -0.5, eps=eps, out_scale=out_scale, weight=p + "decay")
    m = model_of(pkg, store, [st], dtype, 8, batch=2, max_seq=64, delta_layers=1)
    x, gate = rng.standard_normal((n, 2 * qk + hv)), rng.standard_normal((n, hv))
    got = np.zeros((2, n, hv))
    for t in range(n + 1):   # sequence 1 is one token behind
        at = [min(t, n - 1), max(t - 1, 0)]
        if t == n:
            at[0] = 0        # (sequence 0 starts again: whatever its slot holds, position 0 begins from zeros)
        m.set_positions(at)
        m.write_buffer_f32(P.BUF_S2, np.concatenate([np.zeros((2, 8)), x[at]], axis=1))
        m.write_buffer_f32(P.BUF_S1, np.concatenate([np.zeros((2, gate_at)), gate[at]], axis=1))
        m.run_step(st)
        out = m.read_buffer_f32(P.BUF_S0, 2, out_at + hv)[:, out_at:]
        if t < n:
            got[0, t] = out[0]
        else:
            again = out[0]
        got[1, max(t - 1, 0)] = out[1]
    y = act(x, dtype)
    q, k, v = y[:, :qk].reshape(n, heads, dim), y[:, qk:2 * qk].reshape(n, heads, dim) * dim ** -0.5, y[:, 2 * qk:].reshape(n, heads, vdim)
    o = plain.rms_unit(plain.retention_scan(q, k, v, decay.astype(np.float64)), eps).reshape(n, hv)
    want = o * plain.silu(act(gate, dtype)) * out_scale
    # (at the first token of a sequence sequence 1 ran twice from zeros: the same)
    close(got[0], want, dtype, slack=4.0)
    close(got[1], want, dtype, slack=4.0)
    close(again, want[0], dtype, slack=4.0)
    m.close()


# ---- routed feed-forward -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 3, 4, 5, 17, 64])
@pytest.mark.parametrize("experts, top, groups, keep, n, k, shared", [(12, 4, 3, 2, 160, 72, 96), (7, 3, 1, 1, 133, 33, 19), (64, 8, 8, 4, 264, 136, 0), (3, 1, 3, 1, 40, 8, 300), (5, 5, 1, 1, 96, 300, 8), (1, 1, 1, 1, 72, 40, 40)])
def test_routed_feed_forward_alone(pkg, store, dtype, rows, experts, top, groups, keep, n, k, shared):
    P, rng, p = pkg.plan, np.random.default_rng(experts + rows), f"sm.{experts}.{top}."
    w = {}
    for e in range(experts):
        for part, shape in (("up", (k, n)), ("down", (n, k))):
            b = kc.to_bf16_bits(rng.standard_normal(shape) / np.sqrt(shape[1]))
            store.add_matrix(f"{p}e{e}.{part}", b)
            w[f"e{e}.{part}"] = kc.from_bf16_bits(b)
    extra = {}
    if shared:
        w.update({"shared." + a: v for a, v in weights(store, p + "shared.", up=rng.standard_normal((shared, n)) / np.sqrt(n), down=rng.standard_normal((n, shared)) / np.sqrt(shared)).items()})
        extra = dict(weight5=p + "shared.up", weight6=p + "shared.down", k2=shared)
    st = P._step(P.STEP_ROUTED_MLP, in_buf=P.BUF_S0, in2_buf=P.BUF_S3, out_buf=P.BUF_HIDDEN, n=n, k=k, experts=experts, top=top, groups=groups, groups_keep=keep,
                 scale=1.0, score_act=P.SCORE_SOFTMAX, group_best=1, raw_weights=1, weight=p + "e", weight3=".up", weight4=".down", **extra)
    m = model_of(pkg, store, [st], dtype, n, batch=rows)
    x, z = act(rng.standard_normal((rows, n)), dtype), 2 * rng.standard_normal((rows, experts + 1)).astype(np.float32).astype(np.float64)
    if rows > 4:
        z[:5] = z[0]   # several rows meet at the same experts
    m.write_buffer_f32(P.BUF_S0, x)
    m.write_buffer_f32(P.BUF_S3, z[:, :experts + (1 if shared else 0)])
    weight = plain.route(z[:, :experts], {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}})
    want = sum(weight[:, e:e + 1] * plain.expert(x, w, f"e{e}.") for e in range(experts))
    if shared:
        want = want + plain.sigmoid(z[:, experts:]) * plain.expert(x, w, "shared.")
    for _ in range(2):   # (the second run finds what the first left in the counters)
        m.run_step(st)
        close(m.read_buffer_f32(P.BUF_HIDDEN, rows, n), want, dtype, slack=2.0)
    m.close()


@pytest.mark.parametrize("rows", [2, 7])
def test_far_apart_logits(pkg, store, rows):
    """Scores that underflow still rank, and a softmax over large logits stays finite."""
    P, n, experts, rng = pkg.plan, 16, 6, np.random.default_rng(4)
    w = {}
    for e in range(experts):
        for part in ("up", "down"):
            b = kc.to_bf16_bits(rng.standard_normal((n, n)) / 4)
            store.add_matrix(f"fa.e{e}.{part}", b)
            w[f"e{e}.{part}"] = kc.from_bf16_bits(b)
    st = P._step(P.STEP_ROUTED_MLP, in_buf=P.BUF_S0, in2_buf=P.BUF_S3, out_buf=P.BUF_HIDDEN, n=n, k=n, experts=experts, top=2, groups=3, groups_keep=2,
                 scale=1.0, score_act=P.SCORE_SOFTMAX, group_best=1, raw_weights=1, weight="fa.e", weight3=".up", weight4=".down")
    m = model_of(pkg, store, [st], "bfloat16", n, batch=rows)
    z, x = np.tile([500.0, -500.0, 499.0, 0.0, 100.0, 100.0], (rows, 1)), act(rng.standard_normal((rows, n)), "bfloat16")
    z[1] = 300.0
    m.write_buffer_f32(P.BUF_S0, x)
    m.write_buffer_f32(P.BUF_S3, z)
    m.run_step(st)
    a = 1.0 / (1.0 + np.exp(-1.0))
    want = a * plain.expert(x, w, "e0.") + (1.0 - a) * plain.expert(x, w, "e2.")
    want[1] = (plain.expert(x[1:2], w, "e0.") + plain.expert(x[1:2], w, "e1."))[0] / 6.0   # equal scores go to the lower index
    close(m.read_buffer_f32(P.BUF_HIDDEN, rows, n), want, "bfloat16", slack=2.0)
    m.close()
