"""Every step kind of fp32-stream plans alone, on a GPU, against the plain implementation."""
import numpy as np
import pytest

import plain_vuzunex as plain
import vuzunex_cases as vc

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
LIMIT = {"float32": 3e-6, "bfloat16": 6e-3}   # of the largest magnitude


def dtype_id(pkg, dtype):
    return pkg.plan.STREAM_ALL_F32 if dtype == "float32" else pkg.plan.STREAM_F32


def act(x, dtype):
    """What an activation buffer keeps of x."""
    return np.asarray(x, dtype=np.float32).astype(np.float64) if dtype == "float32" else vc.from_bf16_bits(vc.to_bf16_bits(x))


def close(got, want, dtype, slack=1.0):
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)
    assert err <= slack * LIMIT[dtype], err


@pytest.fixture(scope="module")
def store(pkg):
    s = pkg.WeightStore(0)
    yield s
    s.close()


def model_of(pkg, store, steps, dtype, hidden, vocab=8, batch=3, **kw):
    desc = pkg.plan.BuffersDesc(hidden=hidden, vocab=vocab, max_seq=kw.pop("max_seq", 64), max_batch=batch, stream_dtype=dtype_id(pkg, dtype), **kw)
    return pkg.InferenceModel(store, steps, desc)


@pytest.mark.parametrize("dtype", DTYPES)
def test_embedding_times_scale(pkg, store, dtype):
    P, rng = pkg.plan, np.random.default_rng(1)
    table = vc.to_bf16_bits(rng.standard_normal((37, 52)))
    store.add_dense("t.embed", table)
    m = model_of(pkg, store, [P._step(P.STEP_EMBED, out_buf=P.BUF_HIDDEN, n=52, scale=7.25, weight="t.embed")], dtype, 52, vocab=37)
    m.run_step(P._step(P.STEP_EMBED, out_buf=P.BUF_HIDDEN, n=52, scale=7.25, weight="t.embed"), token_in=[36, 0, 5])
    assert np.array_equal(m.read_buffer_f32(P.BUF_HIDDEN, 3, 52), (plain.embed_rows(vc.from_bf16_bits(table), [36, 0, 5], 7.25)).astype(np.float32))
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [24, 132, 1000])
@pytest.mark.parametrize("kind", ["copy", "add", "add_last", "post", "post_last"])
def test_norms(pkg, store, dtype, width, kind):
    P, rng, eps, bias = pkg.plan, np.random.default_rng(width), 0.05, 1.0
    wa, wb = vc.to_bf16_bits(0.3 * rng.standard_normal(width)), vc.to_bf16_bits(0.3 * rng.standard_normal(width))
    store.add_dense(f"t.na{width}", wa)
    store.add_dense(f"t.nb{width}", wb)
    number = {"copy": P.STEP_COPY_RMSNORM, "add": P.STEP_RESADD_COPY_RMSNORM, "add_last": P.STEP_RESADD_RMSNORM,
              "post": P.STEP_POSTNORM_RESADD_COPY_RMSNORM, "post_last": P.STEP_POSTNORM_RESADD_RMSNORM}[kind]
    post = kind.startswith("post")
    st = P._step(number, in_buf=P.BUF_HIDDEN, out_buf=P.BUF_S0, n=width, eps=eps, weight_bias=bias, weight=f"t.na{width}",
                 **(dict(weight2=f"t.nb{width}") if post else {}))
    m = model_of(pkg, store, [st], dtype, width)
    x, res = rng.standard_normal((3, width)).astype(np.float32), (5 * rng.standard_normal((3, width))).astype(np.float32)
    x[1] *= 1e-3   # eps matters
    m.write_buffer_f32(P.BUF_HIDDEN, x)
    m.write_buffer_f32(P.BUF_RESIDUAL, res)
    m.run_step(st)
    fa, fb, x, res = vc.from_bf16_bits(wa), vc.from_bf16_bits(wb), x.astype(np.float64), res.astype(np.float64)
    h = x if kind == "copy" else res + (plain.rms_norm(x, fa, eps, bias) if post else x)
    close(m.read_buffer_f32(P.BUF_S0, 3, width), plain.rms_norm(h, fb if post else fa, eps, bias), dtype)
    close(m.read_buffer_f32(P.BUF_RESIDUAL, 3, width), res if kind.endswith("last") else h, "float32")
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 2, 3, 4, 5, 16, 33, 64])
@pytest.mark.parametrize("n, k", [(7, 9), (300, 132), (129, 72), (264, 1000), (40, 3000)])
def test_product(pkg, store, dtype, rows, n, k):
    P, rng = pkg.plan, np.random.default_rng(n)
    w = vc.to_bf16_bits(rng.standard_normal((n, k)) / np.sqrt(k))
    store.add_matrix(f"t.w{n}x{k}", w)
    for dst in (P.BUF_S1, P.BUF_HIDDEN):   # activation type and fp32
        st = P._step(P.STEP_PRODUCT, in_buf=P.BUF_S0, out_buf=dst, n=n, k=k, weight=f"t.w{n}x{k}")
        m = model_of(pkg, store, [st], dtype, n, batch=rows)
        x = rng.standard_normal((rows, k)).astype(np.float32)
        m.write_buffer_f32(P.BUF_S0, x)
        m.run_step(st)
        want = plain.linear(act(x, dtype), vc.from_bf16_bits(w))
        close(m.read_buffer_f32(dst, rows, n), want, "float32" if dst == P.BUF_HIDDEN else dtype, slack=2.0)
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 2, 4, 6, 40])
@pytest.mark.parametrize("act_name, n, k", [("geglu", 37, 52), ("geglu", 400, 264), ("swiglu", 130, 72)])
def test_gate_and_up_in_one_launch(pkg, store, dtype, rows, act_name, n, k):
    """gate, up and activation as a plan compiles them, with the norm in front."""
    P, rng = pkg.plan, np.random.default_rng(n + k)
    g, u = (vc.to_bf16_bits(2 * rng.standard_normal((n, k)) / np.sqrt(k)) for _ in range(2))
    head, table, nw = vc.to_bf16_bits(rng.standard_normal((n, n)) / np.sqrt(n)), vc.to_bf16_bits(rng.standard_normal((16, k))), vc.to_bf16_bits(0.2 * rng.standard_normal(k))
    for name, v in ((f"t.g{n}", g), (f"t.u{n}", u), (f"t.h{n}", head)):
        store.add_matrix(name, v)
    store.add_dense(f"t.e{n}", table)
    store.add_dense(f"t.n{n}", nw)
    steps = [P._step(P.STEP_EMBED, out_buf=P.BUF_HIDDEN, n=k, weight=f"t.e{n}"),
             P._step(P.STEP_COPY_RMSNORM, in_buf=P.BUF_HIDDEN, out_buf=P.BUF_S0, n=k, eps=1e-5, weight_bias=1.0, weight=f"t.n{n}"),
             P._step(P.STEP_PRODUCT, in_buf=P.BUF_S0, out_buf=P.BUF_S1, n=n, k=k, weight=f"t.g{n}"),
             P._step(P.STEP_PRODUCT, in_buf=P.BUF_S0, out_buf=P.BUF_S2, n=n, k=k, weight=f"t.u{n}"),
             P._step(P.STEP_GEGLU if act_name == "geglu" else P.STEP_SWIGLU, in_buf=P.BUF_S1, in2_buf=P.BUF_S2, out_buf=P.BUF_S1, n=n)]
    m = model_of(pkg, store, steps, dtype, k, vocab=16, batch=rows)
    assert m.describe().count("\n") == 2 and "product+gate" in m.describe()
    m.decode(np.arange(rows) % 16)
    h = plain.rms_norm(vc.from_bf16_bits(table)[np.arange(rows) % 16], vc.from_bf16_bits(nw), 1e-5, 1.0)
    a, b = plain.linear(h, vc.from_bf16_bits(g)), plain.linear(h, vc.from_bf16_bits(u))
    want = (plain.gelu_tanh(a) if act_name == "geglu" else a * plain.sigmoid(a)) * b
    close(m.read_buffer_f32(P.BUF_S1, rows, n), want, dtype, slack=2.0)
    m.close()
    # the activation on its own
    st = steps[-1]
    m = model_of(pkg, store, [st], dtype, k, batch=rows)
    x, y = 3 * rng.standard_normal((rows, n)), rng.standard_normal((rows, n))
    m.write_buffer_f32(P.BUF_S1, x)
    m.write_buffer_f32(P.BUF_S2, y)
    m.run_step(st)
    x, y = act(x, dtype), act(y, dtype)
    close(m.read_buffer_f32(P.BUF_S1, rows, n), (plain.gelu_tanh(x) if act_name == "geglu" else x * plain.sigmoid(x)) * y, dtype, slack=1.5)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_argmax_takes_the_lowest_of_equal_logits(pkg, store, dtype):
    P, rng = pkg.plan, np.random.default_rng(4)
    m = model_of(pkg, store, [P._step(P.STEP_ARGMAX, in_buf=P.BUF_LOGITS, n=1003)], dtype, 8, vocab=1003, batch=5)
    x = rng.standard_normal((5, 1003)).astype(np.float32)
    x[1, [700, 31, 990]] = 9.0
    x[2, 1002] = 1e-6 + x[2].max()
    m.write_buffer_f32(P.BUF_LOGITS, x)
    assert m.run_step(P._step(P.STEP_ARGMAX, in_buf=P.BUF_LOGITS, n=1003)).tolist() == np.argmax(x, axis=1).tolist()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("gated", [True, False])
@pytest.mark.parametrize("name", ["mid", "odd", "wide", "huge"])
def test_latent_attention_alone(pkg, store, dtype, gated, name):
    """One attention step at a time over 70 positions: cached rows, rotation, scores, values, gate."""
    P, lay = pkg.plan, vc.cases()[name]["layers"][0]["mixer"]
    heads, dim, rot, vdim, rank = lay["heads"], lay["dim"], lay["rot_dim"], lay["vdim"], lay["kv_rank"]
    n, seqs, eps, rng = 70, 2, 1e-5, np.random.default_rng(11)
    nw = vc.to_bf16_bits(1 + 0.3 * rng.standard_normal(rank))
    uk, uv = vc.to_bf16_bits(rng.standard_normal((heads * dim, rank)) / np.sqrt(rank)), vc.to_bf16_bits(rng.standard_normal((heads * vdim, rank)) / np.sqrt(rank))
    store.add_dense(f"t.cn{name}", nw)
    store.add_matrix(f"t.uk{name}", uk)
    store.add_matrix(f"t.uv{name}", uv)
    sc = lay["rot"].get("scaling")
    st = P._step(P.STEP_LATENT_ATTN, layer=0, in_buf=P.BUF_S1, in2_buf=P.BUF_S3, in3_buf=P.BUF_S4 if gated else -1, out_buf=P.BUF_S0, n=rank, heads=heads,
                 head_dim=dim, key_dim=rot, value_dim=vdim, rope_dim=lay["rot"]["dims"], rope_base=lay["rot"]["base"], scale=2 * lay["scale"], eps=eps,
                 weight=f"t.cn{name}", weight2=f"t.uk{name}", weight3=f"t.uv{name}",
                 **({} if sc is None else dict(rope_factor=sc["factor"], rope_original=sc["original"], rope_fast=sc["fast"], rope_slow=sc["slow"])))
    m = model_of(pkg, store, [st], dtype, 8, batch=seqs, max_seq=n, latent_layers=1)
    q, kv, g = rng.standard_normal((seqs, n, heads * (dim + rot))), rng.standard_normal((seqs, n, rank + rot)), rng.standard_normal((seqs, n, heads))
    got = np.empty((seqs, n, heads * vdim))
    for t in range(n):
        m.set_positions([t] * seqs)
        m.write_buffer_f32(P.BUF_S1, q[:, t])
        m.write_buffer_f32(P.BUF_S3, kv[:, t])
        if gated:
            m.write_buffer_f32(P.BUF_S4, g[:, t])
        m.run_step(st)
        got[:, t] = m.read_buffer_f32(P.BUF_S0, seqs, heads * vdim)
    pos, turn = np.arange(n), dict(dims=lay["rot"]["dims"], base=lay["rot"]["base"], scaling=sc)
    for b in range(seqs):
        x = act(q[b], dtype).reshape(n, heads, dim + rot)
        latent = plain.rms_norm(kv[b, :, :rank], vc.from_bf16_bits(nw), eps, 0.0)
        k_turned = plain.rotate(kv[b, :, rank:], pos, **turn)
        cached = m.read_latent(0, b, n, rank + rot)
        close(cached, np.concatenate([latent, k_turned], axis=1), dtype)
        scores = (np.einsum("qhd,khd->hqk", x[..., :dim], plain.linear(latent, vc.from_bf16_bits(uk)).reshape(n, heads, dim)) +
                  np.einsum("qhd,kd->hqk", plain.rotate(x[..., dim:], pos, **turn), k_turned)) * 2 * lay["scale"]
        want = np.einsum("hqk,khv->qhv", plain.causal_softmax(scores), plain.linear(latent, vc.from_bf16_bits(uv)).reshape(n, heads, vdim))
        if gated:
            want = want * plain.sigmoid(g[b])[:, :, None]
        close(got[b], want.reshape(n, heads * vdim), dtype, slack=4.0)
    m.close()
