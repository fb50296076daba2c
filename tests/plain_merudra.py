"""Plain, slow statement of the Merudra design in numpy, one function per mechanism. Test infrastructure only: it shares no code
with the package (no import of it, no kernels), works on whole sequences without any cache or carried state, and computes in
whatever floating type its inputs have (float64 by default).

Weights are a dict name -> float array under the names of a checkpoint (`embed`, `side.embed`, `l0.norm1`, ..., `head`).
"""
import numpy as np


# ---- shapes --------------------------------------------------------------------------------------------------------
def mixer_shapes(layer, width):
    """Suffix -> shape of a mixer's tensors."""
    m = layer["mixer"]
    heads, kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    if layer["type"] == "attention":
        return {"q": (heads * dim, width), "q.b": (heads * dim,), "k": (kv * dim, width), "k.b": (kv * dim,),
                "g": (heads * vdim, width), "o": (width, heads * vdim)}
    out = {}
    for name, rows in (("q", kv * dim), ("k", kv * dim), ("v", heads * vdim)):
        out[name], out[name + ".conv"] = (rows, width), (rows, m["conv"])
    out.update({"b": (heads, width), "a": (heads, width), "A_log": (heads,), "dt_bias": (heads,), "norm": (vdim,),
                "g": (heads * vdim, width), "o": (width, heads * vdim)})
    return out


def tensor_shapes(config):
    """name -> shape of every tensor a checkpoint of this configuration holds."""
    width, taps, side, layers = config["width"], config["canon"]["taps"], config["token_side"]["dim"], config["layers"]
    out = {"embed": (config["vocab"], width), "side.embed": (config["vocab"], len(layers) * side)}
    for i, layer in enumerate(layers):
        p, mlp = f"l{i}.", layer.get("mlp")
        out.update({p + "mix." + k: v for k, v in mixer_shapes(layer, width).items()})
        for j in ("1", "2") if mlp else ("1",):
            out.update({p + "norm" + j: (width,), p + "canon" + j: (width, taps), p + "rg" + j: (width, width), p + f"rg{j}.b": (width,)})
        out.update({p + "dwa": (i + 2,), p + "side.gate": (side, width), p + "side.proj": (width, side), p + "side.norm": (width,)})
        if mlp:
            router, ff = mlp["router"], mlp["expert"]["ff"]
            for e in range(router["experts"]):
                out[f"{p}mlp.e{e}.gate"] = out[f"{p}mlp.e{e}.up"] = (ff, width)
                out[f"{p}mlp.e{e}.down"] = (width, ff)
            scored = router["experts"] + router["identity"]
            out.update({p + "mlp.router": (scored, width), p + "mlp.correction": (scored,)})
    out["final.norm"] = (width,)
    out["head"] = (config["vocab"], width)
    return out


# ---- small parts ---------------------------------------------------------------------------------------------------
def linear(x, weight, bias=0.0):
    return x @ weight.T + bias


def over_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, weight, eps):
    return over_rms(x, eps) * weight


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.logaddexp(0.0, z)


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def short_conv(x, taps):
    """x [tokens, channels], taps [channels, count]: causal, the last tap meets the current token, zeros before the start."""
    n, count = x.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((count - 1, x.shape[1]), dtype=x.dtype), x])
    return sum(padded[j:j + n] * taps[:, j] for j in range(count))


# ---- attention -----------------------------------------------------------------------------------------------------
def causal_softmax(scores):
    """scores [heads, query, key]."""
    n = scores.shape[-1]
    s = np.where(np.tril(np.ones((n, n), dtype=bool))[None], scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def query_temperature(n, coef, every):
    """Factor of the query at positions 0 .. n - 1."""
    return 1.0 + coef * np.log(np.floor((np.arange(n) + 1) / every) + 1.0)


def attention(h, w, p, m, eps):
    """Grouped-query attention without rotation whose values are the keys as projected."""
    n, heads, kv, dim = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = over_rms(linear(h, w[p + "q"], w[p + "q.b"]).reshape(n, heads, dim), eps)
    q = q * query_temperature(n, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None, None]
    v = np.repeat(linear(h, w[p + "k"], w[p + "k.b"]).reshape(n, kv, dim), heads // kv, axis=1)
    weights = causal_softmax(np.einsum("qhd,khd->hqk", q, over_rms(v, eps)) * m["scale"])
    o = np.einsum("hqk,khv->qhv", weights, v).reshape(n, heads * dim)
    return linear(o * sigmoid(linear(h, w[p + "g"])), w[p + "o"])


# ---- gated delta rule ----------------------------------------------------------------------------------------------
def delta_scan(q, k, v, g, beta):
    """q, k [tokens, heads, dim], v [tokens, heads, vdim], g and beta [tokens, heads]: the state is decayed, corrected towards v
    along k, then read with q."""
    n, heads, dim = k.shape
    state = np.zeros((heads, dim, v.shape[2]), dtype=v.dtype)
    out = np.empty_like(v)
    for t in range(n):
        state = g[t][:, None, None] * state
        miss = v[t] - np.einsum("hdv,hd->hv", state, k[t])
        state = state + k[t][:, :, None] * (beta[t][:, None] * miss)[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", state, q[t])
    return out


def delta_mixer(h, w, p, m, eps):
    n, heads, kv, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(linear(h, w[p + t]), w[p + t + ".conv"])) for t in "qkv")
    q = np.repeat(unit(q.reshape(n, kv, dim)) * dim ** -0.5, heads // kv, axis=1)
    k = np.repeat(unit(k.reshape(n, kv, dim)), heads // kv, axis=1)
    g = np.exp(-np.exp(w[p + "A_log"]) * softplus(linear(h, w[p + "a"]) + w[p + "dt_bias"]))
    o = rms_norm(delta_scan(q, k, v.reshape(n, heads, vdim), g, sigmoid(linear(h, w[p + "b"]))), w[p + "norm"], eps)
    return linear(o.reshape(n, heads * vdim) * silu(linear(h, w[p + "g"])), w[p + "o"])


def mixer(h, w, p, layer, eps):
    return (attention if layer["type"] == "attention" else delta_mixer)(h, w, p, layer["mixer"], eps)


# ---- feed-forward --------------------------------------------------------------------------------------------------
def route(z, correction, top):
    """z [tokens, scored] -> weights [tokens, scored], zero where an expert is not chosen: the choice looks at corrected scores,
    the weights are the scores themselves."""
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    s = e / e.sum(axis=-1, keepdims=True)
    out = np.zeros_like(s)
    for t in range(s.shape[0]):
        chosen = sorted(range(s.shape[1]), key=lambda i: (-(s[t, i] + correction[i]), i))[:top]
        out[t, chosen] = s[t, chosen]
    return out


def routed_mlp(h, w, p, mlp):
    experts = mlp["router"]["experts"]
    weights = route(linear(h, w[p + "router"]), w[p + "correction"], mlp["router"]["top"])
    out = weights[:, experts:].sum(axis=1)[:, None] * h   # the identity experts
    for e in range(experts):
        rows = np.nonzero(weights[:, e])[0]
        if rows.size:
            x, q = h[rows], f"{p}e{e}."
            out[rows] += weights[rows, e][:, None] * linear(silu(linear(x, w[q + "gate"])) * linear(x, w[q + "up"]), w[q + "down"])
    return out


# ---- around the sublayers ------------------------------------------------------------------------------------------
def sublayer(x, w, p, j, eps, run):
    """x + norm of what `run` makes of x and its recent past, gated by x itself."""
    y = run(x + short_conv(x, w[f"{p}canon{j}"]))
    return x + rms_norm(y * sigmoid(linear(x, w[f"{p}rg{j}"], w[f"{p}rg{j}.b"])), w[f"{p}norm{j}"], eps)


def token_input(x, w, p, rows, eps):
    """rows: what the tokens bring to this layer, [tokens, side]."""
    return x + rms_norm(linear(gelu_tanh(linear(x, w[p + "side.gate"])) * rows, w[p + "side.proj"]), w[p + "side.norm"], eps)


def forward(config, w, tokens):
    """(logits [tokens, vocab], what every layer passes on [layers, tokens, width]) of one sequence."""
    eps, side, tokens = config["norm"]["eps"], config["token_side"]["dim"], np.asarray(tokens)
    x = w["embed"][tokens]
    results, after = [x], []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = sublayer(x, w, p, 1, eps, lambda h: mixer(h, w, p + "mix.", layer, eps))
        if layer.get("mlp"):
            x = sublayer(x, w, p, 2, eps, lambda h: routed_mlp(h, w, p + "mlp.", layer["mlp"]))
        x = token_input(x, w, p, w["side.embed"][tokens, i * side:(i + 1) * side], eps)
        results.append(x)
        x = sum(c * r for c, r in zip(w[p + "dwa"], results))
        after.append(x)
    return linear(rms_norm(x, w["final.norm"], eps), w["head"]), np.stack(after)


def greedy(config, w, prompt, steps):
    """Token by token without a cache: the whole sequence is computed again for every token."""
    tokens, margins = list(prompt), []
    for _ in range(steps):
        last = forward(config, w, tokens)[0][-1]
        order = np.sort(last)
        margins.append(float(order[-1] - order[-2]))
        tokens.append(int(np.argmax(last)))
    return tokens[len(prompt):], margins
