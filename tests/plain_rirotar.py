"""Plain, slow statement of the Rirotar design in numpy, one function per mechanism. Test infrastructure only: it shares no
code with the package (no import of it, no kernels), works on whole sequences without any cache or carried state, and computes
in whatever floating type its inputs have (float64 by default).

Weights are a dict name -> float array under the names of a checkpoint (`embed`, `l0.norm1`, `l0.mix.q`, ..., `head`).
"""
import numpy as np


# ---- shapes --------------------------------------------------------------------------------------------------------
def mixer_shapes(layer, width, low_rank):
    """Suffix -> shape of a mixer's tensors. `low_rank`: inner size of the two-factor projections."""
    kind, m = layer["type"], layer["mixer"]
    heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
    if kind == "latent_attention":
        rank = m["kv_rank"]
        return {"q": (heads * dim, width), "dkv": (rank, width), "dkv.norm": (rank,), "uk": (heads * dim, rank),
                "uv": (heads * vdim, rank), "sink": (heads,), "o": (width, heads * vdim)}
    kv, taps = m["kv_heads"], m["conv"]
    out = {}
    for name, rows in (("q", kv * dim), ("k", kv * dim), ("v", heads * vdim)):
        out[name], out[name + ".conv"] = (rows, width), (rows, taps)
    out.update({"b": (heads, width), "A_log": (heads,), "norm": (vdim,)})
    if kind == "channel_delta":
        out.update({"a1": (low_rank, width), "a2": (heads * dim, low_rank), "dt_bias": (heads * dim,),
                    "g1": (low_rank, width), "g2": (heads * vdim, low_rank)})
    else:
        out.update({"a": (heads, width), "dt_bias": (heads,), "g": (heads * vdim, width)})
    out["o"] = (width, heads * vdim)
    return out


def tensor_shapes(config, low_rank=12):
    """name -> shape of every tensor a checkpoint of this configuration holds. `low_rank` may be a number or one per layer."""
    width = config["width"]
    out = {"embed": (config["vocab"], width)}
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        out[p + "norm1"] = (width,)
        rank = low_rank if isinstance(low_rank, int) else low_rank[i]
        out.update({p + "mix." + k: v for k, v in mixer_shapes(layer, width, rank).items()})
        mlp = layer.get("mlp")
        if not mlp:
            continue
        out[p + "norm2"] = (width,)

        def feed_forward(prefix, ff):
            out[prefix + "gate"] = out[prefix + "up"] = (ff, width)
            out[prefix + "down"] = (width, ff)

        if mlp["kind"] == "dense":
            feed_forward(p + "mlp.", mlp["ff"])
        else:
            for e in range(mlp["router"]["experts"]):
                feed_forward(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
            out[p + "mlp.router"] = (mlp["router"]["experts"], width)
    out["final.norm"] = (width,)
    out["head"] = (config["vocab"], width)
    return out


# ---- small parts ---------------------------------------------------------------------------------------------------
def rms_norm(x, weight, eps, weight_bias):
    """x / sqrt(mean(x^2) + eps) * (weight_bias + weight) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * (weight_bias + weight)


def linear(x, weight):
    return x @ weight.T


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


# ---- latent attention ----------------------------------------------------------------------------------------------
def window_mask(n, window):
    """[query, key]: query i sees keys i - window + 1 .. i."""
    i = np.arange(n)
    back = i[:, None] - i[None, :]
    return (back >= 0) & (back < window)


def sink_softmax(scores, seen, sink):
    """scores [heads, query, key]; exp(sink_h) joins the denominator of every row of head h."""
    s = np.where(seen[None], scores, -np.inf)
    top = np.maximum(s.max(axis=-1, keepdims=True), sink[:, None, None])
    e = np.exp(s - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink[:, None, None] - top))


def latent_attention(h, w, p, m, eps):
    """h [tokens, width] -> [tokens, width]; keys and values come out of one latent row per token, no positions."""
    n = h.shape[0]
    heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
    q = linear(h, w[p + "q"]).reshape(n, heads, dim)
    latent = rms_norm(linear(h, w[p + "dkv"]), w[p + "dkv.norm"], eps, 0.0)
    k = linear(latent, w[p + "uk"]).reshape(n, heads, dim)
    v = linear(latent, w[p + "uv"]).reshape(n, heads, vdim)
    scores = np.einsum("qhd,khd->hqk", q, k) * m["scale"]
    weights = sink_softmax(scores, window_mask(n, m["mask"]["size"]), w[p + "sink"])
    return linear(np.einsum("hqk,khv->qhv", weights, v).reshape(n, heads * vdim), w[p + "o"])


# ---- gated delta rule ----------------------------------------------------------------------------------------------
def short_conv(x, taps):
    """x [tokens, channels], taps [channels, count]: causal, the last tap meets the current token, zeros before the start."""
    n, count = x.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((count - 1, x.shape[1]), dtype=x.dtype), x])
    return sum(padded[j:j + n] * taps[:, j] for j in range(count))


def delta_scan(q, k, v, g, beta):
    """q, k [tokens, heads, dim], v [tokens, heads, vdim], g [tokens, heads, dim] decays, beta [tokens, heads]. Token by token:
    the state is decayed, corrected towards v along k, then read with q."""
    n, heads, dim = k.shape
    state = np.zeros((heads, dim, v.shape[2]), dtype=v.dtype)
    out = np.empty_like(v)
    for t in range(n):
        state = g[t][:, :, None] * state
        miss = v[t] - np.einsum("hdv,hd->hv", state, k[t])
        state = state + k[t][:, :, None] * (beta[t][:, None] * miss)[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", state, q[t])
    return out


def delta_inputs(h, w, p, m, kind):
    """(q, k, v, g, beta) of delta_scan."""
    n = h.shape[0]
    heads, kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(linear(h, w[p + t]), w[p + t + ".conv"])) for t in "qkv")
    share = heads // kv
    q = np.repeat(unit(q.reshape(n, kv, dim)) * dim ** -0.5, share, axis=1)
    k = np.repeat(unit(k.reshape(n, kv, dim)), share, axis=1)
    beta = sigmoid(linear(h, w[p + "b"]))
    rate = np.exp(w[p + "A_log"])
    if kind == "channel_delta":
        raw = linear(linear(h, w[p + "a1"]), w[p + "a2"]) + w[p + "dt_bias"]
        g = np.exp(-rate[:, None] * softplus(raw).reshape(n, heads, dim))
    else:
        g = np.exp(-rate * softplus(linear(h, w[p + "a"]) + w[p + "dt_bias"]))
        g = np.repeat(g[:, :, None], dim, axis=2)
    return q, k, v.reshape(n, heads, vdim), g, beta


def delta_mixer(h, w, p, m, kind, eps):
    n, heads, vdim = h.shape[0], m["heads"], m["vdim"]
    o = rms_norm(delta_scan(*delta_inputs(h, w, p, m, kind)), w[p + "norm"], eps, 0.0)
    gate = sigmoid(linear(linear(h, w[p + "g1"]), w[p + "g2"])) if kind == "channel_delta" else silu(linear(h, w[p + "g"]))
    return linear((o * gate.reshape(n, heads, vdim)).reshape(n, heads * vdim), w[p + "o"])


def mixer(h, w, p, layer, eps):
    if layer["type"] == "latent_attention":
        return latent_attention(h, w, p, layer["mixer"], eps)
    return delta_mixer(h, w, p, layer["mixer"], layer["type"], eps)


# ---- feed-forward --------------------------------------------------------------------------------------------------
def clamped_gate(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def clamped_mlp(h, w, p, limit):
    return linear(clamped_gate(linear(h, w[p + "gate"]), linear(h, w[p + "up"]), limit), w[p + "down"])


def route(z, router):
    """z [tokens, experts] -> weights [tokens, experts], zero where an expert is not chosen."""
    s = sigmoid(z)
    n, experts = s.shape
    groups = router.get("groups") or {"count": 1, "keep": 1}
    per = experts // groups["count"]
    out = np.zeros_like(s)
    for t in range(n):
        strength = [np.sort(s[t, i * per:(i + 1) * per])[::-1][:2].sum() for i in range(groups["count"])]
        kept = sorted(range(groups["count"]), key=lambda i: (-strength[i], i))[:groups["keep"]]
        allowed = [e for e in range(experts) if e // per in kept]
        chosen = sorted(allowed, key=lambda e: (-s[t, e], e))[:router["top"]]
        out[t, chosen] = s[t, chosen] / (s[t, chosen].sum() + 1e-20) * router["scale"]
    return out


def routed_mlp(h, w, p, mlp):
    weights = route(linear(h, w[p + "router"]), mlp["router"])
    out = np.zeros_like(h)
    for e in range(weights.shape[1]):
        rows = np.nonzero(weights[:, e])[0]
        if rows.size:
            out[rows] += weights[rows, e][:, None] * clamped_mlp(h[rows], w, f"{p}e{e}.", mlp["expert"]["limit"])
    return out


def feed_forward(h, w, p, mlp):
    return clamped_mlp(h, w, p, mlp["limit"]) if mlp["kind"] == "dense" else routed_mlp(h, w, p, mlp)


# ---- the model -----------------------------------------------------------------------------------------------------
def forward(config, w, tokens):
    """(logits [tokens, vocab], residual stream after every layer [layers, tokens, width]) of one sequence."""
    eps = config["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    after = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + mixer(rms_norm(x, w[p + "norm1"], eps, 1.0), w, p + "mix.", layer, eps)
        if layer.get("mlp"):
            x = x + feed_forward(rms_norm(x, w[p + "norm2"], eps, 1.0), w, p + "mlp.", layer["mlp"])
        after.append(x)
    z = linear(rms_norm(x, w["final.norm"], eps, 1.0), w["head"])
    return (soft_cap(z, config["logit_softcap"]) if config.get("logit_softcap") else z), np.stack(after)


def greedy(config, w, prompt, steps):
    """Token by token without a cache: the whole sequence is computed again for every token."""
    tokens, margins = list(prompt), []
    for _ in range(steps):
        last = forward(config, w, tokens)[0][-1]
        order = np.sort(last)
        margins.append(float(order[-1] - order[-2]))
        tokens.append(int(np.argmax(last)))
    return tokens[len(prompt):], margins
