"""Plain, slow statement of the Kalevik design in numpy, one function per mechanism. Test infrastructure only: it shares no code
with the package (no import of it, no kernels), works on whole sequences without any cache or carried state, and computes in
whatever floating type its inputs have (float64 by default).

Weights are a dict name -> float array under the names of a checkpoint (`embed`, `l0.norm1`, `l0.mix.q`, ..., `head`).
"""
import math

import numpy as np

_erf = np.vectorize(math.erf, otypes=[np.float64])


# ---- shapes --------------------------------------------------------------------------------------------------------
def latent_shapes(m, width):
    heads, per = m["heads"], m["dim"] + m["rot_dim"]
    rank = m["kv_rank"]
    return {"q": (heads * per, width), "dkv": (rank + m["rot_dim"], width), "dkv.norm": (rank,), "uk": (heads * m["dim"], rank),
            "uv": (heads * m["vdim"], rank), "o": (width, heads * m["vdim"])}


def parallel_shapes(m, width):
    a, r = m["left"], m["right"]
    out = {"left.q": (a["heads"] * a["dim"], width), "left.k": (a["kv_heads"] * a["dim"], width), "left.v": (a["kv_heads"] * a["vdim"], width),
           "left.q.norm": (a["dim"],), "left.k.norm": (a["dim"],), "left.g": (a["heads"], width), "left.o": (width, a["heads"] * a["vdim"])}
    out.update({"right.q": (r["heads"] * r["dim"], width), "right.k": (r["heads"] * r["dim"], width), "right.v": (r["heads"] * r["vdim"], width),
                "right.g": (r["heads"] * r["vdim"], width), "right.o": (width, r["heads"] * r["vdim"])})
    return out


def mlp_shapes(mlp, width):
    if mlp["kind"] == "dense":
        return {"gate": (mlp["ff"], width), "up": (mlp["ff"], width), "down": (width, mlp["ff"])}
    out = {}
    for e in range(mlp["router"]["experts"]):
        out[f"e{e}.up"], out[f"e{e}.down"] = (mlp["expert"]["ff"], width), (width, mlp["expert"]["ff"])
    out["router"] = (mlp["router"]["experts"], width)
    if mlp.get("shared"):
        ff = mlp["shared"]["ff"]
        out.update({"shared.up": (ff, width), "shared.down": (width, ff), "shared.sg": (1, width)})
    return out


def tensor_shapes(config):
    """name -> shape of every tensor a checkpoint of this configuration holds."""
    width = config["width"]
    out = {"embed": (config["vocab"], width)}
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        norms = ["norm1", "norm1b"] + (["norm2", "norm2b"] if layer.get("mlp") else [])
        out.update({p + n: (width,) for n in norms})
        mixer = (latent_shapes if layer["type"] == "latent_attention" else parallel_shapes)(layer["mixer"], width)
        out.update({p + "mix." + k: v for k, v in mixer.items()})
        if layer.get("mlp"):
            out.update({p + "mlp." + k: v for k, v in mlp_shapes(layer["mlp"], width).items()})
    out["final.norm"] = (width,)
    out["head"] = (config["vocab"], width)
    return out


# ---- small parts ---------------------------------------------------------------------------------------------------
def rms_unit(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, weight, eps):
    return rms_unit(x, eps) * weight


def linear(x, weight):
    return x @ weight.T


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_erf(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


# ---- positions -----------------------------------------------------------------------------------------------------
def angles(n, dims, base, factor=1.0):
    """[position, pair] in double precision."""
    freq = np.float64(base) ** (-2.0 * np.arange(dims // 2) / max(dims, 1)) / factor
    return np.arange(n)[:, None] * freq


def rotate_neighbours(x, dims, base):
    """x [tokens, heads, size]: entries 2i and 2i + 1 of the first `dims` form a pair."""
    a = angles(x.shape[0], dims, base)[:, None, :]
    out = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * np.cos(a) - v * np.sin(a)
    out[..., 1:dims:2] = v * np.cos(a) + u * np.sin(a)
    return out


def rotate_halves(x, dims, base, factor=1.0):
    """x [tokens, heads, size]: entries i and i + dims / 2 of the first `dims` form a pair."""
    a = angles(x.shape[0], dims, base, factor)[:, None, :]
    half = dims // 2
    out = x.copy()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * np.cos(a) - v * np.sin(a)
    out[..., half:dims] = v * np.cos(a) + u * np.sin(a)
    return out


# ---- latent attention ----------------------------------------------------------------------------------------------
def causal_mask(n):
    i = np.arange(n)
    return i[:, None] >= i[None, :]


def masked_softmax(scores, seen):
    return softmax(np.where(seen[None], scores, -np.inf))


def latent_attention(h, w, p, m, eps):
    """h [tokens, width] -> [tokens, width]; keys and values come out of one latent row per token, a rotated key part is shared."""
    n, heads, dim, vdim, rank = h.shape[0], m["heads"], m["dim"], m["vdim"], m["kv_rank"]
    q = linear(h, w[p + "q"]).reshape(n, heads, dim + m["rot_dim"])
    row = linear(h, w[p + "dkv"])
    c = rms_norm(row[:, :rank], w[p + "dkv.norm"], eps)
    q_turned = rotate_neighbours(q[:, :, dim:], m["rot"]["dims"], m["rot"]["base"])
    k_turned = rotate_neighbours(row[:, None, rank:], m["rot"]["dims"], m["rot"]["base"])[:, 0]
    k = linear(c, w[p + "uk"]).reshape(n, heads, dim)
    v = linear(c, w[p + "uv"]).reshape(n, heads, vdim)
    scores = (np.einsum("qhd,khd->hqk", q[:, :, :dim], k) + np.einsum("qhd,kd->hqk", q_turned, k_turned)) * m["scale"]
    weights = masked_softmax(scores, causal_mask(n))
    return linear(np.einsum("hqk,khv->qhv", weights, v).reshape(n, heads * vdim), w[p + "o"])


# ---- grouped attention in chunks -----------------------------------------------------------------------------------
def chunk_mask(n, size):
    """[query, key]: earlier positions of the query's own chunk."""
    i = np.arange(n)
    return causal_mask(n) & (i[:, None] // size == i[None, :] // size)


def softmax_plus_one(scores, seen):
    """exp(s) / (1 + sum exp(s)) over the seen keys."""
    s = np.where(seen[None], scores, -np.inf)
    top = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - top)
    return e / (np.exp(-top) + e.sum(axis=-1, keepdims=True))


def grouped_attention(h, w, p, m, eps):
    """Without the output projection: [tokens, heads * vdim]."""
    n, heads, groups, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    share, rot = heads // groups, m["rot"]
    factor = (rot.get("scaling") or {"factor": 1.0})["factor"]
    q = rms_norm(linear(h, w[p + "q"]).reshape(n, heads, dim), w[p + "q.norm"], eps)
    k = rms_norm(linear(h, w[p + "k"]).reshape(n, groups, dim), w[p + "k.norm"], eps)
    v = linear(h, w[p + "v"]).reshape(n, groups, vdim)
    q, k = (rotate_halves(x, rot["dims"], rot["base"], factor) for x in (q, k))
    k, v = np.repeat(k, share, axis=1), np.repeat(v, share, axis=1)
    scores = np.einsum("qhd,khd->hqk", q, k) * m["scale"]
    weights = softmax_plus_one(scores, chunk_mask(n, m["mask"]["size"]))
    out = np.einsum("hqk,khv->qhv", weights, v) * sigmoid(linear(h, w[p + "g"]))[:, :, None]
    return out.reshape(n, heads * vdim)


# ---- retention -----------------------------------------------------------------------------------------------------
def retention_scan(q, k, v, decay):
    """q, k [tokens, heads, dim], v [tokens, heads, vdim], decay [heads]. Token by token: the state is decayed, gains k v^T, and
    is read with q."""
    n, heads, dim = k.shape
    state = np.zeros((heads, dim, v.shape[2]), dtype=v.dtype)
    out = np.empty_like(v)
    for t in range(n):
        state = decay[:, None, None] * state + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", state, q[t])
    return out


def retention(h, w, p, m, eps):
    """Without the output projection: [tokens, heads * vdim]."""
    n, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(h, w[p + "q"]).reshape(n, heads, dim)
    k = linear(h, w[p + "k"]).reshape(n, heads, dim) * dim ** -0.5
    v = linear(h, w[p + "v"]).reshape(n, heads, vdim)
    o = rms_unit(retention_scan(q, k, v, np.asarray(m["decay"], dtype=h.dtype)), eps)
    return o.reshape(n, heads * vdim) * silu(linear(h, w[p + "g"]))


def parallel(h, w, p, m, eps):
    left = linear(grouped_attention(h, w, p + "left.", m["left"], eps), w[p + "left.o"])
    right = linear(retention(h, w, p + "right.", m["right"], eps), w[p + "right.o"])
    return m["left_scale"] * left + m["right_scale"] * right


def mixer(h, w, p, layer, eps):
    return (latent_attention if layer["type"] == "latent_attention" else parallel)(h, w, p, layer["mixer"], eps)


# ---- feed-forward --------------------------------------------------------------------------------------------------
def dense_mlp(h, w, p):
    return linear(silu(linear(h, w[p + "gate"])) * linear(h, w[p + "up"]), w[p + "down"])


def expert(h, w, p):
    return linear(gelu_erf(linear(h, w[p + "up"])), w[p + "down"])


def route(z, router):
    """z [tokens, experts] -> weights [tokens, experts], zero where an expert is not chosen."""
    s = softmax(z)
    n, experts = s.shape
    groups = router.get("groups") or {"count": 1, "keep": 1}
    per = experts // groups["count"]
    out = np.zeros_like(s)
    for t in range(n):
        best = [s[t, i * per:(i + 1) * per].max() for i in range(groups["count"])]
        kept = sorted(range(groups["count"]), key=lambda i: (-best[i], i))[:groups["keep"]]
        allowed = [e for e in range(experts) if e // per in kept]
        chosen = sorted(allowed, key=lambda e: (-s[t, e], e))[:router["top"]]
        out[t, chosen] = s[t, chosen]
    return out


def routed_mlp(h, w, p, mlp):
    weights = route(linear(h, w[p + "router"]), mlp["router"])
    out = np.zeros_like(h)
    for e in range(weights.shape[1]):
        rows = np.nonzero(weights[:, e])[0]
        if rows.size:
            out[rows] += weights[rows, e][:, None] * expert(h[rows], w, f"{p}e{e}.")
    if mlp.get("shared"):
        out = out + sigmoid(linear(h, w[p + "shared.sg"])) * expert(h, w, p + "shared.")
    return out


def feed_forward(h, w, p, mlp):
    return dense_mlp(h, w, p) if mlp["kind"] == "dense" else routed_mlp(h, w, p, mlp)


# ---- the model -----------------------------------------------------------------------------------------------------
def runs(config):
    """[(layer, does the embedding output join in front of it)] in the order of execution."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    out = [(i, False) for i in range(loop["start"])]
    for turn in range(loop["times"]):
        out += [(i, turn > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return out + [(i, False) for i in range(loop["stop"], n)]


def forward(config, w, tokens):
    """(logits [tokens, vocab], residual stream after every layer run [runs, tokens, width]) of one sequence."""
    eps = config["norm"]["eps"]
    start = w["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    x, after = start, []
    for i, joins in runs(config):
        layer, p = config["layers"][i], f"l{i}."
        if joins:
            x = x + start
        x = x + rms_norm(mixer(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer, eps), w[p + "norm1b"], eps)
        if layer.get("mlp"):
            x = x + rms_norm(feed_forward(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"]), w[p + "norm2b"], eps)
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
