"""Plain, slow statement of the Vuzunex design in numpy, one function per mechanism. Test infrastructure only: it shares
no code with the package (no import of it, no kernels), works on whole sequences without any cache, and computes in
whatever floating type its inputs have (float64 by default).

Weights are a dict name -> float array under the names of a checkpoint (`embed`, `l0.norm1`, `l0.mix.q`, ..., `head`);
a layer that borrows its tensors from layer j is resolved by `tensor_prefix`.
"""
import math

import numpy as np


def tensor_prefix(config, i):
    """`l<j>.` of the layer whose tensors layer i uses."""
    j = i
    while config["layers"][j].get("weights_of") is not None:
        j = config["layers"][j]["weights_of"]
    return f"l{j}."


def tensor_shapes(config):
    """name -> shape of every tensor a checkpoint of this configuration holds."""
    width = config["width"]
    out = {"embed": (config["vocab"], width)}
    for i, layer in enumerate(config["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", layer["mixer"]
        heads, dim, rot, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        out[p + "norm1"] = out[p + "norm1b"] = (width,)
        out[p + "mix.q"] = (heads * (dim + rot), width)
        out[p + "mix.dkv"] = (rank + rot, width)
        out[p + "mix.dkv.norm"] = (rank,)
        out[p + "mix.uk"] = (heads * dim, rank)
        out[p + "mix.uv"] = (heads * vdim, rank)
        out[p + "mix.g"] = (heads, width)
        out[p + "mix.o"] = (width, heads * vdim)
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            out[p + "norm2"] = out[p + "norm2b"] = (width,)
            out[p + "mlp.gate"] = out[p + "mlp.up"] = (ff, width)
            out[p + "mlp.down"] = (width, ff)
    out["final.norm"] = (width,)
    out["head"] = (config["vocab"], width)
    return out


def embed_rows(table, tokens, scale):
    return table[np.asarray(tokens)] * scale


def rms_norm(x, weight, eps, weight_bias):
    """x / sqrt(mean(x^2) + eps) * (weight_bias + weight) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * (weight_bias + weight)


def linear(x, weight):
    return x @ weight.T


def rotary_frequencies(dims, base, scaling):
    """(angle per position of every pair, factor of cos and sin). With `scaling` = {factor, original, fast, slow} the
    frequencies below the slow bound are divided by the factor, those above the fast bound stay, a linear ramp between."""
    i = np.arange(dims // 2, dtype=np.float64)
    f = float(base) ** (-2.0 * i / dims)
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def turns_to_dim(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(turns_to_dim(scaling["fast"])), 0)
    hi = min(math.ceil(turns_to_dim(scaling["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x, positions, dims, base, scaling):
    """Rotate the first `dims` entries of the last axis of x [tokens, ..., size], pairing entry i with i + dims/2."""
    f, magnitude = rotary_frequencies(dims, base, scaling)
    a = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    shape = (a.shape[0],) + (1,) * (x.ndim - 2) + (a.shape[1],)
    c, s = (np.cos(a) * magnitude).reshape(shape), (np.sin(a) * magnitude).reshape(shape)
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1).astype(x.dtype)


def causal_softmax(scores):
    """scores [heads, query, key], query i sees keys 0..i."""
    n = scores.shape[-1]
    seen = np.arange(n)[None, :] <= np.arange(n)[:, None]
    s = np.where(seen[None], scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def latent_attention(h, w, p, m, eps):
    """h [tokens, width] -> [tokens, width]; keys and values come out of one shared latent row per token."""
    n = h.shape[0]
    heads, dim, rot, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(n)
    turn = dict(dims=m["rot"]["dims"], base=m["rot"]["base"], scaling=m["rot"].get("scaling"))
    q = linear(h, w[p + "mix.q"]).reshape(n, heads, dim + rot)
    q_plain, q_turned = q[..., :dim], rotate(q[..., dim:], pos, **turn)
    down = linear(h, w[p + "mix.dkv"])
    latent = rms_norm(down[:, :rank], w[p + "mix.dkv.norm"], eps, 0.0)
    k_turned = rotate(down[:, rank:], pos, **turn)
    k_plain = linear(latent, w[p + "mix.uk"]).reshape(n, heads, dim)
    value = linear(latent, w[p + "mix.uv"]).reshape(n, heads, vdim)
    scores = (np.einsum("qhd,khd->hqk", q_plain, k_plain) + np.einsum("qhd,kd->hqk", q_turned, k_turned)) * m["scale"]
    out = np.einsum("hqk,khv->qhv", causal_softmax(scores), value)
    out = out * sigmoid(linear(h, w[p + "mix.g"]))[:, :, None]
    return linear(out.reshape(n, heads * vdim), w[p + "mix.o"])


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gated_mlp(h, w, p):
    return linear(gelu_tanh(linear(h, w[p + "mlp.gate"])) * linear(h, w[p + "mlp.up"]), w[p + "mlp.down"])


def forward(config, w, tokens):
    """(logits [tokens, vocab], residual stream after every layer [layers, tokens, width]) of one sequence."""
    eps = config["norm"]["eps"]
    x = embed_rows(w["embed"], tokens, config["embedding"]["scale"])
    after = []
    for i, layer in enumerate(config["layers"]):
        p = tensor_prefix(config, i)
        x = x + rms_norm(latent_attention(rms_norm(x, w[p + "norm1"], eps, 1.0), w, p, layer["mixer"], eps), w[p + "norm1b"], eps, 1.0)
        if layer.get("mlp"):
            x = x + rms_norm(gated_mlp(rms_norm(x, w[p + "norm2"], eps, 1.0), w, p), w[p + "norm2b"], eps, 1.0)
        after.append(x)
    return linear(rms_norm(x, w["final.norm"], eps, 1.0), w["head"]), np.stack(after)


def greedy(config, w, prompt, steps):
    """Token by token without a cache: the whole sequence is computed again for every token."""
    tokens = list(prompt)
    margins = []
    for _ in range(steps):
        last = forward(config, w, tokens)[0][-1]
        order = np.sort(last)
        margins.append(float(order[-1] - order[-2]))
        tokens.append(int(np.argmax(last)))
    return tokens[len(prompt):], margins
