"""Small Merudra configurations with random weights for the tests."""
import numpy as np

import plain_merudra as plain
from vuzunex_cases import from_bf16_bits, row_errors, to_bf16_bits, write_model  # noqa: F401


def routed(experts, identity, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top}, "expert": {"ff": ff}}


def attention(heads, kv, dim, mlp, temp=(0.4, 24), sharpen=1.0):
    """temp: (coefficient, positions); sharpen: times the usual scale, so that single keys stand out of the softmax."""
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "scale": sharpen * dim ** -0.5,
                                                       "q_temp": {"coef": temp[0], "every": temp[1]}}}


def delta(heads, kv, dim, vdim, mlp, conv=4):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def config(vocab, width, layers, taps=4, side=24, eps=1e-5):
    return {"architecture": "Merudra", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "canon": {"taps": taps}, "token_side": {"dim": side}}


def cases():
    """name -> configuration; together they reach every kernel form and values a single model would make equal or 1."""
    return {
        # every mechanism, sizes that divide by 8, a layer without feed-forward
        "mid": config(320, 160, [attention(6, 2, 40, routed(6, 3, 4, 56)), delta(4, 2, 48, 40, routed(9, 1, 3, 72), conv=3),
                                 attention(4, 4, 32, None, (1.5, 7), 1.7), delta(3, 3, 32, 64, None), attention(8, 1, 48, routed(4, 4, 2, 40), (-0.2, 50))]),
        # nothing divides by 8 (the stream not even by 4), more taps than the usual four, no identity expert
        "odd": config(301, 133, [delta(5, 1, 13, 7, routed(5, 1, 3, 33), conv=6), attention(5, 1, 13, routed(7, 0, 2, 21), (0.9, 33)),
                                 attention(3, 3, 11, None, (0.3, 1)), delta(3, 1, 20, 37, routed(3, 5, 4, 19), conv=5)], taps=6, side=13, eps=1e-3),
        # sizes of large models' layers, more than 16 query heads to a key head
        "wide": config(264, 256, [attention(40, 2, 128, routed(4, 1, 2, 136)), delta(2, 1, 128, 128, routed(6, 2, 8, 64))], taps=2, side=200),
        # a stream wider than a thread block takes in one go, more taps than its portions have rows
        "broad": config(96, 2184, [attention(2, 1, 64, None), delta(2, 1, 32, 32, routed(2, 1, 1, 48))], taps=3, side=72),
        # wider than prompt kernels hold, and than any tensor-core form holds
        "big": config(128, 96, [attention(2, 1, 200, routed(3, 2, 2, 64)), attention(2, 2, 264, None), delta(1, 1, 272, 264, routed(3, 1, 1, 40)), delta(2, 1, 40, 300, None)], taps=5),
        # one head, one tap, one expert beside one that hands its input through, one entry per token and layer
        "tiny": config(64, 32, [attention(1, 1, 8, routed(1, 1, 1, 8), (2.0, 3)), delta(1, 1, 8, 8, routed(2, 2, 4, 8), conv=1)], taps=1, side=1),
        # no cache at all
        "state_only": config(200, 64, [delta(2, 1, 24, 32, routed(4, 1, 2, 24)), delta(2, 2, 16, 32, routed(2, 4, 5, 32))], taps=3),
    }


def random_weights(cfg, seed):
    """(bf16 bit patterns, the same values as float64). Half of the heads of a gated delta rule forget slowly, so that the first
    tokens still matter after hundreds of others."""
    bits = {}
    for i, (tensor, shape) in enumerate(sorted(plain.tensor_shapes(cfg).items())):
        rng = np.random.default_rng(1000 * seed + i)
        kind = tensor.split(".")[-1]
        if kind in ("norm", "norm1", "norm2"):
            x = 1.0 + 0.2 * rng.standard_normal(shape)
        elif kind == "embed":
            x = rng.standard_normal(shape)
        elif kind in ("canon1", "canon2"):
            x = 0.6 * rng.standard_normal(shape) / np.sqrt(shape[1])
        elif kind == "conv":
            x = 0.6 * rng.standard_normal(shape) / np.sqrt(shape[1]) + (np.arange(shape[1]) == shape[1] - 1)
        elif kind == "A_log":
            x = np.where(np.arange(shape[0]) % 2 == 0, -4.0, 0.0) + 0.3 * rng.standard_normal(shape)
        elif kind == "dt_bias":
            x = -2.0 + rng.standard_normal(shape)
        elif kind == "dwa":
            x = 0.3 * rng.standard_normal(shape) + 0.7 * (np.arange(shape[0]) == shape[0] - 1)
        elif kind == "correction":
            x = 0.1 * rng.standard_normal(shape)
        elif len(shape) == 1:
            x = 0.5 * rng.standard_normal(shape)   # biases
        else:
            x = rng.standard_normal(shape) / np.sqrt(shape[1])
        bits[tensor] = to_bf16_bits(x)
    return bits, {k: from_bf16_bits(v) for k, v in bits.items()}


def builder_of(pkg, cfg, dtype, max_seq=256, max_batch=4, pool_tokens=0):
    return pkg.MerudraPlanBuilder(pkg.merudra.decode_config(cfg, dtype=dtype, max_seq=max_seq, max_batch=max_batch, pool_tokens=pool_tokens))


def routes(cfg):
    return any(layer.get("mlp") and layer["mlp"]["router"]["top"] < layer["mlp"]["router"]["experts"] + layer["mlp"]["router"]["identity"] for layer in cfg["layers"])


def agree(got, want, cfg, dtype, slack=1.0):
    """Rows of logits against the plain model's. In bf16 an expert whose score all but equals another's may be the other one:
    such rows, and what they leave in caches and states, are let through when they are few."""
    err = row_errors(got, want)
    limit = slack * {"float32": 2e-5, "bfloat16": 4e-2}[dtype]
    if dtype == "bfloat16" and routes(cfg):
        assert np.median(err) <= 1.5 * limit and (err > 0.6).mean() <= 0.05, (float(np.median(err)), float(err.max()))
    else:
        assert err.max() <= limit, (float(err.max()), int(err.argmax()))
