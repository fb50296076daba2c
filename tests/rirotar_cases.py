"""Small Rirotar configurations with random weights for the tests."""
import numpy as np

import plain_rirotar as plain
from vuzunex_cases import from_bf16_bits, row_errors, to_bf16_bits, write_model  # noqa: F401


def dense(ff, limit=1.2):
    return {"kind": "dense", "ff": ff, "limit": limit}


def routed(experts, top, ff, groups=None, limit=0.9, scale=1.6):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": router, "expert": {"ff": ff, "limit": limit}}


def delta(heads, kv, dim, vdim, mlp, conv=4, channel=False):
    return {"type": "channel_delta" if channel else "delta",
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def latent(heads, dim, vdim, rank, window, mlp, scale=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": window}}}


def config(vocab, width, layers, cap=9.0, eps=1e-5):
    return {"architecture": "Rirotar", "vocab": vocab, "width": width, "layers": layers, "logit_softcap": cap, "norm": {"eps": eps}}


def cases():
    """name -> configuration; together they reach every kernel form and values a single model would make equal or 1."""
    return {
        # every mechanism, sizes that divide by 8
        "mid": config(320, 160, [delta(4, 2, 48, 40, dense(208), channel=True), delta(6, 3, 32, 72, routed(12, 4, 72, (3, 2)), conv=3),
                                 latent(4, 24, 40, 72, 50, routed(8, 2, 96, (4, 2), limit=1.4, scale=0.7)), delta(2, 2, 64, 24, None, conv=2, channel=True),
                                 latent(3, 32, 16, 48, 7, dense(96, 0.5))]),
        # nothing divides by 8, more taps than the usual four, experts without groups, layers without feed-forward
        "odd": config(301, 132, [delta(5, 1, 13, 7, routed(7, 3, 33), conv=5), delta(3, 1, 20, 37, None, conv=6, channel=True),
                                 latent(5, 13, 7, 33, 19, routed(9, 1, 21, (3, 1))), delta(3, 3, 11, 21, dense(77), channel=True)], cap=4.0, eps=1e-3),
        # sizes of large models' layers, more than 16 heads in latent attention
        "wide": config(264, 256, [delta(2, 1, 128, 128, dense(320), channel=True), latent(18, 128, 128, 512, 130, dense(128)), delta(2, 2, 200, 136, dense(64))]),
        # wider than the fused decode step and the tensor-core attention hold
        "huge": config(128, 96, [delta(1, 1, 272, 264, dense(64), channel=True), latent(2, 256, 144, 640, 33, dense(40)), delta(2, 1, 40, 300, dense(40))]),
        # one head, one tap, a window of one token, groups of one expert
        "tiny": config(64, 32, [delta(1, 1, 8, 8, routed(2, 1, 8, (2, 1)), conv=1, channel=True), latent(1, 8, 8, 8, 1, None), delta(1, 1, 8, 8, dense(8), conv=1)]),
        # no cache at all
        "state_only": config(200, 64, [delta(2, 1, 24, 32, dense(64)), delta(2, 2, 16, 32, routed(4, 4, 24), channel=True)], cap=15.0),
        # windows at the page size and around it, one longer than anything the tests feed
        "windows": config(200, 96, [latent(2, 24, 24, 40, w, dense(48)) for w in (64, 65, 63, 1000, 128)]),
    }


LOW_RANK = {"odd": [0, 5, 0, 9], "tiny": [3, 0, 0]}


def shapes_of(name, cfg):
    return plain.tensor_shapes(cfg, LOW_RANK.get(name, 12))


def random_weights(name, cfg, seed, sharpen=1.0):
    """(bf16 bit patterns, the same values as float64). `sharpen` scales the query projections of latent attention, so that single
    keys stand out of the softmax. Half of the heads of a gated delta rule forget slowly, so that the first tokens still matter
    after hundreds of others."""
    bits = {}
    for i, (tensor, shape) in enumerate(sorted(shapes_of(name, cfg).items())):
        rng = np.random.default_rng(1000 * seed + i)
        kind = tensor.split(".")[-1]
        if tensor.endswith(("dkv.norm", "mix.norm")):
            x = 1.0 + 0.2 * rng.standard_normal(shape)
        elif kind in ("norm1", "norm2", "norm"):
            x = 0.2 * rng.standard_normal(shape)
        elif kind == "embed":
            x = rng.standard_normal(shape)
        elif kind == "conv":
            x = 0.6 * rng.standard_normal(shape) / np.sqrt(shape[1]) + (np.arange(shape[1]) == shape[1] - 1)
        elif kind == "A_log":
            x = np.where(np.arange(shape[0]) % 2 == 0, -4.0, 0.0) + 0.3 * rng.standard_normal(shape)
        elif kind == "dt_bias":
            x = -2.0 + rng.standard_normal(shape)
        elif kind == "sink":
            x = 2.0 * sharpen + rng.standard_normal(shape)   # among the largest scores
        else:
            x = rng.standard_normal(shape) / np.sqrt(shape[1])
            if tensor.endswith("mix.q") and tensor[:-1] + "dkv" in shapes_of(name, cfg):
                x = x * sharpen
            elif kind == "router":
                x = 4.0 * x
            elif kind == "head":
                x = 3.0 * x   # the soft cap bends the logits
        bits[tensor] = to_bf16_bits(x)
    return bits, {k: from_bf16_bits(v) for k, v in bits.items()}


def builder_of(pkg, name, cfg, dtype, max_seq=256, max_batch=4, pool_tokens=0):
    return pkg.RirotarPlanBuilder(pkg.rirotar.decode_config(cfg, shapes_of(name, cfg), dtype=dtype, max_seq=max_seq, max_batch=max_batch, pool_tokens=pool_tokens))


def routes(cfg):
    return any(layer.get("mlp") and layer["mlp"]["kind"] == "moe" and layer["mlp"]["router"]["top"] < layer["mlp"]["router"]["experts"] for layer in cfg["layers"])


def agree(got, want, cfg, dtype, slack=1.0):
    """Rows of logits against the plain model's. In bf16 an expert whose score all but equals another's may be the other one:
    such rows, and what they leave in a state, are let through when they are few."""
    err = row_errors(got, want)
    limit = slack * {"float32": 2e-5, "bfloat16": 3e-2}[dtype]
    if dtype == "bfloat16" and routes(cfg):
        assert np.median(err) <= 1.5 * limit and (err > 0.6).mean() <= 0.05, (float(np.median(err)), float(err.max()))
    else:
        assert err.max() <= limit, (float(err.max()), int(err.argmax()))
