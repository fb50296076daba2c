"""Small Kalevik configurations with random weights for the tests."""
import numpy as np

import plain_kalevik as plain
from vuzunex_cases import from_bf16_bits, row_errors, to_bf16_bits, write_model  # noqa: F401


def dense(ff):
    return {"kind": "dense", "ff": ff}


def routed(experts, top, ff, groups=None, shared=0):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "router": router, "expert": {"ff": ff}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def latent(heads, dim, rot, vdim, rank, mlp, base=10000.0, scale=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": (dim + rot) ** -0.5 if scale is None else scale,
                      "rot": {"base": base, "dims": rot}}}


def left(heads, kv, dim, vdim, chunk, rot, base=10000.0, factor=None, scale=None):
    turn = {"base": base, "dims": rot}
    if factor is not None:
        turn["scaling"] = {"factor": factor}
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": chunk}, "rot": turn}


def right(heads, dim, vdim, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": [1.0 - 2.0 ** (-1.0 - 7.0 * i / max(1, heads - 1)) for i in range(heads)] if decay is None else decay}


def parallel(a, r, mlp, scales=(0.8, 0.5)):
    return {"type": "parallel", "mixer": {"left": a, "right": r, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def config(vocab, width, layers, loop=None, scale=0.7, eps=1e-5):
    out = {"architecture": "Kalevik", "vocab": vocab, "width": width, "layers": layers, "embedding": {"scale": scale}, "norm": {"eps": eps}}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


def cases():
    """name -> configuration; together they reach every kernel form and values a single model would make equal or 1."""
    return {
        # every mechanism, sizes that divide by 8, a loop in the middle
        "mid": config(320, 160, [parallel(left(6, 2, 40, 24, 50, 24, factor=2.5), right(3, 48, 40), routed(12, 3, 56, (3, 2), shared=72)),
                                 latent(3, 24, 8, 40, 72, dense(208)), parallel(left(4, 4, 32, 48, 100, 32, base=500.0), right(2, 24, 72), dense(96), (1.3, 0.4)),
                                 latent(5, 16, 24, 32, 56, routed(8, 2, 40, (4, 3)), base=200.0), latent(2, 32, 16, 16, 40, None)], (1, 4, 3)),
        # nothing divides by 8, experts without groups, layers without feed-forward, no loop
        "odd": config(301, 132, [parallel(left(5, 1, 13, 7, 33, 6), right(3, 11, 21), routed(7, 3, 33, shared=19)), latent(5, 13, 6, 7, 33, None),
                                 parallel(left(3, 3, 18, 21, 70, 10, factor=8.0), right(1, 37, 9), None, (0.3, 1.7)), latent(1, 20, 2, 9, 25, routed(9, 1, 21, (3, 1)))],
                      scale=1.0, eps=1e-3),
        # sizes of large models' layers, more than 16 query heads to a key / value head; the loop runs once
        "wide": config(264, 256, [parallel(left(40, 2, 128, 128, 96, 64), right(2, 128, 128), dense(128)), latent(18, 128, 64, 128, 512, routed(4, 4, 64, shared=136))], (0, 2, 1)),
        # wider than prompt kernels hold
        "big": config(128, 96, [parallel(left(2, 1, 200, 136, 40, 48), right(1, 200, 264), dense(64)), parallel(left(2, 2, 144, 248, 150, 144), right(2, 160, 32), None)]),
        # wider than any tensor-core form holds
        "huge": config(128, 96, [parallel(left(2, 1, 264, 272, 70, 128), right(1, 264, 40), dense(40)), latent(2, 200, 56, 144, 640, dense(64)),
                                 parallel(left(1, 1, 24, 24, 9, 24), right(1, 272, 296), None)]),
        # one head, chunks of one token, groups of one expert, the whole model in a loop
        "tiny": config(64, 32, [parallel(left(1, 1, 8, 8, 1, 4), right(1, 8, 8, [0.5]), routed(2, 1, 8, (2, 1), shared=8)), latent(1, 8, 2, 8, 8, None)], (0, 2, 4), scale=1.5),
        # chunks at the page size and around it, one longer than anything the tests feed; a state that forgets nothing
        "chunks": config(200, 96, [parallel(left(2, 1, 24, 24, c, 16), right(2, 24, 16, [0.3, 1.0] if c == 65 else None), dense(48)) for c in (64, 65, 63, 1000, 128)], (3, 5, 2), eps=0.05),
    }


def random_weights(cfg, seed, sharpen=1.0):
    """(bf16 bit patterns, the same values as float64). `sharpen` scales the queries of both kinds of attention, so that single
    keys stand out of the softmax."""
    bits = {}
    for i, (tensor, shape) in enumerate(sorted(plain.tensor_shapes(cfg).items())):
        rng = np.random.default_rng(1000 * seed + i)
        if len(shape) == 1:
            x = 1.0 + 0.2 * rng.standard_normal(shape)
            if tensor.endswith("left.q.norm"):
                x = x * sharpen
            elif tensor.endswith(("norm1b", "norm2b")):
                x = 0.6 * x
        elif tensor == "embed":
            x = rng.standard_normal(shape)
        else:
            x = rng.standard_normal(shape) / np.sqrt(shape[1])
            if tensor.endswith("mix.q"):
                x = x * sharpen
            elif tensor.endswith(("router", "shared.sg")):
                x = 2.0 * x
        bits[tensor] = to_bf16_bits(x)
    return bits, {k: from_bf16_bits(v) for k, v in bits.items()}


def builder_of(pkg, cfg, dtype, max_seq=256, max_batch=4, pool_tokens=0):
    return pkg.KalevikPlanBuilder(pkg.kalevik.decode_config(cfg, dtype=dtype, max_seq=max_seq, max_batch=max_batch, pool_tokens=pool_tokens))


def routes(cfg):
    return any(layer.get("mlp") and layer["mlp"]["kind"] == "moe" and layer["mlp"]["router"]["top"] < layer["mlp"]["router"]["experts"] for layer in cfg["layers"])


def agree(got, want, cfg, dtype, slack=1.0):
    """Rows of logits against the plain model's. In bf16 an expert whose score all but equals another's may be the other one:
    such rows, and what they leave in caches and states, are let through when they are few."""
    err = row_errors(got, want)
    limit = slack * {"float32": 2e-5, "bfloat16": 4e-2}[dtype]
    if dtype == "bfloat16" and routes(cfg):
        assert np.median(err) <= 1.5 * limit and (err > 0.6).mean() <= 0.05, (float(np.median(err)), float(err.max()))
    elif dtype == "bfloat16":   # (a head's read-out that all but cancels is blown up by its norm)
        assert np.quantile(err, 0.95) <= limit and err.max() <= 4.0 * limit, (float(np.quantile(err, 0.95)), float(err.max()), int(err.argmax()))
    else:
        assert err.max() <= limit, (float(err.max()), int(err.argmax()))
