"""Small Vuzunex configurations with random weights for the tests, and the comparison of logits."""
import json
import os

import numpy as np

import plain_vuzunex as plain


def layer(heads, dim, rot_dim, vdim, rank, ff, rot_dims=None, base=10000.0, scaling=None, scale=None, weights_of=None):
    rot = {"base": base, "dims": rot_dim if rot_dims is None else rot_dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    out = {"type": "latent_attention",
           "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
                     "scale": (dim + rot_dim) ** -0.5 if scale is None else scale, "rot": rot},
           "mlp": None if ff == 0 else {"kind": "dense", "ff": ff}}
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


def config(vocab, width, layers, scale=3.0, eps=1e-5):
    return {"architecture": "Vuzunex", "vocab": vocab, "width": width, "layers": layers, "embedding": {"scale": scale}, "norm": {"eps": eps}}


def cases():
    """name -> configuration; together they reach every kernel form and values a single model would make equal."""
    mid = layer(3, 24, 8, 40, 72, 208, scaling=(8.0, 256.0, 16.0, 0.5))
    odd = layer(5, 20, 6, 36, 52, 180, rot_dims=4)
    first, second = layer(2, 48, 16, 64, 88, 144, base=500.0), layer(4, 16, 32, 24, 120, 0, scaling=(2.0, 64.0, 4.0, 1.0))
    return {
        # span attention, short and medium rows
        "mid": config(384, 192, [mid, layer(6, 32, 24, 16, 48, 96)]),
        # nothing divides by 8: rows are attended one by one, padding everywhere
        "odd": config(301, 132, [odd, layer(1, 13, 2, 7, 9, 33, base=100.0)], scale=1.0, eps=1e-3),
        # unequal layers, one without feed-forward, borrowed tensors (also through a borrower)
        "mixed": config(256, 160, [first, second, layer(2, 48, 16, 64, 88, 144, base=500.0, weights_of=0),
                                   layer(4, 16, 32, 24, 120, 0, scaling=(2.0, 64.0, 4.0, 1.0), weights_of=1),
                                   layer(2, 48, 16, 64, 88, 144, base=500.0, weights_of=2)]),
        # row sizes of a large model, more than 16 heads
        "wide": config(264, 256, [layer(18, 128, 64, 128, 512, 320, scaling=(40.0, 512.0, 32.0, 1.0))]),
        # wider than the tensor-core forms hold
        "huge": config(128, 96, [layer(2, 200, 56, 144, 640, 64)]),
        # a single head, no feed-forward at all
        "tiny": config(64, 32, [layer(1, 8, 2, 8, 8, 0)], scale=2.0),
    }


def to_bf16_bits(x):
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16_bits(b):
    return (np.asarray(b, dtype=np.uint16).astype(np.uint32) << 16).view(np.float32).astype(np.float64)


def random_weights(cfg, seed, sharpen=1.0):
    """(bf16 bit patterns, the same values as float64). `sharpen` scales every query projection, so that single keys stand out
    of the softmax and a key that is missed or seen too much shows in the logits."""
    bits = {}
    for i, (name, shape) in enumerate(sorted(plain.tensor_shapes(cfg).items())):
        rng = np.random.default_rng(1000 * seed + i)
        if name.endswith(".dkv.norm"):
            x = 1.0 + 0.2 * rng.standard_normal(shape)
        elif "norm" in name:
            x = 0.2 * rng.standard_normal(shape)
        elif name == "embed":
            x = 0.5 * rng.standard_normal(shape)
        else:
            x = rng.standard_normal(shape) / np.sqrt(shape[1])
            if name.endswith("mix.q"):
                x = x * sharpen
        bits[name] = to_bf16_bits(x)
    return bits, {k: from_bf16_bits(v) for k, v in bits.items()}


def builder_of(pkg, cfg, dtype, max_seq=256, max_batch=4, pool_tokens=0):
    return pkg.VuzunexPlanBuilder(pkg.vuzunex.decode_config(cfg, dtype=dtype, max_seq=max_seq, max_batch=max_batch, pool_tokens=pool_tokens))


def write_model(pkg, cfg, bits, directory):
    os.makedirs(directory, exist_ok=True)
    with open(os.path.join(directory, "config.json"), "w") as f:
        json.dump(cfg, f)
    pkg.staf.write_safetensors(os.path.join(directory, "model.safetensors"), {k: ("BF16", v) for k, v in bits.items()})


def row_errors(got, want):
    """Root mean square of the difference (mean taken off) of every row, relative to the rows' typical size."""
    d = np.asarray(got, dtype=np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    w = want - want.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / np.sqrt((w * w).mean())


TOLERANCE = {"float32": 2e-5, "bfloat16": 3e-2}
