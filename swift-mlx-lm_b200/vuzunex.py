"""Vuzunex recipe: config.json -> VuzunexConfig -> fp32-stream step list.

A decoder of latent-attention layers with an output gate per head, a dense GELU-gated feed-forward (or none), and a norm
before and after every sublayer. Layers are listed one by one, each with its own sizes; a layer may borrow another layer's
tensors while it keeps a cache of its own. Nothing here computes or caches: the steps run through the same plan, pool,
executor and kernels as any other fp32-stream plan.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass, field
from typing import Dict, List, Optional

from .lib import BuffersDesc, Step
from .plan import (BUF_HIDDEN, BUF_LOGITS, BUF_S0, BUF_S1, BUF_S2, BUF_S3, BUF_S4, SHARD_REPLICATE, STEP_ARGMAX, STEP_COPY_RMSNORM,
                   STEP_EMBED, STEP_GEGLU, STEP_LATENT_ATTN, STEP_POSTNORM_RESADD_COPY_RMSNORM, STEP_POSTNORM_RESADD_RMSNORM,
                   STEP_PRODUCT, STREAM_ALL_F32, STREAM_F32, _step)

ARCHITECTURE = "Vuzunex"


@dataclass(frozen=True)
class RotaryScaling:
    """Rotary frequencies interpolated by parts (YaRN): pairs that turn fewer than `slow` times over `original` positions are
    divided by `factor`, pairs that turn more than `fast` times stay."""
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class LatentAttention:
    heads: int
    dim: int          # query / key entries per head without positions
    rot_dim: int      # query / key entries with positions; the key part is shared by the heads
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int     # how many of the rot_dim entries turn
    rot_scaling: Optional[RotaryScaling] = None


@dataclass(frozen=True)
class Layer:
    mixer: LatentAttention
    ff: int           # 0: no feed-forward
    weights_of: int   # the layer whose tensors are used (its own index: no borrowing)


@dataclass
class VuzunexConfig:
    vocab: int
    width: int
    layers: List[Layer] = field(default_factory=list)
    embedding_scale: float = 1.0
    norm_eps: float = 1e-6
    dtype: str = "bfloat16"      # or "float32": everything in fp32
    max_seq: int = 4224
    max_batch: int = 1
    pool_tokens: int = 0         # tokens the page pool holds over all sequences; 0 = max_batch * max_seq

    def buffers_desc(self) -> BuffersDesc:
        return BuffersDesc(hidden=self.width, vocab=self.vocab, max_seq=self.max_seq, max_batch=self.max_batch,
                           stream_dtype=STREAM_ALL_F32 if self.dtype == "float32" else STREAM_F32,
                           latent_layers=len(self.layers), kv_pool_tokens=self.pool_tokens)

    def weight_elems(self) -> int:
        """Matrix entries one decode step reads (a borrowed layer's matrices count every time they are read)."""
        total = self.vocab * self.width
        for layer in self.layers:
            m, w = layer.mixer, self.width
            total += w * (m.heads * (m.dim + m.rot_dim) + m.kv_rank + m.rot_dim + m.heads) + m.heads * (m.dim + m.vdim) * m.kv_rank
            total += m.heads * m.vdim * w + 3 * w * layer.ff
        return total


def decode_config(config: Dict, dtype: str = "bfloat16", max_seq: int = 4224, max_batch: int = 1, pool_tokens: int = 0) -> VuzunexConfig:
    """config.json of a Vuzunex checkpoint. Every entry is read from the file; a value this recipe cannot express is refused."""
    if config.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {config.get('architecture')!r} is not {ARCHITECTURE}")
    if dtype not in ("bfloat16", "float32"):
        raise ValueError(f"dtype {dtype!r}: bfloat16 or float32")
    layers: List[Layer] = []
    entries = config["layers"]
    for i, entry in enumerate(entries):
        if entry["type"] != "latent_attention":
            raise ValueError(f"layer {i}: mixer type {entry['type']!r}")
        m, mlp = entry["mixer"], entry.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
        rot, scaling = m["rot"], m["rot"].get("scaling")
        if rot["dims"] > m["rot_dim"] or rot["dims"] % 2:
            raise ValueError(f"layer {i}: {rot['dims']} rotated entries of {m['rot_dim']}")
        source, seen = i, set()
        while entries[source].get("weights_of") is not None:
            seen.add(source)
            source = int(entries[source]["weights_of"])
            if source in seen or not 0 <= source < len(entries):
                raise ValueError(f"layer {i}: weights_of does not lead to a layer with tensors")
        layers.append(Layer(
            mixer=LatentAttention(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                                  kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot_base=float(rot["base"]), rot_dims=int(rot["dims"]),
                                  rot_scaling=None if scaling is None else RotaryScaling(
                                      factor=float(scaling["factor"]), original=float(scaling["original"]),
                                      fast=float(scaling["fast"]), slow=float(scaling["slow"]))),
            ff=0 if mlp is None else int(mlp["ff"]), weights_of=source))
    return VuzunexConfig(vocab=int(config["vocab"]), width=int(config["width"]), layers=layers,
                         embedding_scale=float(config["embedding"]["scale"]), norm_eps=float(config["norm"]["eps"]), dtype=dtype,
                         max_seq=max_seq, max_batch=max_batch, pool_tokens=pool_tokens)


class VuzunexPlanBuilder:
    """Tensor inventory and step list of a VuzunexConfig (the counterpart of plan.DispatchPlanBuilder)."""

    def __init__(self, config: VuzunexConfig):
        self.config = config

    def tensors(self):
        """(name, kind, shape, shard kind): `matrix` = operand of a product, `norm0` = norm weight stored around zero,
        `norm` = plain norm weight, `dense` = the embedding table."""
        c, w = self.config, self.config.width
        out = [("embed", "dense", (c.vocab, w), SHARD_REPLICATE)]
        for i, layer in enumerate(c.layers):
            if layer.weights_of != i:
                continue
            p, m = f"l{i}.", layer.mixer
            out += [(p + "norm1", "norm0", (w,), SHARD_REPLICATE), (p + "norm1b", "norm0", (w,), SHARD_REPLICATE),
                    (p + "mix.q", "matrix", (m.heads * (m.dim + m.rot_dim), w), SHARD_REPLICATE),
                    (p + "mix.dkv", "matrix", (m.kv_rank + m.rot_dim, w), SHARD_REPLICATE),
                    (p + "mix.dkv.norm", "norm", (m.kv_rank,), SHARD_REPLICATE),
                    (p + "mix.uk", "matrix", (m.heads * m.dim, m.kv_rank), SHARD_REPLICATE),
                    (p + "mix.uv", "matrix", (m.heads * m.vdim, m.kv_rank), SHARD_REPLICATE),
                    (p + "mix.g", "matrix", (m.heads, w), SHARD_REPLICATE),
                    (p + "mix.o", "matrix", (w, m.heads * m.vdim), SHARD_REPLICATE)]
            if layer.ff:
                out += [(p + "norm2", "norm0", (w,), SHARD_REPLICATE), (p + "norm2b", "norm0", (w,), SHARD_REPLICATE),
                        (p + "mlp.gate", "matrix", (layer.ff, w), SHARD_REPLICATE), (p + "mlp.up", "matrix", (layer.ff, w), SHARD_REPLICATE),
                        (p + "mlp.down", "matrix", (w, layer.ff), SHARD_REPLICATE)]
        return out + [("final.norm", "norm0", (w,), SHARD_REPLICATE), ("head", "matrix", (c.vocab, w), SHARD_REPLICATE)]

    def decode_steps(self, layers: Optional[int] = None, store_final: bool = False) -> List[Step]:
        """The steps of one token. `layers` stops after that many layers; `store_final` keeps the residual stream behind the last
        one in its buffer (both for tests that look at the stream)."""
        c, w = self.config, self.config.width
        steps = [_step(STEP_EMBED, out_buf=BUF_HIDDEN, n=w, scale=c.embedding_scale, weight="embed")]
        post = None   # norm of the sublayer whose output waits in the hidden buffer

        def norm(name: str, last: bool = False):
            common = dict(in_buf=BUF_HIDDEN, out_buf=BUF_S0, n=w, eps=c.norm_eps, weight_bias=1.0)
            if post is None:
                steps.append(_step(STEP_COPY_RMSNORM, weight=name, **common))
            else:
                kind = STEP_POSTNORM_RESADD_RMSNORM if last and not store_final else STEP_POSTNORM_RESADD_COPY_RMSNORM
                steps.append(_step(kind, weight=post, weight2=name, **common))

        def product(name: str, src: int, dst: int, n: int, k: int):
            steps.append(_step(STEP_PRODUCT, in_buf=src, out_buf=dst, n=n, k=k, weight=name))

        for i, layer in enumerate(c.layers[:layers]):
            p, m = f"l{layer.weights_of}.", layer.mixer
            norm(p + "norm1")
            product(p + "mix.q", BUF_S0, BUF_S1, m.heads * (m.dim + m.rot_dim), w)
            product(p + "mix.dkv", BUF_S0, BUF_S3, m.kv_rank + m.rot_dim, w)
            product(p + "mix.g", BUF_S0, BUF_S4, m.heads, w)
            scaling = m.rot_scaling
            steps.append(_step(STEP_LATENT_ATTN, layer=i, in_buf=BUF_S1, in2_buf=BUF_S3, in3_buf=BUF_S4, out_buf=BUF_S0, n=m.kv_rank,
                               heads=m.heads, head_dim=m.dim, key_dim=m.rot_dim, value_dim=m.vdim, rope_dim=m.rot_dims, rope_base=m.rot_base,
                               scale=m.scale, eps=c.norm_eps, weight_bias=0.0, weight=p + "mix.dkv.norm", weight2=p + "mix.uk", weight3=p + "mix.uv",
                               **({} if scaling is None else dict(rope_factor=scaling.factor, rope_original=scaling.original,
                                                                  rope_fast=scaling.fast, rope_slow=scaling.slow))))
            product(p + "mix.o", BUF_S0, BUF_HIDDEN, w, m.heads * m.vdim)
            post = p + "norm1b"
            if layer.ff:
                norm(p + "norm2")
                product(p + "mlp.gate", BUF_S0, BUF_S1, layer.ff, w)
                product(p + "mlp.up", BUF_S0, BUF_S2, layer.ff, w)
                steps.append(_step(STEP_GEGLU, in_buf=BUF_S1, in2_buf=BUF_S2, out_buf=BUF_S1, n=layer.ff))
                product(p + "mlp.down", BUF_S1, BUF_HIDDEN, w, layer.ff)
                post = p + "norm2b"
        norm("final.norm", last=True)
        product("head", BUF_S0, BUF_LOGITS, c.vocab, w)
        steps.append(_step(STEP_ARGMAX, in_buf=BUF_LOGITS, n=c.vocab))
        return steps

    def with_runtime(self, **changes) -> "VuzunexPlanBuilder":
        """The same model with other runtime sizes (max_seq, max_batch, pool_tokens, dtype)."""
        return VuzunexPlanBuilder(dataclasses.replace(self.config, **changes))
