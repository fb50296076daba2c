"""Kalevik recipe: config.json -> KalevikConfig -> fp32-stream step list.

A decoder with a norm before and after every sublayer whose layers are listed one by one. A layer's mixer is latent attention with
a rotated key part ("latent_attention"), or grouped-query attention over chunks of positions and a retention side by side
("parallel"); its feed-forward is dense, routed over experts with a shared one, or missing. A range of layers may run several
times, every pass with caches and states of its own and, from the second on, with the embedding added in front of it. Nothing here
computes or caches: the steps run through the same plan, pools, states, executor and kernels as any other fp32-stream plan.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass, field
from typing import Dict, List, Mapping, Optional, Tuple, Union

import numpy as np

from .lib import BuffersDesc, Step
from .plan import (BUF_HIDDEN, BUF_LOGITS, BUF_S0, BUF_S1, BUF_S2, BUF_S3, BUF_S4, ROPE_HALVES, ROPE_NEIGHBOURS, SCORE_SOFTMAX, SHARD_REPLICATE,
                   STEP_ARGMAX, STEP_COPY_RMSNORM, STEP_EMBED, STEP_GROUPED_ATTN, STEP_LATENT_ATTN, STEP_POSTNORM_RESADD_COPY_RMSNORM,
                   STEP_POSTNORM_RESADD_RMSNORM, STEP_PRODUCT, STEP_RETENTION, STEP_ROUTED_MLP, STEP_SWIGLU, STREAM_ALL_F32, STREAM_F32, _step)

ARCHITECTURE = "Kalevik"


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


@dataclass(frozen=True)
class ChunkedAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int        # a token sees the earlier ones of its own chunk; 0: everything
    rot_base: float
    rot_dims: int
    rot_divisor: float = 1.0


@dataclass(frozen=True)
class Retention:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class Parallel:
    left: ChunkedAttention
    right: Retention
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class DenseFF:
    ff: int


@dataclass(frozen=True)
class RoutedFF:
    ff: int
    experts: int
    top: int
    groups: int
    groups_keep: int
    shared_ff: int    # 0: no shared expert


@dataclass(frozen=True)
class Layer:
    mixer: Union[LatentAttention, Parallel]
    mlp: Union[DenseFF, RoutedFF, None]


@dataclass
class KalevikConfig:
    vocab: int
    width: int
    layers: List[Layer] = field(default_factory=list)
    loop: Tuple[int, int, int] = (0, 0, 1)   # layers [first, past the last) run `times` times in a row
    embedding_scale: float = 1.0
    norm_eps: float = 1e-6
    dtype: str = "bfloat16"      # or "float32": everything in fp32
    max_seq: int = 4224
    max_batch: int = 1
    pool_tokens: int = 0         # tokens the page pools hold over all sequences; 0 = max_batch * max_seq

    def runs(self) -> List[Tuple[int, bool]]:
        """(layer, is the embedding added in front of it) in the order of execution."""
        first, past, times = self.loop
        out = [(i, False) for i in range(first)]
        for turn in range(times):
            out += [(i, turn > 0 and i == first) for i in range(first, past)]
        return out + [(i, False) for i in range(past, len(self.layers))]

    def _count(self, kind) -> int:
        return sum(isinstance(self.layers[i].mixer, kind) for i, _ in self.runs())

    def buffers_desc(self) -> BuffersDesc:
        parallel = self._count(Parallel)
        return BuffersDesc(hidden=self.width, vocab=self.vocab, max_seq=self.max_seq, max_batch=self.max_batch,
                           stream_dtype=STREAM_ALL_F32 if self.dtype == "float32" else STREAM_F32, latent_layers=self._count(LatentAttention),
                           delta_layers=parallel, grouped_layers=parallel, kv_pool_tokens=self.pool_tokens)

    def product_elems(self) -> int:
        """Entries of the matrices the dense products of one decode step read (experts not among them; a layer that runs again
        counts again)."""
        total, w = self.vocab * self.width, self.width
        for i, _ in self.runs():
            m, mlp = self.layers[i].mixer, self.layers[i].mlp
            if isinstance(m, Parallel):
                a, r = m.left, m.right
                total += w * (a.heads * (a.dim + a.vdim + 1) + a.kv_heads * (a.dim + a.vdim))
                total += w * r.heads * (2 * r.dim + 3 * r.vdim)
            else:
                total += w * (m.heads * (m.dim + m.rot_dim + m.vdim) + m.kv_rank + m.rot_dim)
            if isinstance(mlp, DenseFF):
                total += 3 * w * mlp.ff
            elif mlp is not None:
                total += w * (mlp.experts + (1 if mlp.shared_ff else 0))
        return total


def _up8(v: int) -> int:
    return -(-v // 8) * 8


def _rotation(i: int, m: Dict, size: int) -> Tuple[float, int]:
    rot = m["rot"]
    if rot["dims"] > size or rot["dims"] % 2:
        raise ValueError(f"layer {i}: {rot['dims']} rotated entries of {size}")
    return float(rot["base"]), int(rot["dims"])


def _mixer(i: int, entry: Dict) -> Union[LatentAttention, Parallel]:
    m, kind = entry["mixer"], entry["type"]
    if kind == "latent_attention":
        base, dims = _rotation(i, m, m["rot_dim"])
        return LatentAttention(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                               scale=float(m["scale"]), rot_base=base, rot_dims=dims)
    if kind != "parallel":
        raise ValueError(f"layer {i}: mixer type {kind!r}")
    a, r = m["left"], m["right"]
    heads, kv = int(a["heads"]), int(a["kv_heads"])
    if heads % kv:
        raise ValueError(f"layer {i}: {heads} heads over {kv} key / value heads")
    mask = a.get("mask")
    chunk = 0 if mask is None else int(mask["size"])
    if mask is not None and chunk < 1:
        raise ValueError(f"layer {i}: chunks of {chunk}")
    base, dims = _rotation(i, a, a["dim"])
    scaling = a["rot"].get("scaling")
    left = ChunkedAttention(heads=heads, kv_heads=kv, dim=int(a["dim"]), vdim=int(a["vdim"]), scale=float(a["scale"]), chunk=chunk, rot_base=base,
                            rot_dims=dims, rot_divisor=1.0 if scaling is None else float(scaling["factor"]))
    right = Retention(heads=int(r["heads"]), dim=int(r["dim"]), vdim=int(r["vdim"]), decay=tuple(float(d) for d in r["decay"]))
    if len(right.decay) != right.heads:
        raise ValueError(f"layer {i}: {len(right.decay)} decays for {right.heads} heads")
    return Parallel(left, right, float(m["left_scale"]), float(m["right_scale"]))


def _feed_forward(i: int, mlp: Optional[Dict]) -> Union[DenseFF, RoutedFF, None]:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return DenseFF(ff=int(mlp["ff"]))
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
    router, groups, shared = mlp["router"], mlp["router"].get("groups") or {"count": 1, "keep": 1}, mlp.get("shared")
    out = RoutedFF(ff=int(mlp["expert"]["ff"]), experts=int(router["experts"]), top=int(router["top"]), groups=int(groups["count"]),
                   groups_keep=int(groups["keep"]), shared_ff=0 if shared is None else int(shared["ff"]))
    if out.experts % out.groups or not 1 <= out.groups_keep <= out.groups or not 1 <= out.top <= out.groups_keep * (out.experts // out.groups):
        raise ValueError(f"layer {i}: {out.top} of {out.experts} experts, {out.groups_keep} of {out.groups} groups")
    return out


def decode_config(config: Dict, shapes: Optional[Mapping[str, Tuple[int, ...]]] = None, dtype: str = "bfloat16", max_seq: int = 4224, max_batch: int = 1,
                  pool_tokens: int = 0) -> KalevikConfig:
    """config.json of a Kalevik checkpoint. Every entry is read from the file; a value this recipe cannot express is refused."""
    if config.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {config.get('architecture')!r} is not {ARCHITECTURE}")
    if dtype not in ("bfloat16", "float32"):
        raise ValueError(f"dtype {dtype!r}: bfloat16 or float32")
    layers = [Layer(mixer=_mixer(i, entry), mlp=_feed_forward(i, entry.get("mlp"))) for i, entry in enumerate(config["layers"])]
    loop = config.get("loop")
    span = (0, 0, 1) if loop is None else (int(loop["start"]), int(loop["stop"]), int(loop["times"]))
    if not 0 <= span[0] <= span[1] <= len(layers) or span[2] < 1:
        raise ValueError(f"loop over layers {span[0]} .. {span[1]} of {len(layers)}, {span[2]} times")
    return KalevikConfig(vocab=int(config["vocab"]), width=int(config["width"]), layers=layers, loop=span,
                         embedding_scale=float(config["embedding"]["scale"]), norm_eps=float(config["norm"]["eps"]), dtype=dtype, max_seq=max_seq,
                         max_batch=max_batch, pool_tokens=pool_tokens)


class KalevikPlanBuilder:
    """Tensor inventory and step list of a KalevikConfig (the counterpart of plan.DispatchPlanBuilder)."""

    def __init__(self, config: KalevikConfig):
        self.config = config

    def tensors(self):
        """(name, kind, shape, shard kind): `matrix` = operand of a product, `norm` = norm weight, `dense` = the embedding table."""
        c, w = self.config, self.config.width
        out = [("embed", "dense", (c.vocab, w))]
        for i, layer in enumerate(c.layers):
            p, m, mlp = f"l{i}.", layer.mixer, layer.mlp
            x = p + "mix."
            out += [(p + "norm1", "norm", (w,)), (p + "norm1b", "norm", (w,))]
            if isinstance(m, LatentAttention):
                out += [(x + "q", "matrix", (m.heads * (m.dim + m.rot_dim), w)), (x + "dkv", "matrix", (m.kv_rank + m.rot_dim, w)),
                        (x + "dkv.norm", "norm", (m.kv_rank,)), (x + "uk", "matrix", (m.heads * m.dim, m.kv_rank)),
                        (x + "uv", "matrix", (m.heads * m.vdim, m.kv_rank)), (x + "o", "matrix", (w, m.heads * m.vdim))]
            else:
                a, r = m.left, m.right
                out += [(x + "left.q", "matrix", (a.heads * a.dim, w)), (x + "left.k", "matrix", (a.kv_heads * a.dim, w)),
                        (x + "left.v", "matrix", (a.kv_heads * a.vdim, w)), (x + "left.q.norm", "norm", (a.dim,)), (x + "left.k.norm", "norm", (a.dim,)),
                        (x + "left.g", "matrix", (a.heads, w)), (x + "left.o", "matrix", (w, a.heads * a.vdim)),
                        (x + "right.q", "matrix", (r.heads * r.dim, w)), (x + "right.k", "matrix", (r.heads * r.dim, w)),
                        (x + "right.v", "matrix", (r.heads * r.vdim, w)), (x + "right.g", "matrix", (r.heads * r.vdim, w)),
                        (x + "right.o", "matrix", (w, r.heads * r.vdim))]
            if mlp is None:
                continue
            out += [(p + "norm2", "norm", (w,)), (p + "norm2b", "norm", (w,))]
            if isinstance(mlp, DenseFF):
                out += [(p + "mlp.gate", "matrix", (mlp.ff, w)), (p + "mlp.up", "matrix", (mlp.ff, w)), (p + "mlp.down", "matrix", (w, mlp.ff))]
                continue
            feeds = [(f"{p}mlp.e{e}", mlp.ff) for e in range(mlp.experts)]
            out.append((p + "mlp.router", "matrix", (mlp.experts, w)))
            if mlp.shared_ff:
                feeds.append((p + "mlp.shared", mlp.shared_ff))
                out.append((p + "mlp.shared.sg", "matrix", (1, w)))
            for name, ff in feeds:
                out += [(name + ".up", "matrix", (ff, w)), (name + ".down", "matrix", (w, ff))]
        out += [("final.norm", "norm", (w,)), ("head", "matrix", (c.vocab, w))]
        return [t + (SHARD_REPLICATE,) for t in out]

    def constants(self) -> Dict[str, np.ndarray]:
        """fp32 tensors of the plan that stand in the configuration instead of the checkpoint."""
        return {f"l{i}.mix.right.decay": np.asarray(layer.mixer.right.decay, dtype=np.float32)
                for i, layer in enumerate(self.config.layers) if isinstance(layer.mixer, Parallel)}

    def decode_steps(self, runs: Optional[int] = None, store_final: bool = False) -> List[Step]:
        """The steps of one token. `runs` stops after that many layer runs; `store_final` keeps the residual stream behind the
        last one in its buffer (both for tests that look at the stream)."""
        c, w = self.config, self.config.width
        steps = [_step(STEP_EMBED, out_buf=BUF_HIDDEN, n=w, scale=c.embedding_scale, weight="embed")]
        post = None   # norm of the sublayer whose output waits in the hidden buffer
        latent = parallel = 0

        def norm(name: str, last: bool = False, joins: bool = False):
            common = dict(in_buf=BUF_HIDDEN, out_buf=BUF_S0, n=w, eps=c.norm_eps, weight_bias=0.0)
            if post is None:
                steps.append(_step(STEP_COPY_RMSNORM, weight=name, **common))
                return
            if joins:
                common.update(weight3="embed", scale=c.embedding_scale)
            kind = STEP_POSTNORM_RESADD_RMSNORM if last and not store_final else STEP_POSTNORM_RESADD_COPY_RMSNORM
            steps.append(_step(kind, weight=post, weight2=name, **common))

        def product(name: str, src: int, dst: int, n: int, k: int, dst_off: int = 0, **more):
            steps.append(_step(STEP_PRODUCT, in_buf=src, out_buf=dst, n=n, k=k, out_off=dst_off, weight=name, **more))

        for i, joins in c.runs()[:runs]:
            p, m, mlp = f"l{i}.", c.layers[i].mixer, c.layers[i].mlp
            x = p + "mix."
            norm(p + "norm1", joins=joins)
            if isinstance(m, LatentAttention):
                product(x + "q", BUF_S0, BUF_S1, m.heads * (m.dim + m.rot_dim), w)
                product(x + "dkv", BUF_S0, BUF_S3, m.kv_rank + m.rot_dim, w)
                steps.append(_step(STEP_LATENT_ATTN, layer=latent, in_buf=BUF_S1, in2_buf=BUF_S3, out_buf=BUF_S0, n=m.kv_rank, heads=m.heads,
                                   head_dim=m.dim, key_dim=m.rot_dim, value_dim=m.vdim, rope_dim=m.rot_dims, rope_base=m.rot_base,
                                   rope_pairs=ROPE_NEIGHBOURS, scale=m.scale, eps=c.norm_eps, weight_bias=0.0, weight=x + "dkv.norm",
                                   weight2=x + "uk", weight3=x + "uv"))
                product(x + "o", BUF_S0, BUF_HIDDEN, w, m.heads * m.vdim)
                latent += 1
            else:
                self._parallel(steps, product, x, m, parallel)
                parallel += 1
            post = p + "norm1b"
            if mlp is None:
                continue
            norm(p + "norm2")
            post = p + "norm2b"
            if isinstance(mlp, DenseFF):
                product(p + "mlp.gate", BUF_S0, BUF_S1, mlp.ff, w)
                product(p + "mlp.up", BUF_S0, BUF_S2, mlp.ff, w)
                steps.append(_step(STEP_SWIGLU, in_buf=BUF_S1, in2_buf=BUF_S2, out_buf=BUF_S1, n=mlp.ff))
                product(p + "mlp.down", BUF_S1, BUF_HIDDEN, w, mlp.ff)
                continue
            product(p + "mlp.router", BUF_S0, BUF_S3, mlp.experts, w)
            shared = {}
            if mlp.shared_ff:
                product(p + "mlp.shared.sg", BUF_S0, BUF_S3, 1, w, dst_off=mlp.experts)
                shared = dict(weight5=p + "mlp.shared.up", weight6=p + "mlp.shared.down", k2=mlp.shared_ff)
            steps.append(_step(STEP_ROUTED_MLP, in_buf=BUF_S0, in2_buf=BUF_S3, out_buf=BUF_HIDDEN, n=w, k=mlp.ff, experts=mlp.experts, top=mlp.top,
                               groups=mlp.groups, groups_keep=mlp.groups_keep, scale=1.0, score_act=SCORE_SOFTMAX, group_best=1, raw_weights=1,
                               weight=p + "mlp.e", weight3=".up", weight4=".down", **shared))
        norm("final.norm", last=True)
        product("head", BUF_S0, BUF_LOGITS, c.vocab, w)
        steps.append(_step(STEP_ARGMAX, in_buf=BUF_LOGITS, n=c.vocab))
        return steps

    def _parallel(self, steps: List[Step], product, x: str, m: Parallel, index: int) -> None:
        """Everything that reads the normed stream is one product over concatenated rows; both mixers leave their heads side by
        side, already scaled, so that one product over both output matrices ends the layer."""
        w, a, r = self.config.width, m.left, m.right
        qa, ka, va, qr, vr = a.heads * a.dim, a.kv_heads * a.dim, a.kv_heads * a.vdim, r.heads * r.dim, r.heads * r.vdim
        gate_at, right_at = _up8(qa + ka + va), _up8(a.heads * a.vdim)
        product(x + "left.q", BUF_S0, BUF_S1, qa, w)
        product(x + "left.k", BUF_S0, BUF_S1, ka, w, dst_off=qa)
        product(x + "left.v", BUF_S0, BUF_S1, va, w, dst_off=qa + ka)
        product(x + "right.g", BUF_S0, BUF_S1, vr, w, dst_off=gate_at)
        product(x + "left.g", BUF_S0, BUF_S4, a.heads, w)
        product(x + "right.q", BUF_S0, BUF_S2, qr, w)
        product(x + "right.k", BUF_S0, BUF_S2, qr, w, dst_off=qr)
        product(x + "right.v", BUF_S0, BUF_S2, vr, w, dst_off=2 * qr)
        steps.append(_step(STEP_GROUPED_ATTN, layer=index, in_buf=BUF_S1, in3_buf=BUF_S4, out_buf=BUF_S0, heads=a.heads, kv_heads=a.kv_heads,
                           head_dim=a.dim, value_dim=a.vdim, rope_dim=a.rot_dims, rope_base=a.rot_base, rope_divisor=a.rot_divisor,
                           rope_pairs=ROPE_HALVES, scale=a.scale, chunk=a.chunk, sink_one=1, eps=self.config.norm_eps, weight_bias=0.0,
                           out_scale=m.left_scale, weight=x + "left.q.norm", weight2=x + "left.k.norm"))
        steps.append(_step(STEP_RETENTION, layer=index, in_buf=BUF_S2, in4_buf=BUF_S1, in4_off=gate_at, out_buf=BUF_S0, out_off=right_at,
                           heads=r.heads, key_dim=r.dim, value_dim=r.vdim, scale=r.dim ** -0.5, eps=self.config.norm_eps,
                           out_scale=m.right_scale, weight=x + "right.decay"))
        product(x + "left.o", BUF_S0, BUF_HIDDEN, w, a.heads * a.vdim, weight2=x + "right.o", k2=vr)

    def with_runtime(self, **changes) -> "KalevikPlanBuilder":
        """The same model with other runtime sizes (max_seq, max_batch, pool_tokens, dtype)."""
        return KalevikPlanBuilder(dataclasses.replace(self.config, **changes))
