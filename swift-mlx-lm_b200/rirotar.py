"""Rirotar recipe: config.json -> RirotarConfig -> fp32-stream step list.

A pre-norm decoder whose layers are listed one by one. A layer's mixer is a gated delta rule with one decay per head ("delta")
or per head and key channel ("channel_delta"), or latent attention without positions over a sliding window with a sink
("latent_attention"); its feed-forward is a clamped gated one, dense or routed over experts, or missing. The logits are soft
capped. Nothing here computes or caches: the steps run through the same plan, pool, executor and kernels as any other
fp32-stream plan.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass, field
from typing import Dict, List, Mapping, Optional, Tuple, Union

from .lib import BuffersDesc, Step
from .plan import (BUF_HIDDEN, BUF_LOGITS, BUF_S0, BUF_S1, BUF_S2, BUF_S3, BUF_S4, GATE_SIGMOID, GATE_SILU, SHARD_REPLICATE, STEP_ARGMAX,
                   STEP_CLAMPED_GLU, STEP_COPY_RMSNORM, STEP_EMBED, STEP_GATED_DELTA, STEP_LATENT_ATTN, STEP_PRODUCT,
                   STEP_RESADD_COPY_RMSNORM, STEP_RESADD_RMSNORM, STEP_ROUTED_MLP, STEP_SOFTCAP, STREAM_ALL_F32, STREAM_F32, _step)

ARCHITECTURE = "Rirotar"

# constants of the design
GLU_ALPHA = 1.702
UNIT_EPS = 1e-6


@dataclass(frozen=True)
class WindowedLatentAttention:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int       # a token sees itself and the window - 1 before it; 0: everything


@dataclass(frozen=True)
class GatedDelta:
    heads: int
    kv_heads: int     # q and k heads; heads / kv_heads value heads share one
    dim: int
    vdim: int
    conv: int         # taps of the short convolutions
    channel: bool     # a decay per key channel instead of one per head, and a sigmoid output gate instead of a silu one
    decay_rank: int = 0   # inner sizes of the two-factor projections (channel only)
    gate_rank: int = 0


@dataclass(frozen=True)
class DenseFF:
    ff: int
    limit: float


@dataclass(frozen=True)
class RoutedFF:
    ff: int
    limit: float
    experts: int
    top: int
    groups: int
    groups_keep: int
    scale: float


@dataclass(frozen=True)
class Layer:
    mixer: Union[WindowedLatentAttention, GatedDelta]
    mlp: Union[DenseFF, RoutedFF, None]


@dataclass
class RirotarConfig:
    vocab: int
    width: int
    layers: List[Layer] = field(default_factory=list)
    norm_eps: float = 1e-5
    logit_softcap: float = 0.0   # 0: none
    dtype: str = "bfloat16"      # or "float32": everything in fp32
    max_seq: int = 4224
    max_batch: int = 1
    pool_tokens: int = 0         # tokens the page pool holds over all sequences; 0 = max_batch * max_seq

    def _count(self, kind) -> int:
        return sum(isinstance(layer.mixer, kind) for layer in self.layers)

    def buffers_desc(self) -> BuffersDesc:
        return BuffersDesc(hidden=self.width, vocab=self.vocab, max_seq=self.max_seq, max_batch=self.max_batch,
                           stream_dtype=STREAM_ALL_F32 if self.dtype == "float32" else STREAM_F32,
                           latent_layers=self._count(WindowedLatentAttention), delta_layers=self._count(GatedDelta), kv_pool_tokens=self.pool_tokens)

    def product_elems(self) -> int:
        """Entries of the matrices the dense products of one decode step read (the routed experts not among them)."""
        total = self.vocab * self.width
        for layer in self.layers:
            m, w = layer.mixer, self.width
            if isinstance(m, GatedDelta):
                total += w * (2 * m.kv_heads * m.dim + 2 * m.heads * m.vdim + m.heads)
                if m.channel:
                    total += m.decay_rank * (w + m.heads * m.dim) + m.gate_rank * (w + m.heads * m.vdim)
                else:
                    total += w * (m.heads + m.heads * m.vdim)
            else:
                total += w * (m.heads * (m.dim + m.vdim) + m.kv_rank)
            if isinstance(layer.mlp, DenseFF):
                total += 3 * w * layer.mlp.ff
            elif layer.mlp is not None:
                total += layer.mlp.experts * w
        return total


def _mixer(i: int, entry: Dict, shapes: Mapping[str, Tuple[int, ...]]) -> Union[WindowedLatentAttention, GatedDelta]:
    m, kind = entry["mixer"], entry["type"]
    if kind == "latent_attention":
        if m.get("rot_dim"):
            raise ValueError(f"layer {i}: latent attention of this design has no rotated part")
        mask = m.get("mask")
        window = 0 if mask is None else int(mask["size"])
        if mask is not None and window < 1:
            raise ValueError(f"layer {i}: window of {window}")
        return WindowedLatentAttention(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                                       scale=float(m["scale"]), window=window)
    if kind not in ("delta", "channel_delta"):
        raise ValueError(f"layer {i}: mixer type {kind!r}")
    channel = kind == "channel_delta"
    heads, kv = int(m["heads"]), int(m["kv_heads"])
    if heads % kv:
        raise ValueError(f"layer {i}: {heads} heads over {kv} query / key heads")
    ranks = {}
    if channel:   # config.json does not give these; the tensors do
        ranks = {"decay_rank": int(shapes[f"l{i}.mix.a1"][0]), "gate_rank": int(shapes[f"l{i}.mix.g1"][0])}
    return GatedDelta(heads=heads, kv_heads=kv, dim=int(m["dim"]), vdim=int(m["vdim"]), conv=int(m["conv"]), channel=channel, **ranks)


def _feed_forward(i: int, mlp: Optional[Dict]) -> Union[DenseFF, RoutedFF, None]:
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return DenseFF(ff=int(mlp["ff"]), limit=float(mlp["limit"]))
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
    router, expert = mlp["router"], mlp["expert"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    out = RoutedFF(ff=int(expert["ff"]), limit=float(expert["limit"]), experts=int(router["experts"]), top=int(router["top"]),
                   groups=int(groups["count"]), groups_keep=int(groups["keep"]), scale=float(router["scale"]))
    if out.experts % out.groups or not 1 <= out.groups_keep <= out.groups or not 1 <= out.top <= out.groups_keep * (out.experts // out.groups):
        raise ValueError(f"layer {i}: {out.top} of {out.experts} experts, {out.groups_keep} of {out.groups} groups")
    return out


def decode_config(config: Dict, shapes: Mapping[str, Tuple[int, ...]], dtype: str = "bfloat16", max_seq: int = 4224, max_batch: int = 1,
                  pool_tokens: int = 0) -> RirotarConfig:
    """config.json of a Rirotar checkpoint; `shapes` are those of its tensors (the inner sizes of the two-factor projections stand
    nowhere else). A value this recipe cannot express is refused."""
    if config.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {config.get('architecture')!r} is not {ARCHITECTURE}")
    if dtype not in ("bfloat16", "float32"):
        raise ValueError(f"dtype {dtype!r}: bfloat16 or float32")
    layers = [Layer(mixer=_mixer(i, entry, shapes), mlp=_feed_forward(i, entry.get("mlp"))) for i, entry in enumerate(config["layers"])]
    return RirotarConfig(vocab=int(config["vocab"]), width=int(config["width"]), layers=layers, norm_eps=float(config["norm"]["eps"]),
                         logit_softcap=float(config.get("logit_softcap") or 0.0), dtype=dtype, max_seq=max_seq, max_batch=max_batch,
                         pool_tokens=pool_tokens)


class RirotarPlanBuilder:
    """Tensor inventory and step list of a RirotarConfig (the counterpart of plan.DispatchPlanBuilder)."""

    def __init__(self, config: RirotarConfig):
        self.config = config

    def tensors(self):
        """(name, kind, shape, shard kind): `matrix` = operand of a product, `norm0` = norm weight stored around zero,
        `norm` = plain norm weight, `dense` = the embedding table and small vectors, `taps` = a short convolution's."""
        c, w = self.config, self.config.width
        out = [("embed", "dense", (c.vocab, w))]
        for i, layer in enumerate(c.layers):
            p, m = f"l{i}.", layer.mixer
            x = p + "mix."
            out.append((p + "norm1", "norm0", (w,)))
            if isinstance(m, WindowedLatentAttention):
                out += [(x + "q", "matrix", (m.heads * m.dim, w)), (x + "dkv", "matrix", (m.kv_rank, w)), (x + "dkv.norm", "norm", (m.kv_rank,)),
                        (x + "uk", "matrix", (m.heads * m.dim, m.kv_rank)), (x + "uv", "matrix", (m.heads * m.vdim, m.kv_rank)),
                        (x + "sink", "dense", (m.heads,))]
            else:
                for t, rows in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.heads * m.vdim)):
                    out += [(x + t, "matrix", (rows, w)), (x + t + ".conv", "taps", (rows, m.conv))]
                out += [(x + "b", "matrix", (m.heads, w)), (x + "A_log", "dense", (m.heads,)), (x + "norm", "norm", (m.vdim,))]
                if m.channel:
                    out += [(x + "a1", "matrix", (m.decay_rank, w)), (x + "a2", "matrix", (m.heads * m.dim, m.decay_rank)),
                            (x + "dt_bias", "dense", (m.heads * m.dim,)),
                            (x + "g1", "matrix", (m.gate_rank, w)), (x + "g2", "matrix", (m.heads * m.vdim, m.gate_rank))]
                else:
                    out += [(x + "a", "matrix", (m.heads, w)), (x + "dt_bias", "dense", (m.heads,)), (x + "g", "matrix", (m.heads * m.vdim, w))]
            out.append((x + "o", "matrix", (w, m.heads * m.vdim)))
            if layer.mlp is None:
                continue
            out.append((p + "norm2", "norm0", (w,)))
            ff = layer.mlp.ff
            routed = isinstance(layer.mlp, RoutedFF)
            for prefix in ([f"{p}mlp.e{e}." for e in range(layer.mlp.experts)] if routed else [p + "mlp."]):
                out += [(prefix + "gate", "matrix", (ff, w)), (prefix + "up", "matrix", (ff, w)), (prefix + "down", "matrix", (w, ff))]
            if routed:
                out.append((p + "mlp.router", "matrix", (layer.mlp.experts, w)))
        out += [("final.norm", "norm0", (w,)), ("head", "matrix", (c.vocab, w))]
        return [t + (SHARD_REPLICATE,) for t in out]

    def decode_steps(self, layers: Optional[int] = None, store_final: bool = False) -> List[Step]:
        """The steps of one token. `layers` stops after that many layers; `store_final` keeps the residual stream behind the last
        one in its buffer (both for tests that look at the stream)."""
        c, w = self.config, self.config.width
        steps = [_step(STEP_EMBED, out_buf=BUF_HIDDEN, n=w, weight="embed")]
        latent = delta = 0

        def norm(name: str, last: bool = False):
            kind = STEP_COPY_RMSNORM if len(steps) == 1 else STEP_RESADD_RMSNORM if last and not store_final else STEP_RESADD_COPY_RMSNORM
            steps.append(_step(kind, in_buf=BUF_HIDDEN, out_buf=BUF_S0, n=w, eps=c.norm_eps, weight_bias=1.0, weight=name))

        def product(name: str, src: int, dst: int, n: int, k: int, src_off: int = 0, dst_off: int = 0):
            steps.append(_step(STEP_PRODUCT, in_buf=src, out_buf=dst, n=n, k=k, in_off=src_off, out_off=dst_off, weight=name))

        for i, layer in enumerate(c.layers[:layers]):
            p, m = f"l{i}.", layer.mixer
            x = p + "mix."
            norm(p + "norm1")
            if isinstance(m, WindowedLatentAttention):
                product(x + "q", BUF_S0, BUF_S1, m.heads * m.dim, w)
                product(x + "dkv", BUF_S0, BUF_S3, m.kv_rank, w)
                steps.append(_step(STEP_LATENT_ATTN, layer=latent, in_buf=BUF_S1, in2_buf=BUF_S3, out_buf=BUF_S0, n=m.kv_rank, heads=m.heads,
                                   head_dim=m.dim, key_dim=0, value_dim=m.vdim, rope_dim=0, scale=m.scale, eps=c.norm_eps, weight_bias=0.0,
                                   window_left=m.window, weight=x + "dkv.norm", weight2=x + "uk", weight3=x + "uv", weight4=x + "sink"))
                latent += 1
            else:
                self._delta(steps, product, x, m, delta)
                delta += 1
            product(x + "o", BUF_S0, BUF_HIDDEN, w, m.heads * m.vdim)
            if layer.mlp is None:
                continue
            norm(p + "norm2")
            ff, mlp = layer.mlp.ff, layer.mlp
            if isinstance(mlp, DenseFF):
                product(p + "mlp.gate", BUF_S0, BUF_S1, ff, w)
                product(p + "mlp.up", BUF_S0, BUF_S2, ff, w)
                steps.append(_step(STEP_CLAMPED_GLU, in_buf=BUF_S1, in2_buf=BUF_S2, out_buf=BUF_S1, n=ff, scale=GLU_ALPHA, limit=mlp.limit))
                product(p + "mlp.down", BUF_S1, BUF_HIDDEN, w, ff)
            else:
                product(p + "mlp.router", BUF_S0, BUF_S3, mlp.experts, w)
                steps.append(_step(STEP_ROUTED_MLP, in_buf=BUF_S0, in2_buf=BUF_S3, out_buf=BUF_HIDDEN, n=w, k=ff, experts=mlp.experts, top=mlp.top,
                                   groups=mlp.groups, groups_keep=mlp.groups_keep, scale=mlp.scale, limit=mlp.limit, glu_alpha=GLU_ALPHA,
                                   weight=p + "mlp.e", weight2=".gate", weight3=".up", weight4=".down"))
        norm("final.norm", last=True)
        product("head", BUF_S0, BUF_LOGITS, c.vocab, w)
        if c.logit_softcap:
            steps.append(_step(STEP_SOFTCAP, in_buf=BUF_LOGITS, n=c.vocab, scale=c.logit_softcap))
        steps.append(_step(STEP_ARGMAX, in_buf=BUF_LOGITS, n=c.vocab))
        return steps

    def _delta(self, steps: List[Step], product, x: str, m: GatedDelta, index: int) -> None:
        """q | k | v side by side in one buffer; everything that reads the normed stream is one product over concatenated rows."""
        w, gk, hv = self.config.width, m.kv_heads * m.dim, m.heads * m.vdim

        def up8(v: int) -> int:
            return -(-v // 8) * 8

        product(x + "q", BUF_S0, BUF_S1, gk, w)
        product(x + "k", BUF_S0, BUF_S1, gk, w, dst_off=gk)
        product(x + "v", BUF_S0, BUF_S1, hv, w, dst_off=2 * gk)
        product(x + "b", BUF_S0, BUF_S3, m.heads, w)
        if m.channel:
            at = up8(m.decay_rank)
            product(x + "a1", BUF_S0, BUF_S2, m.decay_rank, w)
            product(x + "g1", BUF_S0, BUF_S2, m.gate_rank, w, dst_off=at)
            product(x + "a2", BUF_S2, BUF_S4, m.heads * m.dim, m.decay_rank)
            product(x + "g2", BUF_S2, BUF_S0, hv, m.gate_rank, src_off=at)
            gate, inputs, act = BUF_S0, m.dim, GATE_SIGMOID
        else:
            product(x + "a", BUF_S0, BUF_S4, m.heads, w)
            product(x + "g", BUF_S0, BUF_S2, hv, w)
            gate, inputs, act = BUF_S2, 1, GATE_SILU
        steps.append(_step(STEP_GATED_DELTA, layer=index, in_buf=BUF_S1, in2_buf=BUF_S3, in3_buf=BUF_S4, in4_buf=gate, out_buf=BUF_S0, k=inputs,
                           heads=m.heads, groups=m.kv_heads, key_dim=m.dim, value_dim=m.vdim, conv_kernel=m.conv, eps=self.config.norm_eps,
                           eps2=UNIT_EPS, scale=m.dim ** -0.5, gate_act=act, weight=x + "q.conv", weight2=x + "k.conv", weight3=x + "v.conv",
                           weight4=x + "norm", weight5=x + "A_log", weight6=x + "dt_bias"))

    def with_runtime(self, **changes) -> "RirotarPlanBuilder":
        """The same model with other runtime sizes (max_seq, max_batch, pool_tokens, dtype)."""
        return RirotarPlanBuilder(dataclasses.replace(self.config, **changes))
