"""Merudra recipe: config.json -> MerudraConfig -> fp32-stream step list.

A decoder whose sublayers read the residual stream itself, joined with a short causal convolution over it, and whose results are
gated by the stream and normed before they are added. Layers are listed one by one; a layer's mixer is grouped-query attention
without rotation whose values are its keys ("attention"), or a gated delta rule with one decay per head ("delta"); its
feed-forward is routed over experts, some of which hand their input through, or missing. Behind the feed-forward every layer
takes an input of its own per token, and what it passes on is a weighted sum of the results of all layers so far. Nothing here
computes or caches: the steps run through the same plan, pools, states, executor and kernels as any other fp32-stream plan.
"""
from __future__ import annotations

import dataclasses
from dataclasses import dataclass, field
from typing import Dict, List, Mapping, Optional, Tuple, Union

from .lib import BuffersDesc, Step
from .plan import (BUF_HIDDEN, BUF_LOGITS, BUF_RESIDUAL, BUF_S0, BUF_S1, BUF_S2, BUF_S3, BUF_S4, EXPERT_SILU, GATE_SILU, SCORE_SOFTMAX, SHARD_REPLICATE,
                   STEP_ARGMAX, STEP_COPY_RMSNORM, STEP_DEPTH_AVG, STEP_EMBED, STEP_GATED_DELTA, STEP_GATED_POSTNORM_ADD, STEP_GROUPED_ATTN, STEP_PRODUCT,
                   STEP_ROUTED_MLP, STEP_STREAM_CONV, STEP_STREAM_COPY, STEP_TOKEN_GATE, STREAM_ALL_F32, STREAM_F32, _step)

ARCHITECTURE = "Merudra"

# constant of the design
UNIT_EPS = 1e-6


@dataclass(frozen=True)
class KeyValueAttention:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    temp_coef: float = 0.0
    temp_every: int = 0   # 0: no query temperature


@dataclass(frozen=True)
class GatedDelta:
    heads: int
    kv_heads: int     # q and k heads; heads / kv_heads value heads share one
    dim: int
    vdim: int
    conv: int         # taps of the short convolutions of q, k and v


@dataclass(frozen=True)
class RoutedFF:
    ff: int
    experts: int
    identity: int     # experts without tensors behind them
    top: int


@dataclass(frozen=True)
class Layer:
    mixer: Union[KeyValueAttention, GatedDelta]
    mlp: Optional[RoutedFF]


@dataclass
class MerudraConfig:
    vocab: int
    width: int
    taps: int                    # of the convolutions over the stream
    side: int                    # entries a token brings to a layer
    layers: List[Layer] = field(default_factory=list)
    norm_eps: float = 1e-6
    dtype: str = "bfloat16"      # or "float32": everything in fp32
    max_seq: int = 4224
    max_batch: int = 1
    pool_tokens: int = 0         # tokens the page pools hold over all sequences; 0 = max_batch * max_seq

    def _count(self, kind, layers=None) -> int:
        return sum(isinstance(layer.mixer, kind) for layer in self.layers[:layers])

    def buffers_desc(self, layers: Optional[int] = None) -> BuffersDesc:
        """Of the first `layers` layers (None: all)."""
        part = self.layers[:layers]
        return BuffersDesc(hidden=self.width, vocab=self.vocab, max_seq=self.max_seq, max_batch=self.max_batch,
                           stream_dtype=STREAM_ALL_F32 if self.dtype == "float32" else STREAM_F32, grouped_layers=self._count(KeyValueAttention, layers),
                           delta_layers=self._count(GatedDelta, layers), kv_pool_tokens=self.pool_tokens,
                           stream_convs=len(part) + sum(layer.mlp is not None for layer in part), depth_results=len(part) + 1)

    def product_elems(self) -> int:
        """Entries of the matrices the dense products of one decode step read (the routed experts not among them)."""
        w = self.width
        total = self.vocab * w
        for layer in self.layers:
            m = layer.mixer
            if isinstance(m, GatedDelta):
                total += w * (2 * m.kv_heads * m.dim + 3 * m.heads * m.vdim + 2 * m.heads)
            else:
                total += w * m.dim * (3 * m.heads + m.kv_heads)
            total += w * (w + 2 * self.side)
            if layer.mlp is not None:
                total += w * (w + layer.mlp.experts + layer.mlp.identity)
        return total


def _up8(v: int) -> int:
    return -(-v // 8) * 8


def _mixer(i: int, entry: Dict) -> Union[KeyValueAttention, GatedDelta]:
    m, kind = entry["mixer"], entry["type"]
    if kind not in ("attention", "delta"):
        raise ValueError(f"layer {i}: mixer type {kind!r}")
    heads, kv, dim, vdim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    if kv < 1 or heads % kv:
        raise ValueError(f"layer {i}: {heads} heads over {kv} key heads")
    if kind == "delta":
        return GatedDelta(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=int(m["conv"]))
    if vdim != dim:
        raise ValueError(f"layer {i}: values of {vdim} entries cannot be keys of {dim}")
    temp = m.get("q_temp") or {"coef": 0.0, "every": 0}
    if temp["every"] != int(temp["every"]) or (temp["every"] < 1 and m.get("q_temp")):
        raise ValueError(f"layer {i}: query temperature every {temp['every']} positions")
    return KeyValueAttention(heads=heads, kv_heads=kv, dim=dim, scale=float(m["scale"]), temp_coef=float(temp["coef"]), temp_every=int(temp["every"]))


def _feed_forward(i: int, mlp: Optional[Dict]) -> Optional[RoutedFF]:
    if mlp is None:
        return None
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
    router = mlp["router"]
    out = RoutedFF(ff=int(mlp["expert"]["ff"]), experts=int(router["experts"]), identity=int(router.get("identity") or 0), top=int(router["top"]))
    if out.experts < 1 or out.identity < 0 or not 1 <= out.top <= out.experts + out.identity:
        raise ValueError(f"layer {i}: {out.top} of {out.experts} + {out.identity} experts")
    return out


def decode_config(config: Dict, shapes: Optional[Mapping[str, Tuple[int, ...]]] = None, dtype: str = "bfloat16", max_seq: int = 4224, max_batch: int = 1,
                  pool_tokens: int = 0) -> MerudraConfig:
    """config.json of a Merudra checkpoint. Every entry is read from the file; a value this recipe cannot express is refused."""
    if config.get("architecture") != ARCHITECTURE:
        raise ValueError(f"architecture {config.get('architecture')!r} is not {ARCHITECTURE}")
    if dtype not in ("bfloat16", "float32"):
        raise ValueError(f"dtype {dtype!r}: bfloat16 or float32")
    taps, side = int(config["canon"]["taps"]), int(config["token_side"]["dim"])
    if taps < 1 or side < 1:
        raise ValueError(f"convolutions of {taps} taps, {side} entries per token and layer")
    layers = [Layer(mixer=_mixer(i, entry), mlp=_feed_forward(i, entry.get("mlp"))) for i, entry in enumerate(config["layers"])]
    return MerudraConfig(vocab=int(config["vocab"]), width=int(config["width"]), taps=taps, side=side, layers=layers, norm_eps=float(config["norm"]["eps"]),
                         dtype=dtype, max_seq=max_seq, max_batch=max_batch, pool_tokens=pool_tokens)


class MerudraPlanBuilder:
    """Tensor inventory and step list of a MerudraConfig (the counterpart of plan.DispatchPlanBuilder)."""

    def __init__(self, config: MerudraConfig):
        self.config = config

    def tensors(self):
        """(name, kind, shape, shard kind): `matrix` = operand of a product, `norm` = norm weight, `dense` = tables and small
        vectors, `taps` = a short convolution's."""
        c, w = self.config, self.config.width
        out = [("embed", "dense", (c.vocab, w)), ("side.embed", "dense", (c.vocab, len(c.layers) * c.side))]
        for i, layer in enumerate(c.layers):
            p, m, mlp = f"l{i}.", layer.mixer, layer.mlp
            x = p + "mix."
            if isinstance(m, KeyValueAttention):
                for t, rows in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim)):
                    out += [(x + t, "matrix", (rows, w)), (x + t + ".b", "dense", (rows,))]
                out += [(x + "g", "matrix", (m.heads * m.dim, w)), (x + "o", "matrix", (w, m.heads * m.dim))]
            else:
                for t, rows in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.heads * m.vdim)):
                    out += [(x + t, "matrix", (rows, w)), (x + t + ".conv", "taps", (rows, m.conv))]
                out += [(x + "b", "matrix", (m.heads, w)), (x + "A_log", "dense", (m.heads,)), (x + "norm", "norm", (m.vdim,)),
                        (x + "a", "matrix", (m.heads, w)), (x + "dt_bias", "dense", (m.heads,)), (x + "g", "matrix", (m.heads * m.vdim, w)),
                        (x + "o", "matrix", (w, m.heads * m.vdim))]
            for j in ("1", "2") if mlp is not None else ("1",):
                out += [(p + "norm" + j, "norm", (w,)), (p + "canon" + j, "taps", (w, c.taps)), (p + "rg" + j, "matrix", (w, w)),
                        (p + "rg" + j + ".b", "dense", (w,))]
            out += [(p + "dwa", "dense", (i + 2,)), (p + "side.gate", "matrix", (c.side, w)), (p + "side.proj", "matrix", (w, c.side)),
                    (p + "side.norm", "norm", (w,))]
            if mlp is not None:
                for e in range(mlp.experts):
                    q = f"{p}mlp.e{e}."
                    out += [(q + "gate", "matrix", (mlp.ff, w)), (q + "up", "matrix", (mlp.ff, w)), (q + "down", "matrix", (w, mlp.ff))]
                out += [(p + "mlp.router", "matrix", (mlp.experts + mlp.identity, w)), (p + "mlp.correction", "dense", (mlp.experts + mlp.identity,))]
        out += [("final.norm", "norm", (w,)), ("head", "matrix", (c.vocab, w))]
        return [t + (SHARD_REPLICATE,) for t in out]

    def decode_steps(self, layers: Optional[int] = None) -> List[Step]:
        """The steps of one token. `layers` stops after that many layers (for tests that look at the stream)."""
        c, w = self.config, self.config.width
        steps = [_step(STEP_EMBED, out_buf=BUF_RESIDUAL, n=w, weight="embed")]
        counts = {KeyValueAttention: 0, GatedDelta: 0, "conv": 0}

        def product(name: str, src: int, dst: int, n: int, k: int, dst_off: int = 0, bias: bool = False):
            steps.append(_step(STEP_PRODUCT, in_buf=src, out_buf=dst, n=n, k=k, out_off=dst_off, weight=name, weight3=name + ".b" if bias else ""))

        def enter(canon: str):
            """What a sublayer reads: the stream with its convolution in S1, the stream itself (for the gate) in S0."""
            steps.append(_step(STEP_STREAM_CONV, layer=counts["conv"], out_buf=BUF_S1, n=w, conv_kernel=c.taps, weight=canon))
            steps.append(_step(STEP_STREAM_COPY, out_buf=BUF_S0, n=w))
            counts["conv"] += 1

        def leave(norm: str, gate: int = -1):
            steps.append(_step(STEP_GATED_POSTNORM_ADD, in_buf=BUF_HIDDEN, in3_buf=gate, n=w, eps=c.norm_eps, weight=norm))

        for i, layer in enumerate(c.layers[:layers]):
            p, m, mlp = f"l{i}.", layer.mixer, layer.mlp
            enter(p + "canon1")
            product(p + "rg1", BUF_S0, BUF_S3, w, w, bias=True)   # (one product with what the mixer projects, of another input)
            if isinstance(m, KeyValueAttention):
                self._attention(steps, product, p, m, counts[KeyValueAttention])
            else:
                self._delta(steps, product, p, m, counts[GatedDelta])
            counts[type(m)] += 1
            leave(p + "norm1", BUF_S3)
            if mlp is not None:
                enter(p + "canon2")
                product(p + "rg2", BUF_S0, BUF_S3, w, w, bias=True)
                product(p + "mlp.router", BUF_S1, BUF_S4, mlp.experts + mlp.identity, w)
                steps.append(_step(STEP_ROUTED_MLP, in_buf=BUF_S1, in2_buf=BUF_S4, out_buf=BUF_HIDDEN, n=w, k=mlp.ff, experts=mlp.experts, identity=mlp.identity,
                                   top=mlp.top, groups=1, groups_keep=1, scale=1.0, score_act=SCORE_SOFTMAX, group_best=1, raw_weights=1,
                                   expert_act=EXPERT_SILU, weight=p + "mlp.e", weight2=".gate", weight3=".up", weight4=".down", weight7=p + "mlp.correction"))
                leave(p + "norm2", BUF_S3)
            steps.append(_step(STEP_STREAM_COPY, out_buf=BUF_S0, n=w))
            product(p + "side.gate", BUF_S0, BUF_S1, c.side, w)
            steps.append(_step(STEP_TOKEN_GATE, in_buf=BUF_S1, out_buf=BUF_S1, n=c.side, in2_off=i * c.side, weight="side.embed"))
            product(p + "side.proj", BUF_S1, BUF_HIDDEN, w, c.side)
            leave(p + "side.norm")
            steps.append(_step(STEP_DEPTH_AVG, n=w, k=i + 2, weight=p + "dwa"))
        steps.append(_step(STEP_COPY_RMSNORM, in_buf=BUF_RESIDUAL, out_buf=BUF_S0, n=w, eps=c.norm_eps, weight="final.norm"))
        product("head", BUF_S0, BUF_LOGITS, c.vocab, w)
        steps.append(_step(STEP_ARGMAX, in_buf=BUF_LOGITS, n=c.vocab))
        return steps

    def _attention(self, steps: List[Step], product, p: str, m: KeyValueAttention, index: int) -> None:
        """q | k | gate side by side."""
        w, x, qa, ka = self.config.width, p + "mix.", m.heads * m.dim, m.kv_heads * m.dim
        gate_at = _up8(qa + ka)
        product(x + "q", BUF_S1, BUF_S2, qa, w, bias=True)
        product(x + "k", BUF_S1, BUF_S2, ka, w, dst_off=qa, bias=True)
        product(x + "g", BUF_S1, BUF_S2, qa, w, dst_off=gate_at)
        steps.append(_step(STEP_GROUPED_ATTN, layer=index, in_buf=BUF_S2, in4_buf=BUF_S2, in4_off=gate_at, out_buf=BUF_S0, heads=m.heads, kv_heads=m.kv_heads,
                           head_dim=m.dim, value_dim=m.dim, value_is_key=1, head_norm=1, scale=m.scale, eps=self.config.norm_eps, temp_coef=m.temp_coef,
                           temp_every=m.temp_every, out_scale=1.0, rope_base=1.0))
        product(x + "o", BUF_S0, BUF_HIDDEN, w, qa)

    def _delta(self, steps: List[Step], product, p: str, m: GatedDelta, index: int) -> None:
        """q | k | v | gate side by side, step sizes and decay inputs in another buffer."""
        w, x, gk, hv = self.config.width, p + "mix.", m.kv_heads * m.dim, m.heads * m.vdim
        gate_at, decay_at = _up8(2 * gk + hv), _up8(m.heads)
        product(x + "q", BUF_S1, BUF_S2, gk, w)
        product(x + "k", BUF_S1, BUF_S2, gk, w, dst_off=gk)
        product(x + "v", BUF_S1, BUF_S2, hv, w, dst_off=2 * gk)
        product(x + "g", BUF_S1, BUF_S2, hv, w, dst_off=gate_at)
        product(x + "b", BUF_S1, BUF_S4, m.heads, w)
        product(x + "a", BUF_S1, BUF_S4, m.heads, w, dst_off=decay_at)
        steps.append(_step(STEP_GATED_DELTA, layer=index, in_buf=BUF_S2, in2_buf=BUF_S4, in3_buf=BUF_S4, in3_off=decay_at, in4_buf=BUF_S2, in4_off=gate_at,
                           out_buf=BUF_S0, k=1, heads=m.heads, groups=m.kv_heads, key_dim=m.dim, value_dim=m.vdim, conv_kernel=m.conv, eps=self.config.norm_eps,
                           eps2=UNIT_EPS, scale=m.dim ** -0.5, gate_act=GATE_SILU, weight=x + "q.conv", weight2=x + "k.conv", weight3=x + "v.conv",
                           weight4=x + "norm", weight5=x + "A_log", weight6=x + "dt_bias"))
        product(x + "o", BUF_S0, BUF_HIDDEN, w, hv)

    def with_runtime(self, **changes) -> "MerudraPlanBuilder":
        """The same model with other runtime sizes (max_seq, max_batch, pool_tokens, dtype)."""
        return MerudraPlanBuilder(dataclasses.replace(self.config, **changes))
