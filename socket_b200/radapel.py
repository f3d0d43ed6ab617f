"""Radapel: a decoder whose layers are listed one by one - chunk-masked attention with a distance bias,
latent attention, or a state-space mixer, each with or without a clamped gated feed-forward - with a
norm before and after every sublayer, and a range of layers that is run several times with the same
weights and a cache of its own per pass.

The residual stream is fp32; one kernel per sublayer adds the sublayer's normed output and norms the
next sublayer's input (`block_ops.residual_norm`).  Prompt portions and decode steps run the same
stack (`_stack`); a decode step reads its position on the device and is captured in a CUDA graph.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Mapping, Optional, Tuple

import torch
import torch.nn as nn
from torch import Tensor

from . import block_ops as ops
from .layered import LayeredDecoder, LayerSpec
from .mixers import (ChunkedAttention, ClampedFeedForward, LatentAttention, Mamba2, Portion, matmul_f32, projection, vector)

MIXERS = ("attention", "latent_attention", "mamba2")


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class RadapelConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: Tuple[LayerSpec, ...]
    loop: Optional[Loop] = None
    # rows of each layer's distance-bias table, which only the checkpoint's tensor shapes give
    bias_rows: Mapping[int, int] = field(default_factory=dict)

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], shapes: Optional[Mapping[str, Tuple[int, ...]]] = None,
                  bias_rows: int = 32) -> "RadapelConfig":
        """`d`: a parsed config.json; `shapes`: the checkpoint's tensor shapes.  Without them (random
        weights) every distance-bias table has `bias_rows` rows."""
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            mlp = e.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerSpec(e["type"], dict(e["mixer"]), None if mlp is None else dict(mlp)))
        lp = d.get("loop")
        loop = None
        if lp is not None:
            loop = Loop(lp["start"], lp["stop"], lp["times"])
            if not (0 <= loop.start < loop.stop <= len(layers) and loop.times >= 1):
                raise ValueError(f"loop {lp} does not fit {len(layers)} layers")
        rows = {i: (shapes[f"l{i}.mix.rel"][0] if shapes is not None else bias_rows)
                for i, e in enumerate(layers) if e.kind == "attention"}
        return cls(d["vocab"], d["width"], d["norm"]["eps"], d["embedding"]["scale"], tuple(layers), loop, rows)


@dataclass(frozen=True)
class LayerRun:
    """One run of a layer: the layer, and at the head of a loop's pass the number of that pass."""
    layer: int
    new_pass: Optional[int]


def layer_runs(config: RadapelConfig) -> List[LayerRun]:
    n, lp = len(config.layers), config.loop
    if lp is None:
        return [LayerRun(i, None) for i in range(n)]
    runs = [LayerRun(i, None) for i in range(lp.start)]
    for t in range(lp.times):
        runs += [LayerRun(i, t if i == lp.start else None) for i in range(lp.start, lp.stop)]
    return runs + [LayerRun(i, None) for i in range(lp.stop, n)]


def build_mixer(config: RadapelConfig, i: int) -> nn.Module:
    e, m, w = config.layers[i], config.layers[i].mixer, config.width
    if e.kind == "attention":
        return ChunkedAttention(w, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"], m["scale"],
                                config.bias_rows[i], m["bias_max"])
    if e.kind == "latent_attention":
        return LatentAttention(w, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["rot"]["dims"],
                               m["rot"]["base"], m["scale"], config.eps)
    return Mamba2(w, m["heads"], m["vdim"], m["state"], m["groups"], m["conv"], m["norm_groups"], config.eps)


class RadapelLayer(nn.Module):
    def __init__(self, config: RadapelConfig, i: int):
        super().__init__()
        mlp = config.layers[i].mlp
        self.mixer = build_mixer(config, i)
        self.mlp = None if mlp is None else ClampedFeedForward(config.width, mlp["ff"], mlp["limit"])
        self.norm1, self.norm1b = vector(config.width), vector(config.width)
        if mlp is not None:
            self.norm2, self.norm2b = vector(config.width), vector(config.width)

    def tensors(self) -> Dict[str, Tensor]:
        out = {"norm1": self.norm1, "norm1b": self.norm1b}
        out.update({"mix." + k: v for k, v in self.mixer.tensors().items()})
        if self.mlp is not None:
            out.update({"norm2": self.norm2, "norm2b": self.norm2b})
            out.update({"mlp." + k: v for k, v in self.mlp.tensors().items()})
        return out


class Radapel(LayeredDecoder):
    def __init__(self, config: RadapelConfig):
        super().__init__()
        self.config = config
        self.embed = projection(config.vocab, config.width)
        self.layers = nn.ModuleList(RadapelLayer(config, i) for i in range(len(config.layers)))
        self.final_norm = vector(config.width)
        self.head = projection(config.vocab, config.width)
        if config.loop is not None:
            self.loop_in = projection(config.width, 2 * config.width)
            self.loop_step = projection(config.loop.times, config.width)
        self.runs = layer_runs(config)

    # ------------------------------------------------------------------------------- weights
    def tensors(self) -> Dict[str, Tensor]:
        out = {"embed": self.embed, "final.norm": self.final_norm, "head": self.head}
        if self.config.loop is not None:
            out.update({"loop.in": self.loop_in, "loop.step": self.loop_step})
        for i, layer in enumerate(self.layers):
            out.update({f"l{i}.{k}": v for k, v in layer.tensors().items()})
        return out

    def _draw(self, leaf: str, shape_of: Tensor, std: float, g: torch.Generator) -> Tensor:
        draw = torch.empty(shape_of.shape, dtype=torch.float32, device=shape_of.device)
        if leaf == "D":
            return draw.fill_(1.0)
        if leaf == "A_log":
            return torch.log(draw.uniform_(1.0, 16.0, generator=g))
        if leaf == "dt_bias":
            return torch.log(torch.expm1(torch.exp(draw.uniform_(-6.9, -2.3, generator=g))))
        return super()._draw(leaf, shape_of, std, g)

    # ------------------------------------------------------------------------------- the stack
    def _stack(self, idx: Tensor, at: Portion, collect: Optional[list] = None) -> Tensor:
        cfg, eps, dt = self.config, self.config.eps, self.dtype
        x, x0 = ops.embed_rows(idx, self.embed, cfg.embedding_scale, keep_copy=cfg.loop is not None, status=at.status)
        y = w = None                                # a sublayer's output and the norm it still has to pass
        for run, cache in zip(self.runs, self.caches):
            layer = self.layers[run.layer]
            if run.new_pass is not None:
                joined = ops.residual_norm(x, eps, y=y, w_in=w, x0=x0, dtype=dt)
                y = matmul_f32(joined, self.loop_in)
                h = ops.residual_norm(x, eps, y=y, w_in=self.loop_step[run.new_pass], replace=True, w_out=layer.norm1)
            else:
                h = ops.residual_norm(x, eps, y=y, w_in=w, w_out=layer.norm1)
            y, w = layer.mixer(h, cache, at), layer.norm1b
            if layer.mlp is not None:
                h = ops.residual_norm(x, eps, y=y, w_in=w, w_out=layer.norm2)
                y, w = layer.mlp(h), layer.norm2b
            if collect is not None:
                ops.residual_norm(x, eps, y=y, w_in=w)
                collect.append(x.clone())
                y = w = None
        return ops.residual_norm(x, eps, y=y, w_in=w, w_out=self.final_norm)
