"""Timalorn: a decoder whose layers are listed one by one - sliding-window attention whose values are its
unrotated keys, or a matrix memory (mLSTM) - with one layer norm per layer whose output both the mixer and
the feed-forward read (`mixers.ParallelLayer`).  A layer may use another layer's tensors; its cache or state
is its own all the same.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple

import torch
import torch.nn as nn
from torch import Tensor

from . import block_ops as ops
from .layered import LayeredDecoder, LayerSpec
from .mixers import MatrixMemory, ParallelLayer, Portion, WindowAttention, YarnScaling, projection, vector

MIXERS = ("attention", "mlstm")


@dataclass(frozen=True)
class TimalornConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: Tuple[LayerSpec, ...]
    owners: Tuple[int, ...]                        # per layer: the layer whose tensors it uses

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "TimalornConfig":
        """`d`: a parsed config.json."""
        entries = d["layers"]
        layers, owners = [], []
        for i, e in enumerate(entries):
            if e["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            m, mlp = dict(e["mixer"]), e.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            if e["type"] == "attention" and m.get("vdim", m["dim"]) != m["dim"]:
                raise ValueError(f"layer {i}: values of size {m['vdim']} cannot be keys of size {m['dim']}")
            layers.append(LayerSpec(e["type"], m, None if mlp is None else dict(mlp)))
            j, seen = i, []
            while entries[j].get("weights_of") is not None:
                seen.append(j)
                j = entries[j]["weights_of"]
                if not 0 <= j < len(entries) or j in seen:
                    raise ValueError(f"layer {i}: weights_of leads to no layer with tensors")
            owners.append(j)
        for i, j in enumerate(owners):
            if layers[i] != layers[j]:
                raise ValueError(f"layer {i} uses the tensors of layer {j}, but their entries differ")
        return cls(d["vocab"], d["width"], d["norm"]["eps"], d["embedding"]["scale"], tuple(layers), tuple(owners))


@dataclass(frozen=True)
class LayerRun:
    layer: int                                     # the layer whose weights it uses


def build_mixer(config: TimalornConfig, i: int) -> nn.Module:
    e, m = config.layers[i], config.layers[i].mixer
    if e.kind == "attention":
        rot = m["rot"]
        s = rot.get("scaling")
        scaling = None if s is None else YarnScaling(s["factor"], s["original"], s["fast"], s["slow"])
        return WindowAttention(m["heads"], m["kv_heads"], m["dim"], m["mask"]["size"], m["scale"], rot["dims"], rot["base"],
                               scaling, m["softcap"])
    return MatrixMemory(config.width, m["heads"], m["dim"], m["vdim"], m["gate_cap"], config.eps)


class Timalorn(LayeredDecoder):
    def __init__(self, config: TimalornConfig):
        super().__init__()
        self.config = config
        self.embed = projection(config.vocab, config.width)
        self.layers = nn.ModuleDict({
            str(i): ParallelLayer(config.width, build_mixer(config, i),
                                  config.layers[i].mlp["ff"] if config.layers[i].mlp is not None else 0)
            for i in sorted(set(config.owners))})
        self.final_norm = vector(config.width)
        self.head = projection(config.vocab, config.width)
        self.runs: List[LayerRun] = [LayerRun(j) for j in config.owners]

    def layer_of(self, run: LayerRun) -> ParallelLayer:
        return self.layers[str(run.layer)]

    def tensors(self) -> Dict[str, Tensor]:
        out = {"embed": self.embed, "final.norm": self.final_norm, "head": self.head}
        for i, layer in self.layers.items():
            out.update({f"l{i}.{k}": v for k, v in layer.tensors().items()})
        return out

    def _draw(self, leaf: str, shape_of: Tensor, std: float, g: torch.Generator) -> Tensor:
        draw = super()._draw(leaf, shape_of, std, g)
        # the one-dimensional "b" of the gates: forget gates mostly open is what a trained memory has
        return draw.add_(3.0) if leaf == "b" else draw

    def _stack(self, idx: Tensor, at: Portion, collect: Optional[list] = None) -> Tensor:
        eps = self.config.eps
        x, _ = ops.embed_rows(idx, self.embed, self.config.embedding_scale, status=at.status)
        y = None                                   # what the layer before adds to the stream
        for run, cache in zip(self.runs, self.caches):
            layer = self.layer_of(run)
            h = ops.residual_norm(x, eps, y=y, w_out=layer.norm1, centred=True)
            y = layer(h, cache, at)
            if collect is not None:
                ops.residual_norm(x, eps, y=y)
                collect.append(x.clone())
                y = None
        return ops.residual_norm(x, eps, y=y, w_out=self.final_norm, centred=True)
