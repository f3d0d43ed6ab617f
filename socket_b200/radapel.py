"""Radapel: a decoder whose layers are listed one by one - chunk-masked attention with a distance bias,
latent attention, or a state-space mixer, each with or without a clamped gated feed-forward - with a
norm before and after every sublayer, and a range of layers that is run several times with the same
weights and a cache of its own per pass.

The residual stream is fp32; one kernel per sublayer adds the sublayer's normed output and norms the
next sublayer's input (`block_ops.residual_norm`).  Prompt portions and decode steps run the same
stack (`_stack`); a decode step reads its position on the device and is captured in a CUDA graph.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass, field
from typing import Any, Dict, List, Mapping, Optional, Tuple

import torch
import torch.nn as nn
from torch import Tensor

from . import block_ops as ops
from ._lib import blocks
from .decoder import Decoder
from .mixers import (ChunkedAttention, ClampedFeedForward, LatentAttention, Mamba2, Portion, projection, vector)

MIXERS = ("attention", "latent_attention", "mamba2")


@dataclass(frozen=True)
class LayerSpec:
    """One entry of the layer list: the mixer's kind and sizes, and the feed-forward (or none)."""
    kind: str
    mixer: Mapping[str, Any]
    mlp: Optional[Mapping[str, Any]]


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


class Radapel(Decoder):
    libraries = ("blocks",)

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
        self.caches: List[Any] = []
        self._status = self._workspace = None

    # ------------------------------------------------------------------------------- weights
    @property
    def embedding_table(self) -> Tensor:
        return self.embed

    def tensors(self) -> Dict[str, Tensor]:
        """Checkpoint name -> the parameter (or the rows of a fused parameter) that holds it."""
        out = {"embed": self.embed, "final.norm": self.final_norm, "head": self.head}
        if self.config.loop is not None:
            out.update({"loop.in": self.loop_in, "loop.step": self.loop_step})
        for i, layer in enumerate(self.layers):
            out.update({f"l{i}.{k}": v for k, v in layer.tensors().items()})
        return out

    @torch.no_grad()
    def load_tensors(self, tensors: Mapping[str, Tensor]) -> None:
        own = self.tensors()
        if set(own) != set(tensors):
            raise ValueError(f"checkpoint does not fit the model: {sorted(set(own) ^ set(tensors))[:8]}")
        for name, dst in own.items():
            if dst.shape != tensors[name].shape:
                raise ValueError(f"{name}: {tuple(tensors[name].shape)} in the checkpoint, {tuple(dst.shape)} in the model")
            dst.copy_(tensors[name])
        self.finish_loading()

    @torch.no_grad()
    def finish_loading(self) -> None:
        """Derived buffers of the mixers (bias per distance, expansion of latent rows, fp32 constants)."""
        for layer in self.layers:
            layer.mixer.finish_loading()

    @torch.no_grad()
    def init_random(self, seed: int = 0, std: float = 0.02) -> "Radapel":
        """Random weights drawn in the parameters' dtype on their device: norms one, the recurrence's
        constants in their usual ranges, everything else normal."""
        g = torch.Generator(device=self.device).manual_seed(seed)
        for name, p in self.tensors().items():
            leaf = name.rsplit(".", 1)[-1]
            draw = torch.empty(p.shape, dtype=torch.float32, device=p.device)
            if leaf.startswith("norm") or leaf == "D":
                p.fill_(1.0)
            elif leaf == "A_log":
                p.copy_(torch.log(draw.uniform_(1.0, 16.0, generator=g)))
            elif leaf == "dt_bias":
                p.copy_(torch.log(torch.expm1(torch.exp(draw.uniform_(-6.9, -2.3, generator=g)))))
            else:
                p.copy_(draw.normal_(0.0, std if p.dim() > 1 else 0.1, generator=g))
        self.finish_loading()
        return self

    # ------------------------------------------------------------------------------- caches
    def _alloc_caches(self, batch: int, length: int) -> None:
        """One cache or state per layer run: the passes of a loop share weights, not caches."""
        dev, dt = self.device, self.dtype
        self.caches = [self.layers[r.layer].mixer.make_cache(batch, length, dt, dev) for r in self.runs]
        self._status = torch.zeros(1, dtype=torch.int32, device=dev)
        need = 0
        for r, cache in zip(self.runs, self.caches):
            shapes = getattr(self.layers[r.layer].mixer, "decode_shapes", None)
            if shapes is not None:
                q_shape, k, v = shapes(cache, batch)
                for s in {1, q_shape[1]}:
                    q = torch.empty(q_shape[0], s, *q_shape[2:], dtype=dt, device="meta")
                    o = torch.empty(q_shape[0], s, q_shape[2], v.shape[3], dtype=dt, device="meta")
                    ring = isinstance(self.layers[r.layer].mixer, ChunkedAttention)
                    p = ops.attn_params(q, k, v, o, scale=1.0, ring=ring, chunk=k.shape[1] if ring else 0, meta=True)
                    need = max(need, int(blocks().skb_attn_workspace_bytes(ctypes.byref(p))))
        self._workspace = torch.zeros(need, dtype=torch.uint8, device=dev) if need else None

    def device_flags(self) -> int:
        """Flags the kernels have raised so far (0: none).  Synchronises."""
        return int(self._status.item())

    # ------------------------------------------------------------------------------- the stack
    def _stack(self, idx: Tensor, at: Portion, collect: Optional[list] = None) -> Tensor:
        """Residual stream [B*S, width] (fp32) and its final norm; returns the latter.  `collect` takes a
        copy of the stream after every layer run."""
        cfg, eps, dt = self.config, self.config.eps, self.dtype
        x, x0 = ops.embed_rows(idx, self.embed, cfg.embedding_scale, keep_copy=cfg.loop is not None, status=at.status)
        y = w = None                                # a sublayer's output and the norm it still has to pass
        for run, cache in zip(self.runs, self.caches):
            layer = self.layers[run.layer]
            if run.new_pass is not None:
                joined = ops.residual_norm(x, eps, y=y, w_in=w, x0=x0, dtype=dt)
                y = torch.mm(joined, self.loop_in.t(), out_dtype=torch.float32) if dt != torch.float32 else \
                    torch.mm(joined, self.loop_in.t())
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

    def _portion(self, idx: Tensor, start: int, collect: Optional[list] = None) -> Tensor:
        B, S = idx.shape
        at = Portion(B, S, start, status=self._status, workspace=self._workspace)
        return self._stack(idx, at, collect).view(B, S, -1)

    def _head(self, hidden: Tensor) -> Tensor:
        rows = hidden.reshape(-1, hidden.shape[-1])
        if rows.dtype == torch.float32:
            logits = torch.mm(rows, self.head.t())
        else:
            logits = torch.mm(rows, self.head.t(), out_dtype=torch.float32)
        return logits.view(*hidden.shape[:-1], -1)

    def _decode_logits(self, mode: str) -> Tensor:
        B = self._tok.shape[0]
        at = Portion(B, 1, 0, pos=self._pos, status=self._status, workspace=self._workspace)
        return self._head(self._stack(self._tok, at))
