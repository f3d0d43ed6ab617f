"""Decoders whose layers are listed one by one in a configuration and built on the block library: an fp32
residual stream, one cache or state per layer RUN, weights by checkpoint name.

A model class supplies `embed`, `head`, `runs` (each with the number of the layer whose weights it uses), the
layers themselves, and `_stack`, which takes token ids through them.  Prompt portions and decode steps run the
same stack; a decode step reads its position on the device and is captured in a CUDA graph.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional

import torch
from torch import Tensor

from .decoder import Decoder
from .mixers import Portion, matmul_f32


@dataclass(frozen=True)
class LayerSpec:
    """One entry of the layer list: the mixer's kind and sizes, and the feed-forward (or none)."""
    kind: str
    mixer: Mapping[str, Any]
    mlp: Optional[Mapping[str, Any]]


class LayeredDecoder(Decoder):
    libraries = ("blocks",)
    runs: List[Any]                            # entries with a field `layer`

    def __init__(self):
        super().__init__()
        self.caches: List[Any] = []
        self._status = self._workspace = None

    # ------------------------------------------------------------------------------- hooks
    def layer_of(self, run):
        """The layer module a run uses; its `mixer` makes caches and has derived buffers."""
        return self.layers[run.layer]

    def tensors(self) -> Dict[str, Tensor]:
        """Checkpoint name -> the parameter (or the slice of a fused parameter) that holds it."""
        raise NotImplementedError

    def _stack(self, idx: Tensor, at: Portion, collect: Optional[list] = None) -> Tensor:
        """Final norm of the residual stream [B*S, width]; `collect` takes a copy of the stream after every run."""
        raise NotImplementedError

    def _draw(self, leaf: str, shape_of: Tensor, std: float, g: torch.Generator) -> Tensor:
        """Random values of the parameter whose name ends in `leaf`."""
        draw = torch.empty(shape_of.shape, dtype=torch.float32, device=shape_of.device)
        if "norm" in leaf:
            return draw.fill_(1.0)
        return draw.normal_(0.0, std if shape_of.dim() > 1 else 0.1, generator=g)

    # ------------------------------------------------------------------------------- weights
    @property
    def embedding_table(self) -> Tensor:
        return self.embed

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
        for run in self.runs:
            self.layer_of(run).mixer.finish_loading()

    @torch.no_grad()
    def init_random(self, seed: int = 0, std: float = 0.02) -> "LayeredDecoder":
        """Random weights drawn on the parameters' device: norms one, a recurrence's constants in their usual
        ranges, everything else normal."""
        g = torch.Generator(device=self.device).manual_seed(seed)
        for name, p in self.tensors().items():
            p.copy_(self._draw(name.rsplit(".", 1)[-1], p, std, g))
        self.finish_loading()
        return self

    # ------------------------------------------------------------------------------- caches
    def _alloc_caches(self, batch: int, length: int) -> None:
        """One cache or state per layer run: runs that share weights do not share caches."""
        dev, dt = self.device, self.dtype
        self.caches = [self.layer_of(r).mixer.make_cache(batch, length, dt, dev) for r in self.runs]
        self._status = torch.zeros(1, dtype=torch.int32, device=dev)
        need = max([self.layer_of(r).mixer.workspace_bytes(c, batch) for r, c in zip(self.runs, self.caches)], default=0)
        self._workspace = torch.zeros(need, dtype=torch.uint8, device=dev) if need else None

    def device_flags(self) -> int:
        """Flags the kernels have raised so far (0: none).  Synchronises."""
        return int(self._status.item())

    # ------------------------------------------------------------------------------- the decoder's hooks
    def _portion(self, idx: Tensor, start: int, collect: Optional[list] = None) -> Tensor:
        B, S = idx.shape
        at = Portion(B, S, start, status=self._status, workspace=self._workspace)
        return self._stack(idx, at, collect).view(B, S, -1)

    def _head(self, hidden: Tensor) -> Tensor:
        logits = matmul_f32(hidden.reshape(-1, hidden.shape[-1]), self.head)
        return logits.view(*hidden.shape[:-1], -1)

    def _decode_logits(self, mode: str) -> Tensor:
        B = self._tok.shape[0]
        at = Portion(B, 1, 0, pos=self._pos, status=self._status, workspace=self._workspace)
        return self._head(self._stack(self._tok, at))
