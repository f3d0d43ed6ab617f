"""Token mixers and feed-forwards built on the block library (`block_ops.py`): chunk-masked attention
with a learned distance bias, attention on a low-rank latent, sliding-window attention whose values are
its unrotated keys, a selective state-space layer, a matrix memory, and gated units.  Every size and
constant is a parameter, so that any decoder can list them.

A mixer maps hidden rows [B*S, width] of a portion to rows of the same shape and advances its cache:
`make_cache(...)` builds it, `forward(h, cache, at)` uses it.  `at` (`Portion`) says where the portion
sits; a decode step is the portion of one token whose position is read on the device.

The mixers of a `ParallelLayer` leave their large projections to the layer, which runs them together with
the feed-forward's as one matrix product in and one out: they name them (`in_sizes`, `out_size`) and
`mix(parts, h, cache, at, out)` takes the projected rows to the rows in front of the output projection.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn
from torch import Tensor

from . import block_ops as ops


@dataclass
class Portion:
    """S consecutive tokens of each of B sequences, the first at position `start` (host) or, with `pos`
    (device int64 [1]), wherever that says."""
    B: int
    S: int
    start: int
    pos: Optional[Tensor] = None
    status: Optional[Tensor] = None       # device int32, collects flags of the kernels
    workspace: Optional[Tensor] = None    # scratch of the split decode kernel, shared by all layers

    @property
    def end(self) -> int:
        return self.start + self.S


def padded_rows(weight_rows: int) -> int:
    """Rows of a fused projection: a multiple of 8, so that rows of its output stay 16-byte aligned."""
    return (weight_rows + 7) // 8 * 8


def projection(rows: int, cols: int) -> nn.Parameter:
    return nn.Parameter(torch.zeros(rows, cols), requires_grad=False)


def vector(n: int) -> nn.Parameter:
    return nn.Parameter(torch.zeros(n), requires_grad=False)


def matmul_f32(x: Tensor, w: Tensor) -> Tensor:
    """x w^T whose fp32 sums are not rounded."""
    if x.dtype == torch.float32:
        return torch.mm(x, w.t())
    return torch.mm(x, w.t(), out_dtype=torch.float32)


# ---------------------------------------------------------------------------------- attention
def distance_buckets(n_max: int, rows: int, far: float) -> Tensor:
    """Row of the bias table for the distances 0..n_max: the first half of the rows are one distance
    each, the others grow logarithmically and end at `far`; everything beyond takes the last row."""
    half = rows // 2
    out = []
    for n in range(n_max + 1):
        if n < half:
            out.append(n)
        elif n >= far:
            out.append(rows - 1)
        else:
            # the small term keeps a distance that lies exactly on a bucket's edge on its upper side
            out.append(min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-9)))
    return torch.tensor(out, dtype=torch.long)


class RingCache:
    """Keys and values of the current chunk: position p lives in row p % ring."""

    def __init__(self, batch: int, ring: int, kv_heads: int, dim: int, vdim: int, dtype, device):
        self.k = torch.zeros(batch, ring, kv_heads, dim, dtype=dtype, device=device)
        self.v = torch.zeros(batch, ring, kv_heads, vdim, dtype=dtype, device=device)


class ChunkedAttention(nn.Module):
    """Grouped-query attention without rotation: a token sees the tokens of its own chunk (counted from
    position 0), scores get a learned bias per head and distance bucket.  Only one chunk of keys and
    values is kept."""

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, chunk: int, scale: float,
                 bias_rows: int, bias_max: float):
        super().__init__()
        self.H, self.G, self.D, self.E = heads, kv_heads, dim, vdim
        self.chunk, self.scale, self.bias_max = chunk, scale, bias_max
        self.sizes = [heads * dim, kv_heads * dim, kv_heads * vdim]
        self.wqkv = projection(padded_rows(sum(self.sizes)), width)
        self.wo = projection(width, heads * vdim)
        self.rel = nn.Parameter(torch.zeros(bias_rows, heads), requires_grad=False)
        self.register_buffer("bias", torch.zeros(heads, max(math.ceil(bias_max), bias_rows) + 1), persistent=False)

    def tensors(self) -> dict:
        q, k, v = self.wqkv[:sum(self.sizes)].split(self.sizes)
        return {"q": q, "k": k, "v": v, "rel": self.rel, "o": self.wo}

    def finish_loading(self) -> None:
        """The bias per distance, fp32, from the table per bucket."""
        buckets = distance_buckets(self.bias.shape[1] - 1, self.rel.shape[0], self.bias_max).to(self.rel.device)
        self.bias = self.rel.float()[buckets].t().contiguous()

    def make_cache(self, batch: int, length: int, dtype, device) -> RingCache:
        return RingCache(batch, min(self.chunk, length), self.G, self.D, self.E, dtype, device)

    def workspace_bytes(self, cache: RingCache, batch: int) -> int:
        return ops.attn_workspace((batch, 1, self.H, self.D), cache.k, cache.v, scale=1.0, ring=True, chunk=cache.k.shape[1])

    def forward(self, h: Tensor, cache: RingCache, at: Portion) -> Tensor:
        B, S = at.B, at.S
        qkv = torch.mm(h, self.wqkv.t()).view(B, S, -1)
        a, b, c = self.sizes
        q = qkv[..., :a].unflatten(-1, (self.H, self.D))
        k = qkv[..., a:a + b].unflatten(-1, (self.G, self.D))
        v = qkv[..., a + b:a + b + c].unflatten(-1, (self.G, self.E))
        args = dict(scale=self.scale, chunk=self.chunk, bias=self.bias, status=at.status)
        if at.pos is not None:
            ops.ring_append(k, v, cache.k, cache.v, pos=at.pos)
            y = ops.attn(q, cache.k, cache.v, pos=at.pos, ring=True, workspace=at.workspace, **args)
        else:
            lo = at.start // self.chunk * self.chunk
            if lo < at.start:                      # the portion starts inside a chunk: its kept keys come first
                n = at.start - lo
                ka, va = torch.cat([cache.k[:B, :n], k], 1), torch.cat([cache.v[:B, :n], v], 1)
            else:
                ka, va = k, v
            y = ops.attn(q, ka, va, start=at.start, kv_start=lo, **args)
            ops.ring_append(k, v, cache.k[:B], cache.v[:B], start=at.start)
        return torch.mm(y.view(B * S, self.H * self.E), self.wo.t())


# ---------------------------------------------------------------------------------- latent attention
@dataclass(frozen=True)
class YarnScaling:
    """Stretched rotary positions: pairs that turn more than `fast` times within `original` tokens keep their
    frequency, pairs that turn less than `slow` times turn `factor` times slower, pairs between are blended; the
    rotation is scaled by 0.1 ln(factor) + 1."""
    factor: float
    original: float
    fast: float
    slow: float


def rotary_frequencies(dims: int, base: float, scaling: Optional[YarnScaling] = None) -> Tensor:
    """Angle per position of each of the dims / 2 pairs (float64)."""
    f = base ** (-torch.arange(0, dims, 2, dtype=torch.float64) / dims)
    if scaling is None:
        return f

    def pair(turns: float) -> float:               # the pair that turns so often within the original length
        return dims * math.log(scaling.original / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(pair(scaling.fast)), 0), min(math.ceil(pair(scaling.slow)), dims - 1)
    ramp = ((torch.arange(dims // 2, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return f / scaling.factor * ramp + f * (1 - ramp)


def rotary_angles(length: int, dims: int, base: float, device, scaling: Optional[YarnScaling] = None) -> Tensor:
    """[length, dims / 2, 2] = (cos, sin) of position * frequency, times the scaling's gain, fp32 (computed in double)."""
    a = torch.outer(torch.arange(length, dtype=torch.float64), rotary_frequencies(dims, base, scaling))
    gain = 1.0 if scaling is None else 0.1 * math.log(scaling.factor) + 1.0
    return (torch.stack([torch.cos(a), torch.sin(a)], -1) * gain).float().contiguous().to(device)


class LatentCache:
    """One row [latent | rotated key part] per token, shared by all heads."""

    def __init__(self, batch: int, length: int, row: int, angles: Tensor, dtype, device):
        self.rows = torch.zeros(batch, length, row, dtype=dtype, device=device)
        self.angles = angles


class LatentAttention(nn.Module):
    """Causal attention whose keys and values are low-rank: per head key = [W_uk c | rotated part],
    value = W_uv c, with a learned sink per head.  Short portions attend on the latent rows themselves
    (W_uk moved to the query side, W_uv behind the sum); long ones expand keys and values once."""

    expand_from = 33                               # portions of at least this many tokens are expanded

    def __init__(self, width: int, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, rot_dims: int,
                 rot_base: float, scale: float, eps: float):
        super().__init__()
        self.H, self.D, self.R, self.E, self.K = heads, dim, rot_dim, vdim, kv_rank
        self.rot_dims, self.rot_base, self.scale, self.eps = rot_dims, rot_base, scale, eps
        self.q_rows, self.row = heads * (dim + rot_dim), padded_rows(kv_rank + rot_dim)
        self.wqd = projection(padded_rows(self.q_rows + kv_rank + rot_dim), width)
        self.latent_norm = vector(kv_rank)
        self.uk = projection(heads * dim, kv_rank)
        self.uv = projection(heads * vdim, kv_rank)
        self.wo = projection(width, heads * vdim)
        self.sink = vector(heads)
        # rows of a cache row's expansion: H x [W_uk | 0; 0 | I] for the keys, then H x [W_uv | 0]
        self.register_buffer("expand", torch.zeros(self.q_rows + heads * vdim, self.row), persistent=False)
        self.register_buffer("sink_f32", torch.zeros(heads), persistent=False)

    def tensors(self) -> dict:
        n = self.q_rows + self.K + self.R
        return {"q": self.wqd[:self.q_rows], "dkv": self.wqd[self.q_rows:n], "dkv.norm": self.latent_norm,
                "uk": self.uk, "uv": self.uv, "sink": self.sink, "o": self.wo}

    def finish_loading(self) -> None:
        e = torch.zeros(self.q_rows + self.H * self.E, self.row, dtype=self.uk.dtype, device=self.uk.device)
        keys = e[:self.q_rows].view(self.H, self.D + self.R, self.row)
        keys[:, :self.D, :self.K] = self.uk.view(self.H, self.D, self.K)
        keys[:, self.D:, self.K:self.K + self.R] = torch.eye(self.R, dtype=e.dtype, device=e.device)
        e[self.q_rows:, :self.K] = self.uv
        self.expand, self.sink_f32 = e, self.sink.float()

    def make_cache(self, batch: int, length: int, dtype, device) -> LatentCache:
        return LatentCache(batch, length, self.row, rotary_angles(length, self.rot_dims, self.rot_base, device), dtype,
                           device)

    def workspace_bytes(self, cache: LatentCache, batch: int) -> int:
        rows = cache.rows.unsqueeze(2)
        return max(ops.attn_workspace((batch, s, self.H, self.row), rows, rows[..., :self.K], scale=1.0)
                   for s in (1, self.expand_from - 1))

    def forward(self, h: Tensor, cache: LatentCache, at: Portion) -> Tensor:
        B, S = at.B, at.S
        qd = torch.mm(h, self.wqd.t())
        q = qd[:, :self.q_rows]
        dkv = qd[:, self.q_rows:self.q_rows + self.K + self.R]
        rows = cache.rows[:B]
        ops.latent_append(dkv, q, self.latent_norm, cache.angles, rows, S=S, n_heads=self.H, dim=self.D, rot=self.R,
                          rank=self.K, eps=self.eps, start=at.start, pos=at.pos, status=at.status)
        args = dict(scale=self.scale, sink=self.sink_f32, start=at.start, status=at.status)
        if at.pos is not None or S < self.expand_from:
            ql = ops.latent_absorb(q, self.uk, self.H, self.D, self.R, self.row).view(B, S, self.H, self.row)
            shared = rows.unsqueeze(2)
            o = ops.attn(ql, shared, shared[..., :self.K], pos=at.pos, workspace=at.workspace, **args)
            y = ops.latent_up(o.view(B * S, self.H, self.K), self.uv, self.E)
        else:
            kv = torch.matmul(rows[:, :at.end], self.expand.t())
            k = kv[..., :self.q_rows].unflatten(-1, (self.H, self.D + self.R))
            v = kv[..., self.q_rows:].unflatten(-1, (self.H, self.E))
            y = ops.attn(q.view(B, S, -1).unflatten(-1, (self.H, self.D + self.R)), k, v, **args)
        return torch.mm(y.view(B * S, self.H * self.E), self.wo.t())


# ---------------------------------------------------------------------------------- window attention
class RingRows:
    """The last rows [key as projected | its turned elements] of a sequence: position p lives in row p % ring."""

    def __init__(self, batch: int, ring: int, kv_heads: int, row: int, angles: Tensor, dtype, device):
        self.rows = torch.zeros(batch, ring, kv_heads, row, dtype=dtype, device=device)
        self.angles = angles


class WindowAttention(nn.Module):
    """Grouped-query attention over the last `window` positions (a token itself included): rotary positions on the
    first `rot_dims` elements of queries and keys, capped scores, a learned sink per head, and the keys as projected
    for values.  Keys and values share their cache rows; as many rows as the window are kept.  A mixer of
    `ParallelLayer`."""

    def __init__(self, heads: int, kv_heads: int, dim: int, window: int, scale: float, rot_dims: int, rot_base: float,
                 rot_scaling: Optional[YarnScaling], softcap: float):
        super().__init__()
        self.H, self.G, self.D = heads, kv_heads, dim
        self.window, self.scale, self.softcap = window, scale, softcap
        self.rot_dims, self.rot_base, self.rot_scaling = rot_dims, rot_base, rot_scaling
        self.in_sizes = {"q": heads * dim, "k": kv_heads * dim}
        self.out_size = heads * dim
        self.sink = vector(heads)
        self.register_buffer("sink_f32", torch.zeros(heads), persistent=False)
        self._angles: Optional[Tensor] = None

    def tensors(self) -> Dict[str, Tensor]:
        return {"sink": self.sink}

    def finish_loading(self) -> None:
        self.sink_f32 = self.sink.float()

    def make_cache(self, batch: int, length: int, dtype, device) -> RingRows:
        if self._angles is None or self._angles.shape[0] < length or self._angles.device != torch.device(device):
            self._angles = rotary_angles(length, self.rot_dims, self.rot_base, device, self.rot_scaling)
        return RingRows(batch, min(self.window, length), self.G, self.D + self.rot_dims, self._angles, dtype, device)

    def workspace_bytes(self, cache: RingRows, batch: int) -> int:
        k, v = self.keys_values(cache.rows)
        return ops.attn_workspace((batch, 1, self.H, self.D), k, v, scale=1.0, ring=True, window=self.window)

    def keys_values(self, rows: Tensor) -> Tuple[Tensor, Tensor]:
        return rows[..., self.rot_dims:], rows[..., :self.D]

    def mix(self, parts: List[Tensor], h: Tensor, cache: RingRows, at: Portion, out: Tensor) -> None:
        B, S = at.B, at.S
        q, k = parts[0].unflatten(-1, (self.H, self.D)), parts[1].unflatten(-1, (self.G, self.D))
        ring = cache.rows[:B]
        args = dict(scale=self.scale, softcap=self.softcap, window=self.window, sink=self.sink_f32, status=at.status,
                    workspace=at.workspace, out=out.view(B, S, self.H, self.D))
        if at.pos is not None:
            q = ops.rotary_rows(q, k, cache.angles, self.rot_dims, ring, B=B, S=S, pos=at.pos, status=at.status)
            ops.attn(q, *self.keys_values(ring), pos=at.pos, ring=True, **args)
        else:
            prev = min(at.start, self.window - 1)          # earlier positions that the portion's tokens see
            rows = torch.empty(B, prev + S, *ring.shape[2:], dtype=ring.dtype, device=ring.device)
            q = ops.rotary_rows(q, k, cache.angles, self.rot_dims, rows, B=B, S=S, start=at.start, ring=ring, prev=prev,
                                status=at.status)
            ops.attn(q, *self.keys_values(rows), start=at.start, kv_start=at.start - prev, **args)
            ops.ring_append(rows[:, prev:], None, ring, None, start=at.start, keep="window")


# ---------------------------------------------------------------------------------- matrix memory
class MemoryState:
    """Recurrent state per sequence and head, fp32: the memory, its normaliser, the running maximum of the gates."""

    def __init__(self, batch: int, heads: int, dim: int, vdim: int, device):
        self.S = torch.zeros(batch, heads, dim, vdim, dtype=torch.float32, device=device)
        self.n = torch.zeros(batch, heads, dim, dtype=torch.float32, device=device)
        self.m = torch.zeros(batch, heads, dtype=torch.float32, device=device)


class MatrixMemory(nn.Module):
    """Matrix memory of the xLSTM (mLSTM) with capped exponential input gates and sigmoid forget gates, a norm per
    head and a sigmoid output gate.  The gates' pre-activations are a matrix product of their own, whose fp32 sums
    are not rounded.  A mixer of `ParallelLayer`."""

    def __init__(self, width: int, heads: int, dim: int, vdim: int, gate_cap: float, eps: float):
        super().__init__()
        self.H, self.N, self.P, self.cap, self.eps = heads, dim, vdim, gate_cap, eps
        self.in_sizes = {"q": heads * dim, "k": heads * dim, "v": heads * vdim, "g": heads * vdim}
        self.out_size = heads * vdim
        self.w_gates = projection(padded_rows(2 * heads), width)
        self.i_b, self.f_b, self.norm_w = vector(heads), vector(heads), vector(heads * vdim)
        for name in ("i_b_f32", "f_b_f32"):
            self.register_buffer(name, torch.zeros(heads), persistent=False)

    def tensors(self) -> Dict[str, Tensor]:
        return {"i": self.w_gates[:self.H], "f": self.w_gates[self.H:2 * self.H], "i.b": self.i_b, "f.b": self.f_b,
                "norm": self.norm_w}

    def finish_loading(self) -> None:
        self.i_b_f32, self.f_b_f32 = self.i_b.float(), self.f_b.float()

    def make_cache(self, batch: int, length: int, dtype, device) -> MemoryState:
        return MemoryState(batch, self.H, self.N, self.P, device)

    def workspace_bytes(self, cache: MemoryState, batch: int) -> int:
        return 0

    def mix(self, parts: List[Tensor], h: Tensor, cache: MemoryState, at: Portion, out: Tensor) -> None:
        B = at.B
        ops.mlstm(*parts, matmul_f32(h, self.w_gates), self.i_b_f32, self.f_b_f32, self.norm_w, cache.S[:B], cache.n[:B],
                  cache.m[:B], out, S=at.S, cap=self.cap, q_scale=self.N ** -0.5, eps=self.eps, start=at.start, pos=at.pos,
                  status=at.status)


# ---------------------------------------------------------------------------------- state space
class StateCache:
    """Recurrent state per sequence: the fp32 state and the convolution's last inputs."""

    def __init__(self, batch: int, heads: int, state: int, vdim: int, channels: int, taps: int, dtype, device):
        self.state = torch.zeros(batch, heads, state, vdim, dtype=torch.float32, device=device)
        self.conv = torch.zeros(batch, taps - 1, channels, dtype=dtype, device=device)


class Mamba2(nn.Module):
    """Selective state-space layer with scalar decay per head: projection, short causal convolution,
    fp32 recurrence, gate, grouped norm, projection."""

    def __init__(self, width: int, heads: int, vdim: int, state: int, groups: int, taps: int, norm_groups: int, eps: float):
        super().__init__()
        self.H, self.P, self.N, self.G, self.taps, self.parts, self.eps = heads, vdim, state, groups, taps, norm_groups, eps
        self.inner = heads * vdim
        self.channels = self.inner + 2 * groups * state
        self.in_rows = self.inner + self.channels + heads
        self.w_in = projection(padded_rows(self.in_rows), width)
        self.conv_w = projection(self.channels, taps)
        self.conv_b = vector(self.channels)
        self.dt_bias, self.A_log, self.skip = vector(heads), vector(heads), vector(heads)
        self.norm_w = vector(self.inner)
        self.wo = projection(width, self.inner)
        for name in ("dt_bias_f32", "A_log_f32", "skip_f32"):
            self.register_buffer(name, torch.zeros(heads), persistent=False)

    def tensors(self) -> dict:
        return {"in": self.w_in[:self.in_rows], "conv": self.conv_w, "conv.b": self.conv_b, "dt_bias": self.dt_bias,
                "A_log": self.A_log, "D": self.skip, "norm": self.norm_w, "o": self.wo}

    def finish_loading(self) -> None:
        self.dt_bias_f32, self.A_log_f32, self.skip_f32 = self.dt_bias.float(), self.A_log.float(), self.skip.float()

    def make_cache(self, batch: int, length: int, dtype, device) -> StateCache:
        return StateCache(batch, self.H, self.N, self.P, self.channels, self.taps, dtype, device)

    def workspace_bytes(self, cache: StateCache, batch: int) -> int:
        return 0

    def forward(self, h: Tensor, cache: StateCache, at: Portion) -> Tensor:
        proj = torch.mm(h, self.w_in.t())
        y = ops.ssm(proj, self.inner, self.conv_w, self.conv_b, self.dt_bias_f32, self.A_log_f32, self.skip_f32,
                    cache.conv[:at.B], cache.state[:at.B], S=at.S, groups=self.G, start=at.start, pos=at.pos)
        y = ops.gated_group_norm(y, proj, self.norm_w, self.parts, self.eps)
        return torch.mm(y, self.wo.t())


# ---------------------------------------------------------------------------------- feed-forward
class ClampedFeedForward(nn.Module):
    """g = min(W_gate h, limit), u = clamp(W_up h), out = W_down (g sigmoid(1.702 g) (u + 1)); gate and up
    projection are one GEMM."""

    def __init__(self, width: int, ff: int, limit: float):
        super().__init__()
        self.ff, self.limit = ff, limit
        self.w13 = projection(padded_rows(2 * ff), width)
        self.w2 = projection(width, ff)

    def tensors(self) -> dict:
        return {"gate": self.w13[:self.ff], "up": self.w13[self.ff:2 * self.ff], "down": self.w2}

    def forward(self, h: Tensor) -> Tensor:
        return torch.mm(ops.glu_clamped(torch.mm(h, self.w13.t()), self.ff, self.limit), self.w2.t())


class ParallelLayer(nn.Module):
    """A layer whose mixer and feed-forward (silu-gated; ff = 0: none) read the same normed rows and add to the
    stream together: one matrix product makes every projection of both, one takes [mixer | feed-forward] to what
    the stream gets, summed in fp32."""

    def __init__(self, width: int, mixer: nn.Module, ff: int):
        super().__init__()
        self.mixer, self.ff = mixer, ff
        self.norm1 = vector(width)
        sizes = list(mixer.in_sizes.values()) + ([ff, ff] if ff else [])
        self.in_slices, rows = [], 0
        for n in sizes:                            # every slice starts at a multiple of 8 columns of the projected rows
            self.in_slices.append(slice(rows, rows + n))
            rows += padded_rows(n)
        self.w_in = projection(rows, width)
        self.ff_at = padded_rows(mixer.out_size)
        self.cols = self.ff_at + padded_rows(ff)
        self.gaps = self.cols != mixer.out_size + ff
        self.w_out = projection(width, self.cols)

    def tensors(self) -> Dict[str, Tensor]:
        out = {"norm1": self.norm1, "mix.o": self.w_out[:, :self.mixer.out_size]}
        for name, s in zip(self.mixer.in_sizes, self.in_slices):
            out["mix." + name] = self.w_in[s]
        out.update({"mix." + k: v for k, v in self.mixer.tensors().items()})
        if self.ff:
            gate, up = self.in_slices[-2:]
            out.update({"mlp.gate": self.w_in[gate], "mlp.up": self.w_in[up],
                        "mlp.down": self.w_out[:, self.ff_at:self.ff_at + self.ff]})
        return out

    def forward(self, h: Tensor, cache, at: Portion) -> Tensor:
        proj = torch.mm(h, self.w_in.t())
        parts = [proj[:, s] for s in self.in_slices]
        make = torch.zeros if self.gaps else torch.empty           # columns between the two parts meet zero weights
        inner = make(h.shape[0], self.cols, dtype=h.dtype, device=h.device)
        self.mixer.mix(parts[:len(self.mixer.in_sizes)], h, cache, at, inner[:, :self.mixer.out_size])
        if self.ff:
            ops.glu_silu(*parts[-2:], out=inner[:, self.ff_at:self.ff_at + self.ff])
        return matmul_f32(inner, self.w_out)
