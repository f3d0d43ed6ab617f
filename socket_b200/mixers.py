"""Token mixers and the feed-forward built on the block library (`block_ops.py`): chunk-masked attention
with a learned distance bias, attention on a low-rank latent, a selective state-space layer, and a
clamped gated unit.  Every size and constant is a parameter, so that any decoder can list them.

A mixer maps hidden rows [B*S, width] of a portion to rows of the same shape and advances its cache:
`make_cache(...)` builds it, `forward(h, cache, at)` uses it.  `at` (`Portion`) says where the portion
sits; a decode step is the portion of one token whose position is read on the device.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

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

    def decode_shapes(self, cache: RingCache, batch: int):
        return (batch, 1, self.H, self.D), cache.k, cache.v

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
def rotary_angles(length: int, dims: int, base: float, device) -> Tensor:
    """[length, dims / 2, 2] = (cos, sin) of position * base^(-2i / dims), fp32."""
    f = base ** (-torch.arange(0, dims, 2, dtype=torch.float64) / dims)
    a = torch.outer(torch.arange(length, dtype=torch.float64), f)
    return torch.stack([torch.cos(a), torch.sin(a)], -1).float().contiguous().to(device)


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

    def decode_shapes(self, cache: LatentCache, batch: int):
        rows = cache.rows.unsqueeze(2)
        return (batch, self.expand_from - 1, self.H, self.row), rows, rows[..., :self.K]

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
