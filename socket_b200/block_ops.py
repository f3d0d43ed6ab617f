"""Tensor-level wrappers of the building-block library (`include/socket_b200_blocks.h`): shapes and
dtypes are checked here, outputs are allocated with torch, kernels go to torch's current stream.
Nothing synchronises with the host and nothing has a CPU path."""
from __future__ import annotations

import ctypes as C
from typing import Optional

import torch
from torch import Tensor

from . import _lib
from ._lib import blocks, check_blocks, dtype_code, ptr, stream_ptr
from .ops import _require_cuda

ATTN_PATHS = {"auto": 0, "rows": 1, "prefill_tc": 2, "decode": 3}
SSM_PATHS = {"auto": 0, "steps": 1, "chunks": 2}
IN_NONE, IN_ADD_NORM, IN_REPLACE = 0, 1, 2
OUT_NONE, OUT_NORM, OUT_CONCAT = 0, 1, 2
GLU_SLOPE = 1.702


def embed_rows(tokens: Tensor, table: Tensor, scale: float, keep_copy: bool = False,
               status: Optional[Tensor] = None):
    """tokens [...] int64 -> fp32 rows [n, width] = table[token] * scale, and a second copy if asked for."""
    _require_cuda(tokens, table)
    tokens = tokens.contiguous()
    assert tokens.dtype == torch.int64 and table.is_contiguous()
    n, (vocab, width) = tokens.numel(), table.shape
    x = torch.empty(n, width, dtype=torch.float32, device=table.device)
    x0 = torch.empty_like(x) if keep_copy else None
    check_blocks(blocks().skb_embed_rows(ptr(tokens), ptr(table), dtype_code(table), n, vocab, width, float(scale), ptr(x),
                                         ptr(x0), ptr(status), stream_ptr(table.device)), "skb_embed_rows")
    return x, x0


def residual_norm(x: Tensor, eps: float, *, y: Optional[Tensor] = None, w_in: Optional[Tensor] = None,
                  replace: bool = False, w_out: Optional[Tensor] = None, x0: Optional[Tensor] = None,
                  dtype: Optional[torch.dtype] = None) -> Optional[Tensor]:
    """The residual stream x [rows, width] (fp32, updated in place): x += rms_norm(y) * w_in, or x = y + w_in
    with `replace`; then returns rms_norm(x) * w_out, or [x ; x0], or nothing.  `dtype`: element type of the
    weights and of the result (taken from the weights when there are any)."""
    _require_cuda(x, y, w_in, w_out, x0)
    rows, width = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous()
    for w in (w_in, w_out):
        if w is not None:
            assert w.shape == (width,) and w.is_contiguous() and (dtype is None or dtype == w.dtype)
            dtype = w.dtype
    p = _lib.ResidualParams()
    p.x, p.rows, p.width, p.eps = ptr(x), rows, width, float(eps)
    p.dtype = p.y_dtype = _lib.DTYPE_CODE[dtype]
    p.y_ld = width
    if y is not None:
        assert y.shape == (rows, width) and y.stride(1) == 1
        p.y, p.y_ld, p.y_dtype, p.w_in = ptr(y), y.stride(0), dtype_code(y), ptr(w_in)
        p.in_mode = IN_REPLACE if replace else IN_ADD_NORM
    out = None
    if w_out is not None:
        out = torch.empty(rows, width, dtype=dtype, device=x.device)
        p.w_out, p.out_mode = ptr(w_out), OUT_NORM
    elif x0 is not None:
        assert x0.shape == x.shape and x0.dtype == torch.float32 and x0.is_contiguous()
        out = torch.empty(rows, 2 * width, dtype=dtype, device=x.device)
        p.x0, p.out_mode = ptr(x0), OUT_CONCAT
    p.out = ptr(out)
    check_blocks(blocks().skb_residual_norm(C.byref(p), stream_ptr(x.device)), "skb_residual_norm")
    return out


def glu_clamped(gate_up: Tensor, ff: int, limit: float, slope: float = GLU_SLOPE) -> Tensor:
    """gate_up [rows, >= 2 ff] = [gate | up] -> [rows, ff]."""
    _require_cuda(gate_up)
    assert gate_up.stride(1) == 1 and gate_up.shape[1] >= 2 * ff
    out = torch.empty(gate_up.shape[0], ff, dtype=gate_up.dtype, device=gate_up.device)
    check_blocks(blocks().skb_glu_clamped(ptr(gate_up), dtype_code(gate_up), gate_up.shape[0], ff, gate_up.stride(0),
                                          float(limit), float(slope), ptr(out), stream_ptr(out.device)), "skb_glu_clamped")
    return out


def ring_append(k: Tensor, v: Tensor, k_cache: Tensor, v_cache: Tensor, start: int = 0,
                pos: Optional[Tensor] = None) -> None:
    """k [B,S,G,D], v [B,S,G,E] (token rows may be strided) -> k_cache [B,ring,G,D], v_cache [B,ring,G,E]."""
    _require_cuda(k, v, k_cache, v_cache, pos)
    B, S, G, D = k.shape
    E = v.shape[3]
    ring = k_cache.shape[1]
    assert k.stride(3) == 1 and (G == 1 or k.stride(2) == D) and v.stride(3) == 1 and (G == 1 or v.stride(2) == E)
    assert k_cache.is_contiguous() and v_cache.is_contiguous() and k_cache.shape[2:] == (G, D)
    assert v_cache.shape[1:] == (ring, G, E)
    check_blocks(blocks().skb_ring_append(ptr(k), ptr(v), dtype_code(k), B, S, k.stride(0), k.stride(1), v.stride(0),
                                          v.stride(1), G * D, G * E, ring, ptr(pos), start, ptr(k_cache), ptr(v_cache),
                                          stream_ptr(k.device)), "skb_ring_append")


def attn_params(q: Tensor, k: Tensor, v: Tensor, out: Tensor, *, scale: float, start: int = 0,
                pos: Optional[Tensor] = None, kv_start: int = 0, chunk: int = 0, ring: bool = False,
                bias: Optional[Tensor] = None, sink: Optional[Tensor] = None, status: Optional[Tensor] = None,
                workspace: Optional[Tensor] = None, path: str = "auto", meta: bool = False) -> _lib.AttnParams:
    """The parameter block of one call.  With `meta` q and out are shapes only (for a size query)."""
    B, S, H, dqk = q.shape
    G, dv = k.shape[2], v.shape[3]
    assert k.shape[3] == dqk and v.shape[:3] == k.shape[:3] and out.shape == (B, S, H, dv)
    assert q.dtype == k.dtype == v.dtype == out.dtype
    for t in (q, k, v, out):
        assert t.stride(3) == 1
    p = _lib.AttnParams()
    p.q, p.k, p.v, p.out = (0, 0, 0, 0) if meta else (ptr(q), ptr(k), ptr(v), ptr(out))
    p.q_bs, p.q_ss, p.q_hs = q.stride()[:3]
    p.k_bs, p.k_ts, p.k_hs = k.stride()[:3]
    p.v_bs, p.v_ts, p.v_hs = v.stride()[:3]
    p.o_bs, p.o_ss, p.o_hs = out.stride()[:3]
    p.dtype, p.B, p.S, p.H, p.G, p.dqk, p.dv = dtype_code(q), B, S, H, G, dqk, dv
    p.start, p.pos, p.kv_start, p.kv_rows = start, ptr(pos), kv_start, k.shape[1]
    p.chunk, p.ring, p.scale, p.path = chunk, int(ring), float(scale), ATTN_PATHS[path]
    if bias is not None:
        assert bias.dtype == torch.float32 and bias.is_contiguous() and bias.shape[0] == H
        p.bias, p.bias_len = ptr(bias), bias.shape[1]
    if sink is not None:
        assert sink.dtype == torch.float32 and sink.shape == (H,)
        p.sink = ptr(sink)
    p.status = ptr(status)
    if workspace is not None:
        p.workspace, p.workspace_bytes = ptr(workspace), workspace.numel()
    return p


def attn(q: Tensor, k: Tensor, v: Tensor, **kw) -> Tensor:
    """Softmax attention of a portion: q [B,S,H,dqk], k [B,rows,G,dqk], v [B,rows,G,dv] -> [B,S,H,dv].
    Keyword arguments as in `attn_params`; a workspace that is absent or too small is allocated when the kernel needs one."""
    _require_cuda(q, k, v)
    out = torch.empty(*q.shape[:3], v.shape[3], dtype=q.dtype, device=q.device)
    p = attn_params(q, k, v, out, **kw)
    need = int(blocks().skb_attn_workspace_bytes(C.byref(p)))
    if need > p.workspace_bytes:
        ws = torch.empty(need, dtype=torch.uint8, device=q.device)
        p.workspace, p.workspace_bytes = ptr(ws), need
    check_blocks(blocks().skb_attn(C.byref(p), stream_ptr(q.device)), "skb_attn")
    return out


def latent_append(dkv: Tensor, q: Tensor, norm_w: Tensor, angles: Tensor, cache: Tensor, *, S: int, n_heads: int, dim: int,
                  rot: int, rank: int, eps: float, start: int = 0, pos: Optional[Tensor] = None,
                  status: Optional[Tensor] = None) -> None:
    """dkv [B*S, rank + rot] -> rows of cache [B, cap, ld]; q [B*S, H * (dim + rot)] turned in place.
    angles [>= cap, rot_dims / 2, 2] fp32."""
    _require_cuda(dkv, q, norm_w, angles, cache)
    B, cap, ld = cache.shape
    assert dkv.shape == (B * S, rank + rot) and q.shape == (B * S, n_heads * (dim + rot))
    assert dkv.stride(1) == 1 and q.stride(1) == 1 and cache.is_contiguous()
    assert angles.dtype == torch.float32 and angles.is_contiguous() and angles.shape[0] >= cap and angles.shape[2] == 2
    p = _lib.LatentParams()
    p.dkv, p.q, p.norm_w, p.angles, p.cache = ptr(dkv), ptr(q), ptr(norm_w), ptr(angles), ptr(cache)
    p.pos, p.status, p.start = ptr(pos), ptr(status), start
    p.dkv_ld, p.q_ld, p.cap, p.cache_ld = dkv.stride(0), q.stride(0), cap, ld
    p.dtype, p.B, p.S, p.H, p.dim, p.rot, p.rot_dims, p.rank = dtype_code(dkv), B, S, n_heads, dim, rot, 2 * angles.shape[1], rank
    p.eps = float(eps)
    check_blocks(blocks().skb_latent_append(C.byref(p), stream_ptr(dkv.device)), "skb_latent_append")


def latent_absorb(q: Tensor, uk: Tensor, n_heads: int, dim: int, rot: int, out_ld: int) -> Tensor:
    """q [rows, H * (dim + rot)], uk [H * dim, rank] -> [rows, H, out_ld] queries against latent rows."""
    _require_cuda(q, uk)
    rank = uk.shape[1]
    assert uk.shape[0] == n_heads * dim and uk.is_contiguous() and q.stride(1) == 1
    out = torch.empty(q.shape[0], n_heads, out_ld, dtype=q.dtype, device=q.device)
    check_blocks(blocks().skb_latent_absorb(ptr(q), q.stride(0), dtype_code(q), ptr(uk), q.shape[0], n_heads, dim, rot, rank,
                                            out_ld, ptr(out), stream_ptr(q.device)), "skb_latent_absorb")
    return out


def latent_up(o: Tensor, uv: Tensor, vdim: int) -> Tensor:
    """o [rows, H, rank], uv [H * vdim, rank] -> [rows, H * vdim]."""
    _require_cuda(o, uv)
    rows, H, rank = o.shape
    assert o.is_contiguous() and uv.is_contiguous() and uv.shape == (H * vdim, rank)
    out = torch.empty(rows, H * vdim, dtype=o.dtype, device=o.device)
    check_blocks(blocks().skb_latent_up(ptr(o), dtype_code(o), ptr(uv), rows, H, vdim, rank, ptr(out), stream_ptr(o.device)),
                 "skb_latent_up")
    return out


def ssm(proj: Tensor, inner: int, conv_w: Tensor, conv_b: Tensor, dt_bias: Tensor, A_log: Tensor, D: Tensor,
        conv_state: Tensor, state: Tensor, *, S: int, groups: int, start: int = 0, pos: Optional[Tensor] = None,
        path: str = "auto") -> Tensor:
    """proj rows [z | x | B | C | dt] (B*S of them, strided) -> y [B*S, inner] before the gate; conv_state
    [B, taps - 1, channels] and state [B, H, N, P] (fp32) are advanced by the portion."""
    _require_cuda(proj, conv_w, conv_b, dt_bias, A_log, D, conv_state, state)
    B, H, N, P = state.shape
    channels, taps = conv_w.shape
    rows = proj.shape[0]
    assert rows == B * S and inner == H * P and channels == inner + 2 * groups * N and proj.stride(1) == 1
    assert proj.shape[1] >= inner + channels + H and conv_w.is_contiguous() and state.is_contiguous()
    assert state.dtype == torch.float32 and conv_state.shape == (B, taps - 1, channels) and conv_state.dtype == proj.dtype
    assert conv_state.is_contiguous() and all(t.dtype == torch.float32 and t.numel() == H for t in (dt_bias, A_log, D))
    xbc_ld = (channels + 7) // 8 * 8
    xbc = torch.empty(rows, xbc_ld, dtype=proj.dtype, device=proj.device)
    y = torch.empty(rows, inner, dtype=proj.dtype, device=proj.device)
    p = _lib.SsmParams()
    es = proj.element_size()
    p.xbc_in, p.dt_in = ptr(proj) + inner * es, ptr(proj) + (inner + channels) * es
    p.conv_w, p.conv_b, p.conv_state, p.xbc, p.y = ptr(conv_w), ptr(conv_b), ptr(conv_state), ptr(xbc), ptr(y)
    p.dt_bias, p.A_log, p.D, p.state, p.pos, p.start = ptr(dt_bias), ptr(A_log), ptr(D), ptr(state), ptr(pos), start
    p.in_ld, p.xbc_ld = proj.stride(0), xbc_ld
    p.dtype, p.B, p.S, p.H, p.P, p.N, p.G, p.taps = dtype_code(proj), B, S, H, P, N, groups, taps
    p.path = SSM_PATHS[path]
    need = int(blocks().skb_ssm_workspace_bytes(C.byref(p)))
    ws = torch.empty(need, dtype=torch.uint8, device=proj.device) if need else None
    p.workspace, p.workspace_bytes = ptr(ws), need
    st = stream_ptr(proj.device)
    check_blocks(blocks().skb_ssm_conv(C.byref(p), st), "skb_ssm_conv")
    check_blocks(blocks().skb_ssm_scan(C.byref(p), st), "skb_ssm_scan")
    return y


def gated_group_norm(y: Tensor, z: Tensor, w: Tensor, parts: int, eps: float) -> Tensor:
    """y [rows, inner], z rows (strided, at least inner wide) -> [rows, inner]."""
    _require_cuda(y, z, w)
    rows, inner = y.shape
    assert y.is_contiguous() and z.stride(1) == 1 and z.shape[0] == rows and w.shape == (inner,)
    out = torch.empty_like(y)
    check_blocks(blocks().skb_gated_group_norm(ptr(y), ptr(z), z.stride(0), ptr(w), dtype_code(y), rows, inner, parts,
                                               float(eps), ptr(out), stream_ptr(y.device)), "skb_gated_group_norm")
    return out
