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
SSM_PATHS = {"auto": 0, "steps": 1, "chunks": 2, "tensor": 3}
IN_NONE, IN_ADD_NORM, IN_REPLACE, IN_ADD = 0, 1, 2, 3
OUT_NONE, OUT_NORM, OUT_CONCAT, OUT_LAYER_NORM = 0, 1, 2, 3
GLU_CLAMPED, GLU_SILU = 0, 1
RING_KEEP = {"chunk": 0, "window": 1}
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
                  dtype: Optional[torch.dtype] = None, centred: bool = False) -> Optional[Tensor]:
    """The residual stream x [rows, width] (fp32, updated in place): x += rms_norm(y) * w_in, x = y + w_in with
    `replace`, or x += y without w_in; then returns rms_norm(x) * w_out (with `centred`: the layer norm), or
    [x ; x0], or nothing.  `dtype`: element type of the weights and of the result (taken from the weights when
    there are any)."""
    _require_cuda(x, y, w_in, w_out, x0)
    rows, width = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous()
    for w in (w_in, w_out):
        if w is not None:
            assert w.shape == (width,) and w.is_contiguous() and (dtype is None or dtype == w.dtype)
            dtype = w.dtype
    p = _lib.ResidualParams()
    p.x, p.rows, p.width, p.eps = ptr(x), rows, width, float(eps)
    if dtype is None:                              # nothing but x and y: the element type does not matter
        dtype = torch.float32 if y is None else y.dtype
    p.dtype = p.y_dtype = _lib.DTYPE_CODE[dtype]
    p.y_ld = width
    if y is not None:
        assert y.shape == (rows, width) and y.stride(1) == 1
        p.y, p.y_ld, p.y_dtype, p.w_in = ptr(y), y.stride(0), dtype_code(y), ptr(w_in)
        p.in_mode = IN_REPLACE if replace else (IN_ADD if w_in is None else IN_ADD_NORM)
    out = None
    if w_out is not None:
        out = torch.empty(rows, width, dtype=dtype, device=x.device)
        p.w_out, p.out_mode = ptr(w_out), OUT_LAYER_NORM if centred else OUT_NORM
    elif x0 is not None:
        assert x0.shape == x.shape and x0.dtype == torch.float32 and x0.is_contiguous()
        out = torch.empty(rows, 2 * width, dtype=dtype, device=x.device)
        p.x0, p.out_mode = ptr(x0), OUT_CONCAT
    p.out = ptr(out)
    check_blocks(blocks().skb_residual_norm(C.byref(p), stream_ptr(x.device)), "skb_residual_norm")
    return out


def _glu(gate: Tensor, up: Tensor, kind: int, limit: float, slope: float, out: Optional[Tensor]) -> Tensor:
    _require_cuda(gate, up, out)
    rows, ff = gate.shape
    if out is None:
        out = torch.empty(rows, ff, dtype=gate.dtype, device=gate.device)
    assert gate.stride(1) == up.stride(1) == out.stride(1) == 1 and gate.stride(0) == up.stride(0) and up.shape == gate.shape
    assert out.shape == gate.shape and out.dtype == up.dtype == gate.dtype
    check_blocks(blocks().skb_glu(ptr(gate), ptr(up), dtype_code(gate), rows, ff, gate.stride(0), kind, float(limit), float(slope),
                                  ptr(out), out.stride(0), stream_ptr(out.device)), "skb_glu")
    return out


def glu_clamped(gate_up: Tensor, ff: int, limit: float, slope: float = GLU_SLOPE) -> Tensor:
    """gate_up [rows, >= 2 ff] = [gate | up] -> g * sigmoid(slope * g) * (u + 1) of the clamped halves, [rows, ff]."""
    assert gate_up.shape[1] >= 2 * ff
    return _glu(gate_up[:, :ff], gate_up[:, ff:2 * ff], GLU_CLAMPED, limit, slope, None)


def glu_silu(gate: Tensor, up: Tensor, out: Optional[Tensor] = None) -> Tensor:
    """silu(gate) * up of rows [rows, ff] that may be slices of wider ones; `out` too."""
    return _glu(gate, up, GLU_SILU, 0.0, 1.0, out)


def ring_append(k: Tensor, v: Optional[Tensor], k_cache: Tensor, v_cache: Optional[Tensor], start: int = 0,
                pos: Optional[Tensor] = None, keep: str = "chunk") -> None:
    """k [B,S,G,D], v [B,S,G,E] (token rows may be strided) -> k_cache [B,ring,G,D], v_cache [B,ring,G,E]; v and
    v_cache may be None.  `keep`: of a portion longer than the ring, the tokens of its last chunk of `ring`
    positions, or its last `ring` tokens ("window")."""
    _require_cuda(k, v, k_cache, v_cache, pos)
    B, S, G, D = k.shape
    ring = k_cache.shape[1]
    assert k.stride(3) == 1 and (G == 1 or k.stride(2) == D)
    assert k_cache.is_contiguous() and k_cache.shape[2:] == (G, D) and (v is None) == (v_cache is None)
    E = vbs = vss = 0
    if v is not None:
        E, vbs, vss = v.shape[3], v.stride(0), v.stride(1)
        assert v.stride(3) == 1 and (G == 1 or v.stride(2) == E) and v_cache.is_contiguous() and v_cache.shape[1:] == (ring, G, E)
    check_blocks(blocks().skb_ring_append(ptr(k), ptr(v), dtype_code(k), B, S, k.stride(0), k.stride(1), vbs, vss, G * D, G * E,
                                          ring, RING_KEEP[keep], ptr(pos), start, ptr(k_cache), ptr(v_cache),
                                          stream_ptr(k.device)), "skb_ring_append")


def rotary_rows(q: Tensor, k: Tensor, angles: Tensor, rot_dims: int, rows: Tensor, *, B: int, S: int, start: int = 0,
                pos: Optional[Tensor] = None, ring: Optional[Tensor] = None, prev: int = 0,
                status: Optional[Tensor] = None) -> Tensor:
    """q [B*S, H, dim], k [B*S, G, dim]: slices of the same projection rows.  Fills rows [B, cap, G, dim + rot_dims]
    (value = [..., :dim], key = [..., rot_dims:]) with the last `prev` positions before `start` out of `ring`,
    then the new tokens; with `pos`, row pos % cap with the one new token.  Returns the queries [B, S, H, dim]
    in the keys' element order.  angles [positions, rot_dims / 2, 2] fp32."""
    _require_cuda(q, k, angles, rows, ring)
    n, H, dim = q.shape
    G = k.shape[1]
    assert n == B * S == k.shape[0] and k.shape[2] == dim and q.stride(0) == k.stride(0) or n == 1
    assert q.stride()[1:] == (dim, 1) and k.stride()[1:] == (dim, 1)
    assert rows.is_contiguous() and rows.shape[2:] == (G, dim + rot_dims) and rows.shape[0] >= B
    assert angles.dtype == torch.float32 and angles.is_contiguous() and angles.shape[1:] == (rot_dims // 2, 2)
    assert ring is None or (ring.is_contiguous() and ring.shape[2:] == rows.shape[2:])
    out = torch.empty(B, S, H, dim, dtype=q.dtype, device=q.device)
    p = _lib.RotaryRowsParams()
    p.q_in, p.k_in, p.ring, p.q_out, p.rows_out = ptr(q), ptr(k), ptr(ring), ptr(out), ptr(rows)
    p.angles, p.pos, p.status = ptr(angles), ptr(pos), ptr(status)
    p.in_ld, p.start, p.n_pos, p.rows_cap = q.stride(0), start, angles.shape[0], rows.shape[1]
    p.ring_rows = 0 if ring is None else ring.shape[1]
    p.dtype, p.B, p.S, p.H, p.G, p.dim, p.rot_dims, p.prev = dtype_code(q), B, S, H, G, dim, rot_dims, prev
    check_blocks(blocks().skb_rotary_rows(C.byref(p), stream_ptr(q.device)), "skb_rotary_rows")
    return out


def attn_params(q: Tensor, k: Tensor, v: Tensor, out: Tensor, *, scale: float, start: int = 0,
                pos: Optional[Tensor] = None, kv_start: int = 0, chunk: int = 0, window: int = 0, ring: bool = False,
                softcap: float = 0.0, bias: Optional[Tensor] = None, sink: Optional[Tensor] = None, status: Optional[Tensor] = None,
                workspace: Optional[Tensor] = None, path: str = "auto", meta: bool = False) -> _lib.AttnParams:
    """The parameter block of one call.  With `meta` q and out are shapes only (for a size query).  A window of 0
    or a cap of 0 is none."""
    B, S, H, dqk = q.shape
    G, dv = k.shape[2], v.shape[3]
    assert k.shape[3] == dqk and v.shape[:3] == k.shape[:3] and out.shape == (B, S, H, dv)
    assert q.dtype == k.dtype == v.dtype == out.dtype
    for t in (q, k, v, out):
        assert t.stride(3) == 1
    p = _lib.AttnParams()
    p.k, p.v = ptr(k), ptr(v)
    p.q, p.out = (0, 0) if meta else (ptr(q), ptr(out))
    p.q_bs, p.q_ss, p.q_hs = q.stride()[:3]
    p.k_bs, p.k_ts, p.k_hs = k.stride()[:3]
    p.v_bs, p.v_ts, p.v_hs = v.stride()[:3]
    p.o_bs, p.o_ss, p.o_hs = out.stride()[:3]
    p.dtype, p.B, p.S, p.H, p.G, p.dqk, p.dv = dtype_code(q), B, S, H, G, dqk, dv
    p.start, p.pos, p.kv_start, p.kv_rows = start, ptr(pos), kv_start, k.shape[1]
    p.chunk, p.window, p.ring, p.path = chunk, window, int(ring), ATTN_PATHS[path]
    p.scale, p.softcap = float(scale), float(softcap)
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


def attn_workspace(q_shape, k: Tensor, v: Tensor, **kw) -> int:
    """Scratch bytes of `attn` for queries of shape [B,S,H,dqk]; keyword arguments as there."""
    q = torch.empty(q_shape, dtype=k.dtype, device="meta")
    o = torch.empty(*q_shape[:3], v.shape[3], dtype=k.dtype, device="meta")
    return int(blocks().skb_attn_workspace_bytes(C.byref(attn_params(q, k, v, o, meta=True, **kw))))


def attn(q: Tensor, k: Tensor, v: Tensor, out: Optional[Tensor] = None, **kw) -> Tensor:
    """Softmax attention of a portion: q [B,S,H,dqk], k [B,rows,G,dqk], v [B,rows,G,dv] -> [B,S,H,dv] (`out`: rows may be
    slices of wider ones).  Keyword arguments as in `attn_params`; a workspace that is absent or too small is allocated when the kernel needs one."""
    _require_cuda(q, k, v)
    if out is None:
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


def mlstm(q: Tensor, k: Tensor, v: Tensor, z: Tensor, gates: Tensor, i_bias: Tensor, f_bias: Tensor, norm_w: Tensor,
          S_state: Tensor, n_state: Tensor, m_state: Tensor, out: Tensor, *, S: int, cap: float, q_scale: float, eps: float,
          start: int = 0, pos: Optional[Tensor] = None, status: Optional[Tensor] = None, path: str = "auto") -> Tensor:
    """Matrix memory of B * S tokens: q, k [rows, H * N], v, z [rows, H * P] are slices of the same projection rows;
    gates [rows, >= 2 H] = [input | forget] fp32 before their biases.  S_state [B, H, N, P], n_state [B, H, N] and
    m_state [B, H] (fp32) are advanced by the portion; out [rows, H * P] (may be a slice) is normed per head and gated."""
    _require_cuda(q, k, v, z, gates, i_bias, f_bias, norm_w, S_state, n_state, m_state, out)
    B, H, N, P = S_state.shape
    rows = q.shape[0]
    assert rows == B * S and q.shape[1] == k.shape[1] == H * N and v.shape[1] == z.shape[1] == out.shape[1] == H * P
    assert all(t.stride(1) == 1 and t.stride(0) == q.stride(0) and t.dtype == q.dtype for t in (q, k, v, z))
    assert out.stride(1) == 1 and out.dtype == q.dtype and gates.dtype == torch.float32 and gates.stride(1) == 1
    assert gates.shape[0] == rows and gates.shape[1] >= 2 * H and norm_w.shape == (H * P,) and norm_w.dtype == q.dtype
    for t, shape in ((S_state, (B, H, N, P)), (n_state, (B, H, N)), (m_state, (B, H)), (i_bias, (H,)), (f_bias, (H,))):
        assert t.dtype == torch.float32 and t.is_contiguous() and t.shape == shape
    dev = q.device
    num = torch.empty(rows, H * P, dtype=q.dtype, device=dev)
    den = torch.empty(rows, H, dtype=torch.float32, device=dev)
    m_next = torch.empty(B, H, dtype=torch.float32, device=dev)
    p = _lib.MlstmParams()
    p.q, p.k, p.v, p.z, p.norm_w, p.gates, p.i_bias, p.f_bias = (ptr(t) for t in (q, k, v, z, norm_w, gates, i_bias, f_bias))
    p.S_state, p.n_state, p.m_state, p.num, p.den, p.m_next, p.out = (ptr(t) for t in (S_state, n_state, m_state, num, den,
                                                                                       m_next, out))
    p.status = ptr(status)
    p.pos, p.start, p.in_ld, p.gates_ld, p.out_ld = ptr(pos), start, q.stride(0), gates.stride(0), out.stride(0)
    p.dtype, p.B, p.S, p.H, p.N, p.P, p.path = dtype_code(q), B, S, H, N, P, SSM_PATHS[path]
    p.cap, p.q_scale, p.eps = float(cap), float(q_scale), float(eps)
    need = int(blocks().skb_mlstm_workspace_bytes(C.byref(p)))
    ws = torch.empty(need, dtype=torch.uint8, device=dev) if need else None
    p.workspace, p.workspace_bytes = ptr(ws), need
    check_blocks(blocks().skb_mlstm(C.byref(p), stream_ptr(dev)), "skb_mlstm")
    return out


def gated_group_norm(y: Tensor, z: Tensor, w: Tensor, parts: int, eps: float) -> Tensor:
    """y [rows, inner], z rows (strided, at least inner wide) -> [rows, inner]."""
    _require_cuda(y, z, w)
    rows, inner = y.shape
    assert y.is_contiguous() and z.stride(1) == 1 and z.shape[0] == rows and w.shape == (inner,)
    out = torch.empty_like(y)
    check_blocks(blocks().skb_gated_group_norm(ptr(y), ptr(z), z.stride(0), ptr(w), dtype_code(y), rows, inner, parts,
                                               float(eps), ptr(out), stream_ptr(y.device)), "skb_gated_group_norm")
    return out
