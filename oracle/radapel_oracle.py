"""Plain restatement of the Radapel decoder, one function per mechanism, written for reading:
explicit loops over positions and heads, one sequence at a time, no cache, any float dtype
(float64 by default).  Test infrastructure: shares no code with `socket_b200`.

Weights are a dict name -> tensor in the checkpoint's naming; `cfg` is the parsed config.json.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensor = torch.Tensor


# ------------------------------------------------------------------------------- mechanisms
def rms_norm(x: Tensor, w: Optional[Tensor], eps: float) -> Tensor:
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def distance_bucket(n: int, rows: int, far: float) -> int:
    """Bucket of the distance n >= 0: the first half of the rows one distance each, the rest
    logarithmic up to `far`."""
    half = rows // 2
    if n < half:
        return n
    if n >= far:
        return rows - 1
    step = math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-12)
    return min(rows - 1, half + step)


def softmax_attend(scores: Tensor, values: Tensor, sink: Optional[float] = None) -> Tensor:
    """One query: softmax over `scores` [n] (optionally with a weightless extra term exp(sink) in the
    denominator) of the rows of `values` [n, vdim]."""
    top = scores.max()
    if sink is not None:
        top = torch.maximum(top, torch.as_tensor(sink, dtype=scores.dtype))
    e = torch.exp(scores - top)
    den = e.sum()
    if sink is not None:
        den = den + torch.exp(torch.as_tensor(sink, dtype=scores.dtype) - top)
    return (e / den) @ values


def rotate_pairs(x: Tensor, pos: int, dims: int, base: float) -> Tensor:
    """Rotate the interleaved pairs of the first `dims` elements of a vector by the angles of `pos`."""
    y = x.clone()
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        c, s = math.cos(a), math.sin(a)
        u, v = x[2 * i], x[2 * i + 1]
        y[2 * i] = u * c - v * s
        y[2 * i + 1] = v * c + u * s
    return y


def chunked_attention(h: Tensor, w: Dict[str, Tensor], m: dict) -> Tensor:
    """Grouped-query attention inside chunks of fixed size, with a learned distance bias."""
    S, H, G, D, E, C = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["mask"]["size"]
    q = (h @ w["q"].T).view(S, H, D)
    k = (h @ w["k"].T).view(S, G, D)
    v = (h @ w["v"].T).view(S, G, E)
    rel = w["rel"]
    bias = torch.stack([rel[distance_bucket(n, rel.shape[0], m["bias_max"])] for n in range(min(C, S))])   # [n, H]
    out = torch.empty(S, H, E, dtype=h.dtype)
    for i in range(S):
        lo = i // C * C
        for a in range(H):
            g = a // (H // G)
            sc = k[lo:i + 1, g] @ q[i, a] * m["scale"] + torch.flip(bias[:i + 1 - lo, a], [0])
            out[i, a] = softmax_attend(sc, v[lo:i + 1, g])
    return out.reshape(S, H * E) @ w["o"].T


def latent_attention(h: Tensor, w: Dict[str, Tensor], m: dict, eps: float) -> Tensor:
    """Attention on a shared low-rank latent, one rotated key part common to all heads, a sink per head."""
    S, H, D, R, E, K = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w["q"].T).view(S, H, D + R)
    dkv = h @ w["dkv"].T
    c = rms_norm(dkv[:, :K], w["dkv.norm"], eps)
    kr = torch.stack([rotate_pairs(dkv[j, K:], j, m["rot"]["dims"], m["rot"]["base"]) for j in range(S)])
    ku = (c @ w["uk"].T).view(S, H, D)
    v = (c @ w["uv"].T).view(S, H, E)
    out = torch.empty(S, H, E, dtype=h.dtype)
    for i in range(S):
        for a in range(H):
            qr = rotate_pairs(q[i, a, D:], i, m["rot"]["dims"], m["rot"]["base"])
            sc = (ku[:i + 1, a] @ q[i, a, :D] + kr[:i + 1] @ qr) * m["scale"]
            out[i, a] = softmax_attend(sc, v[:i + 1, a], w["sink"][a])
    return out.reshape(S, H * E) @ w["o"].T


def silu(x: Tensor) -> Tensor:
    return x / (1 + torch.exp(-x))


def causal_conv(x: Tensor, w: Tensor, b: Tensor) -> Tensor:
    """Depthwise causal convolution: x [S, ch], w [ch, taps] (last tap = the current token)."""
    S, taps = x.shape[0], w.shape[1]
    y = torch.empty_like(x)
    for t in range(S):
        acc = b.clone()
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                acc = acc + w[:, j] * x[s]
        y[t] = acc
    return y


def gated_group_norm(y: Tensor, z: Tensor, w: Tensor, parts: int, eps: float) -> Tensor:
    """Gate first, then RMS norm of each of `parts` equal slices by itself, then the weight."""
    t = y * silu(z)
    return rms_norm(t.view(t.shape[0], parts, -1), None, eps).reshape(t.shape) * w


def state_space(x: Tensor, B: Tensor, C: Tensor, dt: Tensor, A_log: Tensor, D: Tensor,
                state: Optional[Tensor] = None):
    """The recurrence of all heads: x [S,H,P], B and C [S,G,N], dt [S,H] (after softplus).
    Returns (y [S,H,P], the final state [H,N,P])."""
    S, H, P = x.shape
    G, N = B.shape[1:]
    st = torch.zeros(H, N, P, dtype=x.dtype) if state is None else state.clone()
    y = torch.empty_like(x)
    for t in range(S):
        for a in range(H):
            g = a // (H // G)
            st[a] = torch.exp(-torch.exp(A_log[a]) * dt[t, a]) * st[a] + dt[t, a] * torch.outer(B[t, g], x[t, a])
            y[t, a] = C[t, g] @ st[a] + D[a] * x[t, a]
    return y, st


def softplus(x: Tensor) -> Tensor:
    return torch.log1p(torch.exp(-x.abs())) + x.clamp(min=0)


def mamba2(h: Tensor, w: Dict[str, Tensor], m: dict, eps: float) -> Tensor:
    S, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    I = H * P
    z, xbc, dt = (h @ w["in"].T).split([I, I + 2 * G * N, H], dim=-1)
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = xbc.split([I, G * N, G * N], dim=-1)
    dt = softplus(dt + w["dt_bias"])
    y, _ = state_space(x.reshape(S, H, P), B.reshape(S, G, N), C.reshape(S, G, N), dt, w["A_log"], w["D"])
    return gated_group_norm(y.reshape(S, I), z, w["norm"], m["norm_groups"], eps) @ w["o"].T


def clamped_feed_forward(h: Tensor, w: Dict[str, Tensor], limit: float) -> Tensor:
    g = (h @ w["gate"].T).clamp(max=limit)
    u = (h @ w["up"].T).clamp(-limit, limit)
    return (g / (1 + torch.exp(-1.702 * g)) * (u + 1)) @ w["down"].T


# ------------------------------------------------------------------------------- the whole model
def _sub(w: Dict[str, Tensor], prefix: str) -> Dict[str, Tensor]:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def layer(x: Tensor, w: Dict[str, Tensor], entry: dict, eps: float) -> Tensor:
    m, kind = entry["mixer"], entry["type"]
    h, mw = rms_norm(x, w["norm1"], eps), _sub(w, "mix.")
    if kind == "attention":
        y = chunked_attention(h, mw, m)
    elif kind == "latent_attention":
        y = latent_attention(h, mw, m, eps)
    else:
        y = mamba2(h, mw, m, eps)
    x = x + rms_norm(y, w["norm1b"], eps)
    if entry["mlp"] is not None:
        y = clamped_feed_forward(rms_norm(x, w["norm2"], eps), _sub(w, "mlp."), entry["mlp"]["limit"])
        x = x + rms_norm(y, w["norm2b"], eps)
    return x


def layer_order(cfg: dict) -> List[tuple]:
    """[(layer, pass or None, first layer of a pass)] in the order they run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None, False) for i in range(n)]
    a, b = lp["start"], lp["stop"]
    return ([(i, None, False) for i in range(a)] +
            [(i, t, i == a) for t in range(lp["times"]) for i in range(a, b)] +
            [(i, None, False) for i in range(b, n)])


def forward(tokens: List[int], weights: Dict[str, Tensor], cfg: dict, dtype=torch.float64,
            residuals: Optional[list] = None) -> Tensor:
    """Logits [S, vocab] of one sequence; `residuals` collects the residual stream after every layer run."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    x = x0
    for i, t, first in layer_order(cfg):
        if first:
            x = torch.cat([x, x0], -1) @ w["loop.in"].T + w["loop.step"][t]
        x = layer(x, _sub(w, f"l{i}."), cfg["layers"][i], eps)
        if residuals is not None:
            residuals.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def tensor_shapes(cfg: dict, bias_rows: int = 16) -> Dict[str, tuple]:
    """Checkpoint names and shapes of a configuration."""
    V, W = cfg["vocab"], cfg["width"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    if cfg.get("loop"):
        out["loop.in"], out["loop.step"] = (W, 2 * W), (cfg["loop"]["times"], W)
    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}."
        H = m["heads"]
        out[p + "norm1"] = out[p + "norm1b"] = (W,)
        if e["type"] == "attention":
            mix = {"q": (H * m["dim"], W), "k": (m["kv_heads"] * m["dim"], W), "v": (m["kv_heads"] * m["vdim"], W),
                   "rel": (bias_rows, H), "o": (W, H * m["vdim"])}
        elif e["type"] == "latent_attention":
            K, R = m["kv_rank"], m["rot_dim"]
            mix = {"q": (H * (m["dim"] + R), W), "dkv": (K + R, W), "dkv.norm": (K,), "uk": (H * m["dim"], K),
                   "uv": (H * m["vdim"], K), "sink": (H,), "o": (W, H * m["vdim"])}
        else:
            I, ch = H * m["vdim"], H * m["vdim"] + 2 * m["groups"] * m["state"]
            mix = {"in": (I + ch + H, W), "conv": (ch, m["conv"]), "conv.b": (ch,), "dt_bias": (H,), "A_log": (H,),
                   "D": (H,), "norm": (I,), "o": (W, I)}
        out.update({p + "mix." + k: v for k, v in mix.items()})
        if e["mlp"] is not None:
            F = e["mlp"]["ff"]
            out[p + "norm2"] = out[p + "norm2b"] = (W,)
            out.update({p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
    return out


def random_weights(cfg: dict, seed: int, bias_rows: int = 16) -> Dict[str, Tensor]:
    """bfloat16 weights at which every mechanism shows: attention scores of a few units, biases and sinks
    that matter, decays from slow to fast, norm weights away from one."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, bias_rows).items():
        leaf = name.split(".", 2)[-1] if name.startswith("l") and name[1].isdigit() else name
        x = torch.randn(*shape, generator=g)
        if leaf.endswith("norm") or leaf in ("norm1", "norm1b", "norm2", "norm2b"):
            x = 1.0 + 0.3 * x
        elif leaf in ("mix.q", "mix.k", "mix.dkv", "mix.uk"):
            x = x * 1.6 / shape[-1] ** 0.5
        elif leaf in ("mix.rel", "mix.sink"):
            x = 1.5 * x
        elif leaf == "mix.A_log":
            x = 0.5 * x - 0.5
        elif leaf == "mix.dt_bias":
            x = x - 2.0
        elif leaf in ("mix.D", "mix.conv.b", "embed", "loop.step"):
            x = 0.5 * x
        elif leaf == "mix.conv":
            x = x / shape[-1] ** 0.5
        else:
            x = x / shape[-1] ** 0.5
        out[name] = x.to(torch.bfloat16)
    return out
