"""Plain restatement of the Timalorn decoder, one function per mechanism, written for reading: one
sequence at a time, explicit loops over positions and heads, no cache, any float dtype (float64 by
default).  Test infrastructure: shares no code with `socket_b200`.

Weights are a dict name -> tensor in the checkpoint's naming; `cfg` is the parsed config.json.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Tensor = torch.Tensor


# ------------------------------------------------------------------------------- mechanisms
def layer_norm(x: Tensor, w: Tensor, eps: float) -> Tensor:
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms_unit(x: Tensor, eps: float) -> Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rotary_frequencies(dims: int, base: float, scaling: Optional[dict]) -> List[float]:
    """One angle per position for every pair; with `scaling` slow pairs turn `factor` times slower and the
    pairs between the two turning counts are blended."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return f

    def pair_that_turns(times: float) -> float:             # index of the pair that turns so often in `original` tokens
        return dims * math.log(scaling["original"] / (2 * math.pi * times)) / (2 * math.log(base))

    lo = max(math.floor(pair_that_turns(scaling["fast"])), 0)
    hi = min(math.ceil(pair_that_turns(scaling["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / scaling["factor"] * ramp + x * (1 - ramp))
    return out


def rotary_gain(scaling: Optional[dict]) -> float:
    return 1.0 if scaling is None else 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_halves(x: Tensor, pos: int, rot: dict) -> Tensor:
    """Turn the first rot.dims elements of a vector: element i goes with element i + dims / 2."""
    half = rot["dims"] // 2
    gain = rotary_gain(rot.get("scaling"))
    y = x.clone()
    for i, f in enumerate(rotary_frequencies(rot["dims"], rot["base"], rot.get("scaling"))):
        c, s = math.cos(pos * f) * gain, math.sin(pos * f) * gain
        u, v = x[i], x[i + half]
        y[i] = u * c - v * s
        y[i + half] = v * c + u * s
    return y


def soft_cap(s: Tensor, cap: float) -> Tensor:
    return cap * torch.tanh(s / cap)


def attend(scores: Tensor, values: Tensor, sink: Optional[Tensor] = None) -> Tensor:
    """One query: exp(score) weights of the rows of `values`; exp(sink) stands in the denominator only."""
    top = scores.max() if sink is None else torch.maximum(scores.max(), sink)
    e = torch.exp(scores - top)
    den = e.sum() if sink is None else e.sum() + torch.exp(sink - top)
    return (e / den) @ values


def window_attention(h: Tensor, w: Dict[str, Tensor], m: dict) -> Tensor:
    """Grouped-query attention over the last mask.size positions; the unrotated keys are the values."""
    S, H, G, D, W = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["mask"]["size"]
    q, k = (h @ w["q"].T).view(S, H, D), (h @ w["k"].T).view(S, G, D)
    kr = torch.stack([torch.stack([rotate_halves(k[j, g], j, m["rot"]) for g in range(G)]) for j in range(S)])
    out = torch.empty(S, H, D, dtype=h.dtype)
    for i in range(S):
        lo = max(0, i - W + 1)
        for a in range(H):
            g = a // (H // G)
            qi = rotate_halves(q[i, a], i, m["rot"])
            out[i, a] = attend(soft_cap(kr[lo:i + 1, g] @ qi * m["scale"], m["softcap"]), k[lo:i + 1, g], w["sink"][a])
    return out.reshape(S, H * D) @ w["o"].T


def log_sigmoid(x: Tensor) -> Tensor:
    return x.clamp(max=0) - torch.log1p(torch.exp(-x.abs()))


def matrix_memory(q: Tensor, k: Tensor, v: Tensor, log_in: Tensor, log_forget: Tensor, state=None):
    """One head: q, k [S,N], v [S,P], gates [S] -> (outputs [S,P], (S [N,P], n [N], m))."""
    if state is None:
        state = (torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype), torch.zeros(q.shape[1], dtype=q.dtype),
                 torch.zeros((), dtype=q.dtype))
    st, n, m = state
    out = torch.empty_like(v)
    for t in range(q.shape[0]):
        new = torch.maximum(log_forget[t] + m, log_in[t])
        keep, add = torch.exp(log_forget[t] + m - new), torch.exp(log_in[t] - new)
        st = keep * st + add * torch.outer(k[t], v[t])
        n = keep * n + add * k[t]
        m = new
        out[t] = (q[t] @ st) / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6)
    return out, (st, n, m)


def mlstm(h: Tensor, w: Dict[str, Tensor], x: dict, eps: float) -> Tensor:
    S, H, N, P, cap = h.shape[0], x["heads"], x["dim"], x["vdim"], x["gate_cap"]
    q, k, v = (h @ w["q"].T).view(S, H, N) * N ** -0.5, (h @ w["k"].T).view(S, H, N), (h @ w["v"].T).view(S, H, P)
    i = soft_cap(h @ w["i"].T + w["i.b"], cap)
    f = log_sigmoid(soft_cap(h @ w["f"].T + w["f.b"], cap))
    o = torch.stack([matrix_memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a])[0] for a in range(H)], 1)
    o = rms_unit(o, eps).reshape(S, H * P) * w["norm"]
    return (o / (1 + torch.exp(-(h @ w["g"].T)))) @ w["o"].T


def feed_forward(h: Tensor, w: Dict[str, Tensor]) -> Tensor:
    g = h @ w["gate"].T
    return (g / (1 + torch.exp(-g)) * (h @ w["up"].T)) @ w["down"].T


# ------------------------------------------------------------------------------- the whole model
def _sub(w: Dict[str, Tensor], prefix: str) -> Dict[str, Tensor]:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def owner(cfg: dict, i: int) -> int:
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def layer(x: Tensor, w: Dict[str, Tensor], entry: dict, eps: float) -> Tensor:
    h = layer_norm(x, w["norm1"], eps)
    if entry["type"] == "attention":
        y = window_attention(h, _sub(w, "mix."), entry["mixer"])
    else:
        y = mlstm(h, _sub(w, "mix."), entry["mixer"], eps)
    if entry["mlp"] is not None:
        y = y + feed_forward(h, _sub(w, "mlp."))
    return x + y


def forward(tokens: List[int], weights: Dict[str, Tensor], cfg: dict, dtype=torch.float64,
            residuals: Optional[list] = None) -> Tensor:
    """Logits [S, vocab] of one sequence; `residuals` collects the residual stream after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, entry in enumerate(cfg["layers"]):
        x = layer(x, _sub(w, f"l{owner(cfg, i)}."), entry, eps)
        if residuals is not None:
            residuals.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    """Checkpoint names and shapes of a configuration."""
    V, W = cfg["vocab"], cfg["width"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, e in enumerate(cfg["layers"]):
        if e.get("weights_of") is not None:
            continue
        m, p = e["mixer"], f"l{i}."
        H, D = m["heads"], m["dim"]
        out[p + "norm1"] = (W,)
        if e["type"] == "attention":
            mix = {"q": (H * D, W), "k": (m["kv_heads"] * D, W), "sink": (H,), "o": (W, H * D)}
        else:
            P = m["vdim"]
            mix = {"q": (H * D, W), "k": (H * D, W), "v": (H * P, W), "g": (H * P, W), "o": (W, H * P), "norm": (H * P,),
                   "i": (H, W), "i.b": (H,), "f": (H, W), "f.b": (H,)}
        out.update({p + "mix." + k: v for k, v in mix.items()})
        if e["mlp"] is not None:
            F = e["mlp"]["ff"]
            out.update({p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
    return out


def random_weights(cfg: dict, seed: int) -> Dict[str, Tensor]:
    """bfloat16 weights at which every mechanism shows: attention scores of a few units, sinks that matter,
    forget gates from fast to slow, input gates that move the running maximum, norm weights away from one."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.split(".", 1)[-1] if name[0] == "l" and name[1].isdigit() else name
        x = torch.randn(*shape, generator=g)
        if leaf.endswith("norm") or leaf == "norm1":
            x = 1.0 + 0.3 * x
        elif leaf in ("mix.q", "mix.k"):
            x = x * 1.6 / shape[-1] ** 0.5
        elif leaf == "mix.sink":
            x = 1.5 * x
        elif leaf in ("mix.i", "mix.f"):
            x = x * 1.5 / shape[-1] ** 0.5
        elif leaf == "mix.f.b":
            x = 2.5 + 1.5 * x
        elif leaf in ("mix.i.b", "embed"):
            x = 0.5 * x
        else:
            x = x / shape[-1] ** 0.5
        out[name] = x.to(torch.bfloat16)
    # a query almost orthogonal to the only key of a memory (the first token's, say) has an output whose sign is
    # rounding's; keys that lean towards their queries keep outputs well-conditioned
    for i, e in enumerate(cfg["layers"]):
        if e["type"] == "mlstm" and e.get("weights_of") is None:
            k = out[f"l{i}.mix.k"].float() + out[f"l{i}.mix.q"].float()
            out[f"l{i}.mix.k"] = (k / 2 ** 0.5).to(torch.bfloat16)
    return out
