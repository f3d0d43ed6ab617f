"""The mechanisms Timalorn brought to the building-block library, each alone, against the plain implementation
in float64."""
import math

import pytest
import torch

from oracle import timalorn_oracle as orc
from socket_b200 import block_ops as ops
from socket_b200.mixers import YarnScaling, rotary_angles

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F32, BF16 = torch.float32, torch.bfloat16
D64 = torch.float64


def _rand(*shape, seed=0, dtype=F32, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def _close(got, want, dtype, tol16=1.5e-2, tol32=2e-5):
    """Largest error against the largest entry."""
    got, want = got.detach().cpu().to(D64), want.to(D64)
    assert got.shape == want.shape and torch.isfinite(got).all()
    err, top = (got - want).abs().max().item(), want.abs().max().item()
    assert err <= (tol16 if dtype == BF16 else tol32) * max(top, 1e-3), (err, top)


# ------------------------------------------------------------------------------- residual stream, gated unit
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,width", [(1, 4096), (3, 54), (400, 80), (5, 8192), (7, 129)])
def test_added_sublayer_and_layer_norm(rows, width, dtype):
    eps = 1e-3
    x, y, w = _rand(rows, width, seed=1) + 3.0, _rand(rows, width, seed=3, dtype=F32), _rand(width, seed=5, dtype=dtype)
    added = x.to(D64) + y.to(D64)
    xg = x.to(DEV)
    out = ops.residual_norm(xg, eps, y=y.to(DEV), w_out=w.to(DEV), centred=True)
    assert out.dtype == dtype and xg.dtype == F32
    _close(xg, added, F32)
    _close(out, orc.layer_norm(added, w.to(D64), eps), dtype)
    xg = x.to(DEV)
    _close(ops.residual_norm(xg, eps, w_out=w.to(DEV), centred=True), orc.layer_norm(x.to(D64), w.to(D64), eps), dtype)
    assert torch.equal(xg.cpu(), x)
    y16 = y.to(dtype)
    assert ops.residual_norm(xg, eps, y=y16.to(DEV)) is None            # added and nothing more
    _close(xg, x.to(D64) + y16.to(D64), F32)


def test_layer_norm_of_a_large_mean_and_a_small_spread():
    x = 1000.0 + 1e-2 * _rand(2, 640, seed=1)
    w = torch.ones(640)
    got = ops.residual_norm(x.to(DEV), 1e-5, w_out=w.to(DEV), centred=True)
    _close(got, orc.layer_norm(x.to(D64), w.to(D64), 1e-5), F32, tol32=2e-2)   # the fp32 mean of 1000 +- 3e-5
    x = torch.full((1, 64), 1e-3) * torch.tensor([1.0, -1.0]).repeat(32)
    got = ops.residual_norm(x.to(DEV), 1e-2, w_out=torch.ones(64, device=DEV), centred=True)
    _close(got, orc.layer_norm(x.to(D64), torch.ones(64, dtype=D64), 1e-2), F32)   # eps inside the root


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("ff", [30, 128, 1000])
def test_silu_unit_of_slices(ff, dtype):
    pad = (ff + 7) // 8 * 8
    gu = _rand(37, 2 * pad, seed=1, dtype=dtype, scale=2.0)
    g, u = gu[:, :ff].to(D64), gu[:, pad:pad + ff].to(D64)
    want = g / (1 + torch.exp(-g)) * u
    out = torch.full((37, pad + 16), 7.0, dtype=dtype, device=DEV)
    gg = gu.to(DEV)
    ops.glu_silu(gg[:, :ff], gg[:, pad:pad + ff], out=out[:, 8:8 + ff])
    _close(out[:, 8:8 + ff], want, dtype)
    assert (out[:, :8] == 7).all() and (out[:, 8 + ff:] == 7).all()


# ------------------------------------------------------------------------------- rotary rows
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,dim,rot", [(4, 2, 24, 8), (3, 1, 14, 6), (2, 2, 32, 32), (8, 1, 80, 16), (2, 1, 9, 2), (4, 4, 128, 64)])
def test_rotary_rows(H, G, dim, rot, dtype):
    """Queries and keys against the plain rotation; the earlier rows come out of the ring in their order."""
    B, S, base, ring_rows = 2, 11, 900.0, 7
    s = YarnScaling(3.0, 40, 4.0, 0.7)
    r = {"dims": rot, "base": base, "scaling": dict(factor=3.0, original=40, fast=4.0, slow=0.7)}
    angles = rotary_angles(64, rot, base, DEV, s)
    pq, pk = (H * dim + 7) // 8 * 8, (G * dim + 7) // 8 * 8
    proj = _rand(B * 30, pq + pk + 8, seed=1, dtype=dtype).view(B, 30, -1)
    ring = torch.zeros(B, ring_rows, G, dim + rot, dtype=dtype, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)

    def run(a, b, rows, **kw):
        part = proj[:, a:b].reshape(B * (b - a), -1).to(DEV)
        return ops.rotary_rows(part[:, :H * dim].unflatten(-1, (H, dim)), part[:, pq:pq + G * dim].unflatten(-1, (G, dim)), angles,
                               rot, rows, B=B, S=b - a, status=status, **kw)

    def plain(a, b):
        q = proj[:, a:b, :H * dim].to(D64).view(B, b - a, H, dim).clone()
        k = proj[:, a:b, pq:pq + G * dim].to(D64).view(B, b - a, G, dim)
        rows = torch.empty(B, b - a, G, dim + rot, dtype=D64)
        rows[..., :dim] = k
        for x in range(B):
            for i in range(a, b):
                for h in range(H):
                    y = orc.rotate_halves(q[x, i - a, h], i, r)
                    q[x, i - a, h] = torch.cat([y[rot:], y[:rot]])
                for g in range(G):
                    rows[x, i - a, g, dim:] = orc.rotate_halves(k[x, i - a, g], i, r)[:rot]
        return q, rows

    rows = torch.empty(B, S, G, dim + rot, dtype=dtype, device=DEV)
    q = run(0, S, rows, start=0)
    wq, wr = plain(0, S)
    _close(q, wq, dtype, tol16=4e-3, tol32=3e-6), _close(rows, wr, dtype, tol16=4e-3, tol32=3e-6)
    assert torch.equal(rows[..., :dim].cpu().to(D64), wr[..., :dim])          # values are the keys as projected, exactly
    ops.ring_append(rows, None, ring, None, start=0, keep="window")
    for i in range(S):
        if i >= S - ring_rows:
            assert torch.equal(ring[:, i % ring_rows], rows[:, i])
    for prev in (0, 3, ring_rows):
        more = torch.empty(B, prev + 5, G, dim + rot, dtype=dtype, device=DEV)
        q = run(S, S + 5, more, start=S, ring=ring, prev=prev)
        wq, wr = plain(S, S + 5)
        _close(q, wq, dtype, tol16=4e-3, tol32=3e-6), _close(more[:, prev:], wr, dtype, tol16=4e-3, tol32=3e-6)
        assert torch.equal(more[:, :prev], rows[:, S - prev:S])
    q = run(17, 18, ring, pos=torch.tensor([17], device=DEV))                # one token by a position on the device
    wq, wr = plain(17, 18)
    _close(q, wq, dtype, tol16=4e-3, tol32=3e-6), _close(ring[:, 17 % ring_rows].unsqueeze(1), wr, dtype, tol16=4e-3, tol32=3e-6)
    assert int(status) == 0
    run(0, 1, ring, pos=torch.tensor([64], device=DEV))                      # beyond the angles: reported, not written
    assert int(status) == 1


def test_ring_keeps_the_last_window():
    B, G, D, ring = 2, 1, 8, 10
    for start, S in [(0, 7), (7, 3), (10, 10), (3, 26), (29, 1), (0, 45), (8, 9)]:
        k = _rand(B, S, G, D, seed=S)
        kc = torch.full((B, ring, G, D), 9.0, device=DEV)
        ops.ring_append(k.to(DEV), None, kc, None, start=start, keep="window")
        want = torch.full((B, ring, G, D), 9.0)
        for s in range(max(0, S - ring), S):
            want[:, (start + s) % ring] = k[:, s]
        assert torch.equal(kc.cpu(), want)


# ------------------------------------------------------------------------------- attention
def _plain_attention(q, k, v, scale, start, kv_start, window=0, chunk=0, softcap=0.0, bias=None, sink=None):
    """q [S,H,D], k / v [rows,G,*] in float64; key row r holds position kv_start + r."""
    S, H, _ = q.shape
    G = k.shape[1]
    out = torch.empty(S, H, v.shape[2], dtype=D64)
    for s in range(S):
        i = start + s
        lo = max(kv_start, i - window + 1 if window else 0, i // chunk * chunk if chunk else 0)
        a, b = lo - kv_start, i - kv_start + 1
        for h in range(H):
            g = h // (H // G)
            sc = k[a:b, g] @ q[s, h] * scale
            if softcap:
                sc = orc.soft_cap(sc, softcap)
            if bias is not None:
                sc = sc + bias[h, (i - torch.arange(lo, i + 1)).clamp(max=bias.shape[1] - 1)]
            out[s, h] = orc.attend(sc, v[a:b, g], None if sink is None else sink[h])
    return out


def _needles(q, k, pairs, start, kv_start, gain=7.0):
    """Make the score of (query position i, key position j) stand out, for every head that shares the key."""
    S, H, D = q.shape
    G = k.shape[1]
    for n, (i, j) in enumerate(pairs):
        for g in range(G):
            d = torch.nn.functional.normalize(_rand(D, seed=900 + 10 * n + g), dim=0)
            k[j - kv_start, g] = (d * gain).to(k.dtype)
            for h in range(g * (H // G), (g + 1) * (H // G)):
                q[i - start, h] = (d * gain).to(q.dtype)


ATTN = [
    # queries next to keys just inside and just outside the window (i - j = window - 1, window)
    dict(S=70, H=4, G=2, dqk=24, dv=16, start=0, window=20, softcap=3.0, near=[(39, 20), (58, 38), (69, 69)]),
    dict(S=300, H=2, G=1, dqk=64, dv=64, start=0, window=64, softcap=50.0, sink=True, near=[(63, 0), (64, 0), (200, 137), (255, 191)]),
    dict(S=300, H=2, G=2, dqk=64, dv=80, start=130, kv_start=35, window=96, softcap=2.0, near=[(131, 36), (287, 192), (288, 192)]),
    dict(S=260, H=3, G=3, dqk=80, dv=96, start=0, window=129, softcap=20.0, sink=True, near=[(259, 131), (259, 130), (128, 0), (129, 0)]),
    dict(S=150, H=2, G=2, dqk=192, dv=128, start=333, kv_start=200, window=1000, softcap=9.0, sink=True, near=[(340, 200), (482, 255)]),
    dict(S=129, H=2, G=1, dqk=128, dv=128, start=1, kv_start=0, window=1, near=[(6, 6), (7, 6)]),
    dict(S=2, H=2, G=2, dqk=64, dv=64, start=255, kv_start=192, window=64, softcap=5.0, near=[(255, 192), (256, 192)]),
    dict(S=513, H=1, G=1, dqk=16, dv=8, start=0, window=257, softcap=4.0, near=[(512, 256), (512, 255), (300, 44)]),
    dict(S=200, H=2, G=1, dqk=40, dv=24, start=0, window=30, chunk=64, softcap=7.0, bias=True, sink=True, near=[(130, 128), (127, 98)]),
    dict(S=140, H=2, G=1, dqk=64, dv=64, start=0, window=60, bias=True, near=[(100, 41), (100, 40)]),
]


@pytest.mark.parametrize("case", range(len(ATTN)))
@pytest.mark.parametrize("path", ["rows32", "rows", "prefill_tc"])
def test_window_and_capped_scores_of_a_portion(case, path):
    c = ATTN[case]
    S, H, G, dqk, dv, start = (c[x] for x in ("S", "H", "G", "dqk", "dv", "start"))
    kv_start = c.get("kv_start", 0)
    dtype = F32 if path == "rows32" else BF16
    B, rows = 2, start + S - kv_start
    qs, ks, vs = [], [], []
    for b in range(B):
        q, k, v = _rand(S, H, dqk, seed=b + 1), _rand(rows, G, dqk, seed=b + 11), _rand(rows, G, dv, seed=b + 21)
        _needles(q, k, c["near"], start, kv_start)
        qs.append(q), ks.append(k), vs.append(v)
    q, k, v = (torch.stack(t).to(dtype).to(DEV) for t in (qs, ks, vs))
    bias = _rand(H, 41, seed=5, scale=2.0) if c.get("bias") else None
    sink = _rand(H, seed=6, scale=2.0) + 2.0 if c.get("sink") else None
    kw = dict(window=c["window"], chunk=c.get("chunk", 0), softcap=c.get("softcap", 0.0))
    scale = 1.0 / math.sqrt(dqk)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.full((B * S, H * dv + 8), 7.0, dtype=dtype, device=DEV)      # results may be a slice of wider rows
    ops.attn(q, k, v, out=out[:, :H * dv].view(B, S, H, dv), scale=scale, start=start, kv_start=kv_start, status=status,
             bias=None if bias is None else bias.to(DEV), sink=None if sink is None else sink.to(DEV),
             path="rows" if path == "rows32" else path, **kw)
    assert int(status) == 0 and (out[:, H * dv:] == 7).all()
    for b in range(B):
        want = _plain_attention(q[b].cpu().to(D64), k[b].cpu().to(D64), v[b].cpu().to(D64), scale, start, kv_start,
                                bias=None if bias is None else bias.to(D64), sink=None if sink is None else sink.to(D64), **kw)
        _close(out.view(B, S, -1)[b, :, :H * dv].unflatten(-1, (H, dv)), want, dtype)


@pytest.mark.parametrize("path", ["rows32", "rows", "prefill_tc", "decode"])
@pytest.mark.parametrize("size", [0.05, 1.0, 30.0])
@pytest.mark.parametrize("cap", [10.0, 80.0])
def test_score_cap_of_small_and_of_saturated_scores(cap, size, path):
    """Scores far below the cap (a polynomial in the tensor-core kernel), near it and far beyond it, for a cap whose
    exponentials need no running maximum and for one whose do."""
    S, H, D = 130, 1, 32
    dtype = F32 if path == "rows32" else BF16
    S = 1 if path == "decode" else S
    k, v = _rand(130, 1, D, seed=1, dtype=dtype), _rand(130, 1, D, seed=2, dtype=dtype)
    q = _rand(S, H, D, seed=3, dtype=dtype)
    kw = dict(scale=size * cap / D ** 0.5 / 2, softcap=cap, start=130 - S)
    for sink in (None, -60.0, cap - 1.0, 95.0):
        s = None if sink is None else torch.full((1,), sink)
        got = ops.attn(q[None].to(DEV), k[None].to(DEV), v[None].to(DEV), path="rows" if path == "rows32" else path,
                       sink=None if s is None else s.to(DEV), **kw)
        want = _plain_attention(q.to(D64), k.to(D64), v.to(D64), kw["scale"], kw["start"], 0, softcap=cap,
                                sink=None if s is None else s.to(D64))
        _close(got[0], want, dtype, tol16=8e-3, tol32=4e-5)


DECODE = [
    # H, G, dim, rot (keys and values share their rows), window = ring, position, softcap
    dict(H=8, G=2, dim=64, rot=16, window=96, pos=95), dict(H=8, G=2, dim=64, rot=16, window=96, pos=96),
    dict(H=8, G=2, dim=64, rot=16, window=96, pos=1000), dict(H=4, G=1, dim=80, rot=32, window=130, pos=129 + 130),
    dict(H=6, G=3, dim=128, rot=128, window=700, pos=2000), dict(H=3, G=1, dim=56, rot=8, window=1, pos=5),
    dict(H=5, G=1, dim=40, rot=24, window=64, pos=0), dict(H=24, G=1, dim=128, rot=64, window=300, pos=299),
    dict(H=20, G=1, dim=56, rot=8, window=65, pos=400), dict(H=2, G=2, dim=200, rot=40, window=90, pos=77),
]


@pytest.mark.parametrize("case", range(len(DECODE)))
@pytest.mark.parametrize("path", ["rows32", "rows", "decode"])
def test_attention_over_a_window_ring(case, path):
    """One token, position on the device, keys and values slices of the same ring rows: the oldest position that
    the window still holds, the newest, and the one that has just left it made to stand out."""
    c = DECODE[case]
    H, G, dim, rot, W, pos = c["H"], c["G"], c["dim"], c["rot"], c["window"], c["pos"]
    dtype = F32 if path == "rows32" else BF16
    B, n = 2, pos + 1
    hist = torch.stack([_rand(n, G, dim + rot, seed=b) for b in range(B)])
    q = torch.stack([_rand(1, H, dim, seed=b + 3) for b in range(B)])
    for b in range(B):
        far = [j for j in (max(0, pos - W + 1), pos - W) if j >= 0]
        for j in far:                                                      # both sides of the window's edge
            for g in range(G):
                d = torch.nn.functional.normalize(_rand(dim, seed=77 + g), dim=0) * 5
                hist[b, j, g, rot:] = d
                q[b, 0, g * (H // G):(g + 1) * (H // G)] = d
    ring = torch.zeros(B, W, G, dim + rot, dtype=dtype, device=DEV)
    if n < W:
        ring[:, n:] = 30.0                                                 # rows nobody may look at
    ops.ring_append(hist.to(dtype).to(DEV), None, ring, None, start=0, keep="window")
    sink = _rand(H, seed=6, scale=2.0) + 1.0
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    scale = dim ** -0.5
    got = ops.attn(q.to(dtype).to(DEV), ring[..., rot:], ring[..., :dim], pos=torch.tensor([pos], device=DEV), ring=True, window=W,
                   softcap=12.0, scale=scale, sink=sink.to(DEV), status=status, path="rows" if path == "rows32" else path)
    assert int(status) == 0
    hist, q = hist.to(dtype).to(D64), q.to(dtype).to(D64)
    for b in range(B):
        want = _plain_attention(q[b], hist[b, ..., rot:], hist[b, ..., :dim], scale, pos, 0, window=W, softcap=12.0, sink=sink.to(D64))
        _close(got[b], want, dtype)


@pytest.mark.parametrize("S", [2, 9, 32])
def test_short_portions_of_one_key_head(S):
    """A few tokens at once through the split decode kernel, under a window, in order (no ring)."""
    H, dim, rot, W, start, prev = 6, 80, 16, 50, 200, 49
    rows = _rand(1, prev + S, 1, dim + rot, seed=1)
    q = _rand(1, S, H, dim, seed=2)
    _needles(q[0], rows[0, ..., rot:], [(start, start - 49), (start + S - 1, start + S - 50)], start, start - prev, gain=5.0)
    args = (q.to(BF16).to(DEV), rows.to(BF16).to(DEV)[..., rot:], rows.to(BF16).to(DEV)[..., :dim])
    r16 = rows.to(BF16).to(DEV)
    args = (q.to(BF16).to(DEV), r16[..., rot:], r16[..., :dim])
    kw = dict(scale=0.12, start=start, kv_start=start - prev, window=W, softcap=8.0)
    want = _plain_attention(q[0].to(BF16).to(D64), rows[0, ..., rot:].to(BF16).to(D64), rows[0, ..., :dim].to(BF16).to(D64), 0.12, start,
                            start - prev, window=W, softcap=8.0)
    for path in ("decode", "prefill_tc", "auto"):
        _close(ops.attn(*args, path=path, **kw)[0], want, BF16)


def test_the_fast_kernels_are_the_ones_that_run():
    import ctypes

    from socket_b200._lib import blocks
    z = lambda *s: torch.zeros(*s, dtype=BF16, device=DEV)  # noqa: E731
    rows, ring = z(1, 900, 2, 128 + 64), z(2, 96, 2, 64 + 16)
    for q, k, v, kw, want in [(z(1, 300, 4, 128), rows[..., 64:], rows[..., :128], dict(start=600, window=500), "prefill_tc"),
                              (z(2, 1, 8, 64), ring[..., 16:], ring[..., :64], dict(ring=True, window=96), "decode")]:
        p = ops.attn_params(q, k, v, z(*q.shape[:3], v.shape[3]), scale=1.0, softcap=30.0, **kw)
        assert blocks().skb_attn_path(ctypes.byref(p)) == ops.ATTN_PATHS[want]


def test_a_ring_smaller_than_its_window_is_refused():
    z = lambda *s: torch.zeros(*s, device=DEV)  # noqa: E731
    with pytest.raises(RuntimeError, match="ring"):
        ops.attn(z(1, 1, 2, 8), z(1, 20, 1, 8), z(1, 20, 1, 8), scale=1.0, ring=True, window=19)


# ------------------------------------------------------------------------------- matrix memory
MEM = [dict(H=3, N=16, P=24, cap=4.0), dict(H=2, N=128, P=64, cap=15.0), dict(H=2, N=136, P=96, cap=8.0), dict(H=3, N=13, P=11, cap=2.0),
       dict(H=1, N=256, P=40, cap=15.0), dict(H=35, N=8, P=8, cap=6.0)]


def _memory_inputs(c, B, S, dtype, seed=0, spread=2.0):
    H, N, P = c["H"], c["N"], c["P"]
    pad = lambda n: (n + 7) // 8 * 8  # noqa: E731
    sizes = [H * N, H * N, H * P, H * P]
    at = [sum(map(pad, sizes[:i])) for i in range(4)]
    proj = _rand(B * S, sum(map(pad, sizes)), seed=seed, dtype=dtype)
    gates = _rand(B * S, pad(2 * H), seed=seed + 1, scale=spread)
    bias = [_rand(H, seed=seed + 2), 2.0 + _rand(H, seed=seed + 3)]
    norm = (1 + 0.3 * _rand(H * P, seed=seed + 4)).to(dtype)
    return proj, [slice(a, a + n) for a, n in zip(at, sizes)], gates, bias, norm


def _plain_memory(c, proj, cols, gates, bias, norm, B, S, eps, dtype=D64):
    H, N, P, cap = c["H"], c["N"], c["P"], c["cap"]
    out, states = torch.empty(B * S, H * P, dtype=dtype), []
    for b in range(B):
        r = proj[b * S:(b + 1) * S].to(dtype)
        q, k, v, z = (r[:, s] for s in cols)
        g = gates[b * S:(b + 1) * S].to(dtype)
        i = orc.soft_cap(g[:, :H] + bias[0].to(dtype), cap)
        f = orc.log_sigmoid(orc.soft_cap(g[:, H:2 * H] + bias[1].to(dtype), cap))
        for h in range(H):
            o, st = orc.matrix_memory(q[:, h * N:(h + 1) * N] * N ** -0.5, k[:, h * N:(h + 1) * N], v[:, h * P:(h + 1) * P], i[:, h], f[:, h])
            s = slice(h * P, (h + 1) * P)
            out[b * S:(b + 1) * S, s] = orc.rms_unit(o, eps) * norm[s].to(dtype) / (1 + torch.exp(-z[:, s]))
            states.append(st)
    return out, [torch.stack([s[j] for s in states]) for j in range(3)]


def _run_memory(c, part, cols, gates, bias, norm, state, n, eps, path, **kw):
    out = torch.full((part.shape[0], norm.numel() + 8), 7.0, dtype=part.dtype, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    ops.mlstm(*(part[:, s] for s in cols), gates, *(b.to(DEV) for b in bias), norm.to(DEV), *state, out[:, 8:], S=n, cap=c["cap"],
              q_scale=c["N"] ** -0.5, eps=eps, path=path, status=status, **kw)
    assert (out[:, :8] == 7).all() and int(status) == 0
    return out[:, 8:]


@pytest.mark.parametrize("case", range(len(MEM)))
@pytest.mark.parametrize("path", ["steps32", "steps", "chunks", "tensor"])
def test_matrix_memory_in_portions(case, path):
    """One long portion, and the same tokens in portions of all kinds of sizes (also single tokens by a position on
    the device): the same outputs, the same final state; dirty state is not seen at position 0."""
    c, B, S, eps = MEM[case], 2, 210, 1e-4
    dtype = F32 if path == "steps32" else BF16
    path = "steps" if path == "steps32" else path
    H, N, P = c["H"], c["N"], c["P"]
    if path in ("chunks", "tensor") and (N % 8 or P % 8):
        pytest.skip("sizes of the step kernel only")
    proj, cols, gates, bias, norm = _memory_inputs(c, B, S, dtype)
    want, want_st = _plain_memory(c, proj, cols, gates, bias, norm, B, S, eps)
    pg, gg = proj.to(DEV).view(B, S, -1), gates.to(DEV).view(B, S, -1)
    for sizes in ([S], [1, 2, 2, 59, 64, 1, 65, 16], [64, 128, 3, 15], [128, 82], [2] * 105):
        state = [torch.full(s, 3.0, device=DEV) for s in ((B, H, N, P), (B, H, N), (B, H))]
        out, at = [], 0
        for n in sizes:
            kw = dict(pos=torch.tensor([at], device=DEV)) if n == 1 else dict(start=at)
            y = _run_memory(c, pg[:, at:at + n].reshape(B * n, -1), cols, gg[:, at:at + n].reshape(B * n, -1), bias, norm, state, n, eps,
                            "steps" if n == 1 else path, **kw)
            out.append(y.view(B, n, H * P))
            at += n
        _close(torch.cat(out, 1).reshape(B * S, -1), want, dtype)
        # the state against the plain one, in units of its own stabiliser
        for got, w in zip(state, want_st):
            _close(got.view(w.shape), w, dtype, tol16=1e-4, tol32=1e-5)


@pytest.mark.parametrize("form", ["chunks", "tensor"])
def test_block_forms_keep_more_than_bf16(form):
    """With the same bf16 inputs the block forms and the token-by-token fp32 form differ by far less than the
    output's own rounding; a slowly forgetting head over a long portion included."""
    c, B, S, eps = dict(H=2, N=64, P=32, cap=15.0), 1, 1000, 1e-5
    proj, cols, gates, bias, norm = _memory_inputs(c, B, S, BF16, seed=9)
    bias[1] = torch.tensor([12.0, 0.0])
    states, outs = [], []
    for path in ("steps", form):
        st = [torch.zeros(s, device=DEV) for s in ((1, 2, 64, 32), (1, 2, 64), (1, 2))]
        outs.append(_run_memory(c, proj.to(DEV), cols, gates.to(DEV), bias, norm, st, S, eps, path).float())
        states.append(st)
    for a, b in zip(*states):
        assert (a - b).abs().max() <= 3e-5 * a.abs().max()
    assert (outs[0] - outs[1]).abs().max() <= 1e-2 * outs[0].abs().max()


@pytest.mark.parametrize("path", ["steps32", "chunks", "tensor"])
def test_gates_at_their_extremes(path):
    """The running maximum: a strong input gate long ago that fades slowly, gates closed from the start (m stays at
    or below zero and the floor exp(-m) rules), a jump inside a block, values of the floor and of |n . q| both
    deciding.  With one token ruling a memory, outputs where q is almost orthogonal to its key are ill-conditioned;
    the plain implementation's own error in fp32 says how much."""
    dtype = F32 if path == "steps32" else BF16
    c, B, S, eps = dict(H=4, N=16, P=16, cap=12.0), 1, 200, 1e-6
    proj, cols, gates, bias, norm = _memory_inputs(c, B, S, dtype, seed=3, spread=0.5)
    bias = [torch.zeros(4), torch.zeros(4)]
    g = gates.view(S, -1)
    g[:, 0], g[:, 4] = -11.0, 9.0                        # closed input, open forget
    g[3, 0] = 11.0
    g[:, 1], g[:, 5] = -30.0, -30.0                      # closed, forgetting: both gates at their caps
    g[:, 2], g[:, 6] = -4.0, 6.0
    g[70:75, 2] = 30.0                                   # a jump inside the second block
    g[:, 3], g[:, 7] = 30.0, 30.0                        # everything kept at full strength
    want, want_st = _plain_memory(c, proj, cols, g, bias, norm, B, S, eps)
    out32, st32 = _plain_memory(c, proj, cols, g, bias, norm, B, S, eps, F32)
    rounding, st_rounding = (out32.to(D64) - want).abs(), [float((a.to(D64) - b).abs().max()) for a, b in zip(st32, want_st)]
    for sizes in ([S], [71, 2, 127]):
        state = [torch.zeros(s, device=DEV) for s in ((B, 4, 16, 16), (B, 4, 16), (B, 4))]
        out, at = [], 0
        for n in sizes:
            out.append(_run_memory(c, proj[at:at + n].to(DEV), cols, g[at:at + n].to(DEV), bias, norm, state, n, eps,
                                   "steps" if path == "steps32" else path, start=at))
            at += n
        got = torch.cat(out)
        for h in range(4):                               # head by head: their sizes differ
            s = slice(16 * h, 16 * h + 16)
            err, top = (got[:, s].cpu().to(D64) - want[:, s]).abs(), float(want[:, s].abs().max())
            limit = (1.5e-2 if dtype == BF16 else 2e-5) * top
            assert err.max() <= limit + 4 * rounding[:, s].max() and err.median() <= limit, (h, float(err.max()), top)
        for a, b, r in zip(state, want_st, st_rounding):
            assert (a.cpu().to(D64).view(b.shape) - b).abs().max() <= (1e-4 if dtype == BF16 else 1e-5) * b.abs().max() + 4 * r


@pytest.mark.parametrize("S", [255, 256, 700])
def test_long_portions_take_the_tensor_form_and_go_on_from_any_state(S):
    import ctypes

    from socket_b200 import _lib
    from socket_b200._lib import blocks
    c, B, eps = dict(H=3, N=72, P=136, cap=10.0), 2, 1e-5
    p = _lib.MlstmParams()
    p.dtype, p.B, p.S, p.H, p.N, p.P, p.in_ld = _lib.SK_BF16, B, S, 3, 72, 136, 2 * 3 * (72 + 136)
    assert blocks().skb_mlstm_path(ctypes.byref(p)) == ops.SSM_PATHS["tensor" if S >= 256 else "chunks"]
    proj, cols, gates, bias, norm = _memory_inputs(c, B, S + 40, BF16, seed=6)
    want, want_st = _plain_memory(c, proj, cols, gates, bias, norm, B, S + 40, eps)
    state = [torch.full(s, -2.0, device=DEV) for s in ((B, 3, 72, 136), (B, 3, 72), (B, 3))]
    pg, gg = proj.to(DEV).view(B, S + 40, -1), gates.to(DEV).view(B, S + 40, -1)
    out = []
    for a, b in ((0, 30), (30, S + 30), (S + 30, S + 40)):
        y = _run_memory(c, pg[:, a:b].reshape(B * (b - a), -1), cols, gg[:, a:b].reshape(B * (b - a), -1), bias, norm, state, b - a, eps,
                        "auto", start=a)
        out.append(y.view(B, b - a, -1))
    _close(torch.cat(out, 1).reshape(want.shape), want, BF16)
    for got, w in zip(state, want_st):
        _close(got.view(w.shape), w, BF16, tol16=1e-4)


def test_a_memory_larger_than_the_block_form_takes():
    c, B, S, eps = dict(H=1, N=320, P=48, cap=10.0), 1, 40, 1e-5
    proj, cols, gates, bias, norm = _memory_inputs(c, B, S, BF16, seed=4)
    want, _ = _plain_memory(c, proj, cols, gates, bias, norm, B, S, eps)
    st = [torch.zeros(s, device=DEV) for s in ((1, 1, 320, 48), (1, 1, 320), (1, 1))]
    _close(_run_memory(c, proj.to(DEV), cols, gates.to(DEV), bias, norm, st, S, eps, "auto"), want, BF16)
