"""Every kernel of the building-block library alone, against the plain implementation in float64."""
import math

import pytest
import torch

from oracle import radapel_oracle as orc
from socket_b200 import block_ops as ops
from socket_b200.mixers import distance_buckets, rotary_angles

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
    assert torch.isfinite(got).all()
    err, top = (got - want).abs().max().item(), want.abs().max().item()
    assert err <= (tol16 if dtype == BF16 else tol32) * max(top, 1e-3), (err, top)


# ------------------------------------------------------------------------------- residual stream
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,width", [(1, 4096), (3, 54), (400, 80), (2, 5000), (5, 8192), (7, 129)])
def test_residual_norm(rows, width, dtype):
    eps = 1e-3
    x, x0, y = _rand(rows, width, seed=1), _rand(rows, width, seed=2), _rand(rows, width, seed=3, dtype=dtype, scale=0.05)
    wi, wo = _rand(width, seed=4, dtype=dtype), _rand(width, seed=5, dtype=dtype)
    yd, wid, wod = y.to(D64), wi.to(D64), wo.to(D64)
    added = x.to(D64) + orc.rms_norm(yd, wid, eps)
    xg = x.to(DEV)
    out = ops.residual_norm(xg, eps, y=y.to(DEV), w_in=wi.to(DEV), w_out=wo.to(DEV))
    assert out.dtype == dtype and xg.dtype == F32
    _close(xg, added, F32)                                    # the stream itself is fp32 in both
    _close(out, orc.rms_norm(added, wod, eps), dtype)
    xg = x.to(DEV)                                            # replaced by an fp32 projection + vector, strided rows
    wide = torch.zeros(rows, width + 8, device=DEV)
    wide[:, :width] = y.to(DEV).float()
    out = ops.residual_norm(xg, eps, y=wide[:, :width], w_in=wi.to(DEV), replace=True, w_out=wo.to(DEV))
    _close(xg, yd + wid, F32)
    _close(out, orc.rms_norm(yd + wid, wod, eps), dtype)
    xg = x.to(DEV)
    out = ops.residual_norm(xg, eps, y=y.to(DEV), w_in=wi.to(DEV), x0=x0.to(DEV), dtype=dtype)
    _close(out, torch.cat([added, x0.to(D64)], -1), dtype)
    xg = x.to(DEV)
    assert ops.residual_norm(xg, eps, y=y.to(DEV), w_in=wi.to(DEV)) is None
    _close(xg, added, F32)
    xg = x.to(DEV)
    _close(ops.residual_norm(xg, eps, w_out=wo.to(DEV)), orc.rms_norm(x.to(D64), wod, eps), dtype)
    assert torch.equal(xg.cpu(), x)


def test_residual_norm_keeps_eps_inside_the_root():
    x = torch.full((1, 64), 1e-3)
    w = torch.ones(64)
    got = ops.residual_norm(x.to(DEV), 1e-2, w_out=w.to(DEV))
    _close(got, orc.rms_norm(x.to(D64), w.to(D64), 1e-2), F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_embedding_rows(dtype):
    table = _rand(50, 72, dtype=dtype)
    tok = torch.tensor([[3, 49, 0], [7, 7, 21]])
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    x, x0 = ops.embed_rows(tok.to(DEV), table.to(DEV), 2.5, keep_copy=True, status=status)
    want = table.float()[tok.view(-1)] * 2.5
    assert torch.equal(x.cpu(), want) and torch.equal(x0.cpu(), want) and int(status) == 0
    x, _ = ops.embed_rows(torch.tensor([50, 1], device=DEV), table.to(DEV), 1.0, status=status)
    assert int(status) == 2 and (x[0] == 0).all() and torch.equal(x[1].cpu(), table.float()[1])


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("ff", [30, 128, 1000])
def test_clamped_unit(ff, dtype):
    limit = 0.9
    gu = _rand(37, 2 * ff + 4, seed=1, dtype=dtype, scale=2.0)
    g, u = gu[:, :ff].to(D64).clamp(max=limit), gu[:, ff:2 * ff].to(D64).clamp(-limit, limit)
    want = g / (1 + torch.exp(-1.702 * g)) * (u + 1)
    _close(ops.glu_clamped(gu.to(DEV), ff, limit), want, dtype)
    assert (g == limit).any() and (u == limit).any() and (u == -limit).any() and (g < -limit).any()


# ------------------------------------------------------------------------------- attention
def _plain_attention(q, k, v, scale, start, kv_start, chunk=0, bias=None, sink=None):
    """q [S,H,D], k / v [rows,G,*] in float64; key row r holds position kv_start + r."""
    S, H, _ = q.shape
    G = k.shape[1]
    out = torch.empty(S, H, v.shape[2], dtype=D64)
    for s in range(S):
        i = start + s
        lo = max(kv_start, i // chunk * chunk if chunk else 0)
        a, b = lo - kv_start, i - kv_start + 1
        for h in range(H):
            g = h // (H // G)
            sc = k[a:b, g] @ q[s, h] * scale
            if bias is not None:
                n = (i - torch.arange(lo, i + 1)).clamp(max=bias.shape[1] - 1)
                sc = sc + bias[h, n]
            out[s, h] = orc.softmax_attend(sc, v[a:b, g], None if sink is None else sink[h])
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
    # S, H, G, dqk, dv, start, kv_start, chunk, bias, sink, needles (query, key)
    dict(S=70, H=4, G=2, dqk=24, dv=16, start=0, chunk=20, bias=True, near=[(39, 20), (59, 40), (69, 60)]),
    dict(S=300, H=2, G=1, dqk=64, dv=64, start=0, chunk=64, bias=True, near=[(63, 0), (127, 64), (255, 192), (256, 256)]),
    dict(S=300, H=2, G=2, dqk=64, dv=80, start=130, kv_start=96, chunk=96, bias=True, near=[(191, 96), (287, 192), (192, 192)]),
    dict(S=260, H=3, G=3, dqk=80, dv=96, start=0, sink=True, near=[(259, 0), (128, 1), (127, 0), (256, 128)]),
    dict(S=150, H=2, G=2, dqk=192, dv=128, start=333, sink=True, near=[(340, 0), (482, 127), (400, 128), (355, 355)]),
    dict(S=129, H=2, G=1, dqk=256, dv=128, start=7, near=[(100, 3)]),
    dict(S=33, H=2, G=1, dqk=40, dv=24, start=500, kv_start=480, chunk=240, bias=True, sink=True, near=[(510, 480)]),
    dict(S=2, H=2, G=2, dqk=64, dv=64, start=255, kv_start=192, chunk=64, bias=True, near=[(255, 192)]),
    dict(S=513, H=1, G=1, dqk=16, dv=8, start=0, chunk=1000, near=[(512, 0), (300, 44)]),
    dict(S=257, H=2, G=1, dqk=128, dv=128, start=1, kv_start=0, chunk=7, bias=True, near=[(6, 0), (7, 7), (13, 7)]),
]


@pytest.mark.parametrize("case", range(len(ATTN)))
@pytest.mark.parametrize("path", ["rows32", "rows", "prefill_tc"])
def test_attention_of_a_portion(case, path):
    c = ATTN[case]
    S, H, G, dqk, dv, start = (c[x] for x in ("S", "H", "G", "dqk", "dv", "start"))
    kv_start, chunk = c.get("kv_start", 0), c.get("chunk", 0)
    dtype = F32 if path == "rows32" else BF16
    B, rows = 2, start + S - kv_start
    qs, ks, vs = [], [], []
    for b in range(B):
        q, k, v = _rand(S, H, dqk, seed=b + 1), _rand(rows, G, dqk, seed=b + 11), _rand(rows, G, dv, seed=b + 21)
        _needles(q, k, c["near"], start, kv_start)
        qs.append(q), ks.append(k), vs.append(v)
    # rows wider than the heads, as slices of a fused projection are
    pad = lambda t: torch.cat([t.flatten(2), torch.full((*t.shape[:2], 8), 7.0)], -1)  # noqa: E731
    q, k, v = (pad(torch.stack(t)).to(dtype).to(DEV)[..., :-8].unflatten(-1, (n, d))
               for t, n, d in ((qs, H, dqk), (ks, G, dqk), (vs, G, dv)))
    bias = _rand(H, 61, seed=5, scale=2.0) if c.get("bias") else None
    sink = _rand(H, seed=6, scale=2.0) + 2.0 if c.get("sink") else None
    scale = 1.0 / math.sqrt(dqk)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    got = ops.attn(q, k, v, scale=scale, start=start, kv_start=kv_start, chunk=chunk,
                   bias=None if bias is None else bias.to(DEV), sink=None if sink is None else sink.to(DEV), status=status,
                   path="rows" if path == "rows32" else path)
    assert int(status) == 0
    for b in range(B):
        want = _plain_attention(q[b].cpu().to(D64), k[b].cpu().to(D64), v[b].cpu().to(D64), scale, start, kv_start, chunk,
                                None if bias is None else bias.to(D64), None if sink is None else sink.to(D64))
        _close(got[b], want, dtype)


DECODE = [
    # H, G, dqk, dv, S, position of the first token, chunk (ring), bias, sink
    dict(H=8, G=2, dqk=64, dv=64, pos=63, chunk=64, bias=True), dict(H=8, G=2, dqk=64, dv=64, pos=64, chunk=64, bias=True),
    dict(H=3, G=3, dqk=128, dv=80, pos=700, chunk=512, bias=True), dict(H=16, G=1, dqk=104, dv=72, pos=1500, sink=True),
    dict(H=32, G=1, dqk=576, dv=512, pos=777, sink=True), dict(H=5, G=1, dqk=40, dv=24, pos=0, sink=True),
    dict(H=6, G=1, dqk=136, dv=96, pos=129, S=9, sink=True), dict(H=20, G=1, dqk=328, dv=256, pos=64, S=3, sink=True),
    dict(H=32, G=1, dqk=576, dv=512, pos=0, S=32, sink=True),
]


@pytest.mark.parametrize("case", range(len(DECODE)))
@pytest.mark.parametrize("path", ["rows32", "rows", "decode"])
def test_attention_of_decoded_tokens(case, path):
    """Position on the device, more cache rows than the sequence has; values a prefix of the key rows where
    there is one key head."""
    c = DECODE[case]
    H, G, dqk, dv, pos, S = c["H"], c["G"], c["dqk"], c["dv"], c["pos"], c.get("S", 1)
    chunk = c.get("chunk", 0)
    dtype = F32 if path == "rows32" else BF16
    lo = pos // chunk * chunk if chunk else 0
    live, rows, B = pos + S - lo, (chunk if chunk else pos + S + 200), 2
    k = torch.stack([_rand(rows, G, dqk, seed=b) for b in range(B)])
    v = k[..., :dv] if G == 1 and not chunk else torch.stack([_rand(rows, G, dv, seed=b + 7) for b in range(B)])
    q = torch.stack([_rand(S, H, dqk, seed=b + 3) for b in range(B)])
    for b in range(B):
        _needles(q[b], k[b], [(pos, lo), (pos + S - 1, max(lo, pos - 70))], pos, lo, gain=5.0)
    if not (G == 1 and not chunk):
        kg, vg = k.to(dtype).to(DEV), v.to(dtype).to(DEV)
    else:
        kg = k.to(dtype).to(DEV)
        vg = kg[..., :dv]
    kg[:, live:] = 30.0                                        # rows nobody may look at
    if vg.data_ptr() != kg.data_ptr():
        vg[:, live:] = 1e4
    qg = q.to(dtype).to(DEV)
    bias = _rand(H, 61, seed=5, scale=2.0) if c.get("bias") else None
    sink = _rand(H, seed=6, scale=2.0) + 1.0 if c.get("sink") else None
    scale = 1.0 / math.sqrt(dqk)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    args = dict(scale=scale, chunk=chunk, ring=bool(chunk), bias=None if bias is None else bias.to(DEV),
                sink=None if sink is None else sink.to(DEV), status=status, path="rows" if path == "rows32" else path)
    got = ops.attn(qg, kg, vg, pos=torch.tensor([pos], device=DEV), **args)
    assert int(status) == 0
    for b in range(B):
        want = _plain_attention(qg[b].cpu().to(D64), kg[b].cpu().to(D64), vg[b].cpu().to(D64), scale, pos, lo, chunk,
                                None if bias is None else bias.to(D64), None if sink is None else sink.to(D64))
        _close(got[b], want, dtype)
    # a position beyond the cache is reported
    if not chunk:
        ops.attn(qg, kg, vg, pos=torch.tensor([rows], device=DEV), **args)
        assert int(status) == 1


def test_the_fast_attention_kernels_are_the_ones_that_run():
    import ctypes

    from socket_b200._lib import blocks
    z = lambda *s: torch.zeros(*s, dtype=BF16, device=DEV)  # noqa: E731
    rows = z(1, 900, 1, 576)
    for q, k, v, kw, want in [(z(1, 300, 4, 64), z(1, 300, 2, 64), z(1, 300, 2, 64), {}, "prefill_tc"),
                              (z(1, 64, 4, 192), z(1, 900, 4, 192), z(1, 900, 4, 128), dict(start=836), "prefill_tc"),
                              (z(1, 1, 32, 576), rows, rows[..., :512], dict(start=5), "decode"),
                              (z(2, 1, 8, 64), z(2, 64, 2, 64), z(2, 64, 2, 64), dict(ring=True, chunk=64), "decode")]:
        out = z(*q.shape[:3], v.shape[3])
        p = ops.attn_params(q, k, v, out, scale=1.0, **kw)
        assert blocks().skb_attn_path(ctypes.byref(p)) == ops.ATTN_PATHS[want]


def test_ring_append_keeps_the_last_chunk():
    B, G, D, E, ring = 2, 2, 8, 4, 10
    for start, S in [(0, 7), (7, 3), (10, 10), (3, 26), (29, 1), (0, 45)]:
        k, v = _rand(B, S, G, D, seed=S), _rand(B, S, G, E, seed=S + 1)
        kc, vc = torch.full((B, ring, G, D), 9.0, device=DEV), torch.full((B, ring, G, E), 9.0, device=DEV)
        ops.ring_append(k.to(DEV), v.to(DEV), kc, vc, start=start)
        wk, wv = torch.full((B, ring, G, D), 9.0), torch.full((B, ring, G, E), 9.0)
        for s in range(S):
            if (start + s) // ring == (start + S - 1) // ring:
                wk[:, (start + s) % ring], wv[:, (start + s) % ring] = k[:, s], v[:, s]
        assert torch.equal(kc.cpu(), wk) and torch.equal(vc.cpu(), wv)
    kc, vc = torch.zeros(B, ring, G, D, device=DEV), torch.zeros(B, ring, G, E, device=DEV)
    ops.ring_append(k[:, :1].to(DEV), v[:, :1].to(DEV), kc, vc, pos=torch.tensor([37], device=DEV))
    assert torch.equal(kc[:, 7].cpu(), k[:, 0]) and int((kc != 0).any(-1).any(-1).sum()) == B


# ------------------------------------------------------------------------------- latents
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,dim,rot,rot_dims,rank,vdim", [(3, 24, 8, 8, 56, 40), (2, 9, 6, 4, 19, 7), (16, 128, 64, 64, 512, 128)])
def test_latent_rows_queries_and_values(H, dim, rot, rot_dims, rank, vdim, dtype):
    B, S, start, cap, base, eps = 2, 5, 60, 70, 900.0, 1e-4
    ld = (rank + rot + 7) // 8 * 8
    qd = _rand(B * S, H * (dim + rot) + rank + rot + 3, seed=1, dtype=dtype)
    w, angles = 1 + 0.3 * _rand(rank, seed=2), rotary_angles(cap, rot_dims, base, DEV)
    w = w.to(dtype)
    nq = H * (dim + rot)
    q = qd[:, :nq].to(D64).view(B, S, H, dim + rot)
    dkv = qd[:, nq:nq + rank + rot].to(D64).view(B, S, rank + rot)
    want_q, want_c = q.clone(), torch.zeros(B, cap, ld, dtype=D64)
    for b in range(B):
        for s in range(S):
            i = start + s
            want_c[b, i, :rank] = orc.rms_norm(dkv[b, s, :rank], w.to(D64), eps)
            want_c[b, i, rank:rank + rot] = orc.rotate_pairs(dkv[b, s, rank:], i, rot_dims, base)
            for h in range(H):
                want_q[b, s, h, dim:] = orc.rotate_pairs(q[b, s, h, dim:], i, rot_dims, base)
    g = qd.to(DEV)
    cache = torch.zeros(B, cap, ld, dtype=dtype, device=DEV)
    status = torch.zeros(1, dtype=torch.int32, device=DEV)
    kw = dict(S=S, n_heads=H, dim=dim, rot=rot, rank=rank, eps=eps, status=status)
    ops.latent_append(g[:, nq:nq + rank + rot], g[:, :nq], w.to(DEV), angles, cache, start=start, **kw)
    assert int(status) == 0
    _close(cache, want_c, dtype, tol16=4e-3, tol32=3e-6)
    _close(g[:, :nq].view(B, S, H, -1), want_q, dtype, tol16=4e-3, tol32=3e-6)
    ops.latent_append(g[:, nq:nq + rank + rot], g[:, :nq], w.to(DEV), angles, cache, start=cap - S + 1, **kw)
    assert int(status) == 1                                    # one token beyond the cache: reported, not written
    # the key up-projection on the query side gives the same scores as on the key side
    uk, uv = _rand(H * dim, rank, seed=3, dtype=dtype, scale=rank ** -0.5), _rand(H * vdim, rank, seed=4, dtype=dtype, scale=rank ** -0.5)
    qg = qd[:, :nq].to(DEV)
    got = ops.latent_absorb(qg, uk.to(DEV), H, dim, rot, ld)
    want = torch.zeros(B * S, H, ld, dtype=D64)
    qq = qd[:, :nq].to(D64).view(B * S, H, dim + rot)
    want[:, :, :rank] = torch.einsum("rhd,hdk->rhk", qq[:, :, :dim], uk.to(D64).view(H, dim, rank))
    want[:, :, rank:rank + rot] = qq[:, :, dim:]
    _close(got, want, dtype)
    o = _rand(B * S, H, rank, seed=5, dtype=dtype)
    want = torch.einsum("rhk,hek->rhe", o.to(D64), uv.to(D64).view(H, vdim, rank)).reshape(B * S, H * vdim)
    _close(ops.latent_up(o.to(DEV), uv.to(DEV), vdim), want, dtype)


# ------------------------------------------------------------------------------- state space
SSM = [dict(H=4, P=24, N=16, G=2, taps=3), dict(H=2, P=64, N=128, G=1, taps=4), dict(H=3, P=40, N=24, G=3, taps=2),
       dict(H=2, P=16, N=200, G=2, taps=4), dict(H=2, P=8, N=8, G=1, taps=1)]


def _ssm_inputs(c, B, S, dtype, seed=0):
    H, P, N, G, taps = c["H"], c["P"], c["N"], c["G"], c["taps"]
    inner, ch = H * P, H * P + 2 * G * N
    ld = (inner + ch + H + 7) // 8 * 8
    proj = _rand(B * S, ld, seed=seed, dtype=dtype)
    w = dict(conv_w=_rand(ch, taps, seed=1, dtype=dtype, scale=0.6), conv_b=_rand(ch, seed=2, dtype=dtype, scale=0.3),
             dt_bias=_rand(H, seed=3) - 1.5, A_log=_rand(H, seed=4, scale=1.0) - 1.0, D=_rand(H, seed=5))
    return proj, w, inner, ch


def _plain_ssm(c, proj, w, inner, ch, B, S):
    H, P, N, G = c["H"], c["P"], c["N"], c["G"]
    ys, sts = [], []
    for b in range(B):
        r = proj[b * S:(b + 1) * S].to(D64)
        x = orc.silu(orc.causal_conv(r[:, inner:inner + ch], w["conv_w"].to(D64), w["conv_b"].to(D64)))
        dt = orc.softplus(r[:, inner + ch:inner + ch + H] + w["dt_bias"].to(D64))
        y, st = orc.state_space(x[:, :inner].reshape(S, H, P), x[:, inner:inner + G * N].reshape(S, G, N),
                                x[:, inner + G * N:].reshape(S, G, N), dt, w["A_log"].to(D64), w["D"].to(D64))
        ys.append(y.reshape(S, inner)), sts.append(st)
    return torch.stack(ys), torch.stack(sts)


@pytest.mark.parametrize("case", range(len(SSM)))
@pytest.mark.parametrize("path", ["steps32", "steps", "chunks"])
def test_state_space_in_portions(case, path):
    """One long portion, and the same tokens in portions of all kinds of sizes (also single tokens by a
    position on the device): the same outputs, the same final state; dirty state is not seen at position 0."""
    c, B, S = SSM[case], 2, 210
    dtype = F32 if path == "steps32" else BF16
    path = "steps" if path == "steps32" else path
    proj, w, inner, ch = _ssm_inputs(c, B, S, dtype)
    want, want_st = _plain_ssm(c, proj, w, inner, ch, B, S)
    wg = {k: v.to(DEV) for k, v in w.items()}
    pg = proj.to(DEV).view(B, S, -1)

    def fresh():
        return (torch.full((B, c["taps"] - 1, ch), 5.0, dtype=dtype, device=DEV),
                torch.full((B, c["H"], c["N"], c["P"]), 3.0, device=DEV))

    for sizes in ([S], [1, 2, 2, 59, 64, 1, 65, 16], [64, 128, 3, 15], [2] * 105):
        conv, state = fresh()
        out, at = [], 0
        for n in sizes:
            rows = pg[:, at:at + n].reshape(B * n, -1)
            kw = dict(pos=torch.tensor([at], device=DEV)) if n == 1 else dict(start=at)
            y = ops.ssm(rows, inner, wg["conv_w"], wg["conv_b"], wg["dt_bias"], wg["A_log"], wg["D"], conv, state, S=n,
                        groups=c["G"], path="steps" if n == 1 else path, **kw)
            out.append(y.view(B, n, inner))
            at += n
        _close(torch.cat(out, 1), want, dtype)
        _close(state, want_st, dtype, tol16=1e-2)
        kept = proj.view(B, S, -1)[:, S - (c["taps"] - 1):, inner:inner + ch]
        assert torch.equal(conv.cpu(), kept)


def test_block_recurrence_keeps_more_than_bf16():
    """With the same bf16 inputs the block form and the token-by-token fp32 form differ by far less than the
    output's own rounding; a slowly decaying state over a long portion included."""
    c, B, S = dict(H=2, P=32, N=64, G=1, taps=1), 1, 1000
    proj, w, inner, ch = _ssm_inputs(c, B, S, BF16, seed=9)
    w["A_log"] = torch.tensor([-6.0, 1.0])
    states = []
    for path in ("steps", "chunks"):
        wg = {k: v.to(DEV) for k, v in w.items()}
        conv, state = torch.zeros(B, 0, ch, dtype=BF16, device=DEV), torch.zeros(B, 2, 64, 32, device=DEV)
        ops.ssm(proj.to(DEV), inner, wg["conv_w"], wg["conv_b"], wg["dt_bias"], wg["A_log"], wg["D"], conv, state, S=S, groups=1,
                path=path)
        states.append(state)
    assert (states[0] - states[1]).abs().max() <= 3e-5 * states[0].abs().max()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,inner,parts", [(5, 96, 4), (3, 30, 3), (400, 512, 1), (2, 8192, 2), (1, 5120, 8)])
def test_gated_group_norm(rows, inner, parts, dtype):
    y, z, w = _rand(rows, inner, seed=1, dtype=dtype), _rand(rows, inner + 12, seed=2, dtype=dtype), _rand(inner, seed=3, dtype=dtype)
    want = orc.gated_group_norm(y.to(D64), z[:, :inner].to(D64), w.to(D64), parts, 1e-3)
    _close(ops.gated_group_norm(y.to(DEV), z.to(DEV), w.to(DEV), parts, 1e-3), want, dtype)


def test_bias_table_of_a_layer_reaches_every_bucket():
    from socket_b200.mixers import ChunkedAttention
    m = ChunkedAttention(16, 2, 1, 8, 8, chunk=300, scale=1.0, bias_rows=12, bias_max=100).to(DEV)
    with torch.no_grad():
        m.rel.copy_(torch.arange(24.).view(12, 2))
    m.finish_loading()
    want = distance_buckets(100, 12, 100)
    assert sorted(set(want.tolist())) == list(range(12))
    assert torch.equal(m.bias.cpu(), torch.arange(24.).view(12, 2)[want].t())
