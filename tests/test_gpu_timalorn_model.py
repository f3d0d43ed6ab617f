"""The Timalorn decoder as a whole, against the plain implementation: prompts, token-by-token decoding,
portions, batches, slots that are used again, greedy generation, and trace replay."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import timalorn_oracle as orc
from socket_b200.decoder import generate
from socket_b200.registry import build_model, write_safetensors
from socket_b200.trace import TraceSession
from tests.timalorn_util import CONFIGS, attention, config, memory

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F32, BF16 = torch.float32, torch.bfloat16
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# rms of the logit error over the rms of the logits: (median, largest) over the positions
TOL = {F32: (1e-5, 4e-5), BF16: (4e-2, 2e-1)}

_plain = {}


def _weights(name):
    return orc.random_weights(CONFIGS[name], 17)


def _model(name, dtype):
    w = _weights(name)
    m = build_model(CONFIGS[name], {k: tuple(v.shape) for k, v in w.items()}, dtype, DEV)
    m.load_tensors(w)
    return m


def _tokens(name, n, seed=0):
    return torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _want(name, tokens):
    key = (name, tuple(tokens))
    if key not in _plain:
        _plain[key] = orc.forward(tokens, _weights(name), CONFIGS[name])
    return _plain[key]


def _check(got, want, dtype):
    got = got.detach().cpu().double()
    assert got.shape == want.shape and torch.isfinite(got).all()
    d = got - want
    err = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.std()
    assert err.median() <= TOL[dtype][0] and err.max() <= TOL[dtype][1], (float(err.median()), int(err.argmax()), float(err.max()))


def _idx(tokens):
    return torch.tensor([tokens], device=DEV)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_and_residual_stream(name, dtype):
    m = _model(name, dtype)
    tok = _tokens(name, 150)
    m.setup_caches(1, 160)
    _check(m.forward_portion(_idx(tok), 0, range(len(tok)))[0], _want(name, tok), dtype)
    want, got = [], []
    orc.forward(tok[:30], _weights(name), CONFIGS[name], residuals=want)
    m._portion(_idx(tok[:30]), 0, collect=got)
    assert len(want) == len(got) == len(m.runs)
    for a, b in zip(got, want):
        assert a.dtype == F32                               # the stream is fp32 in either element type
        assert (a.cpu().double() - b).pow(2).mean().sqrt() <= 2 * TOL[dtype][0] * b.pow(2).mean().sqrt()
    assert m.device_flags() == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_and_token_by_token_decoding(name, dtype):
    """All schedules of one sequence give the logits of the whole prompt: portions from two tokens up, cut
    before, at and after a window's length and a block's edge, then single tokens through the captured step."""
    m = _model(name, dtype)
    tok = _tokens(name, 150)
    want = _want(name, tok)
    m.setup_caches(1, 160)
    m.setup_decode(1)
    for sizes in ([2] * 30, [37, 37, 37], [36, 2, 38, 41], [1, 5, 33, 64, 7], [23, 2, 100], [96, 2, 3, 17]):
        rows, at = [], 0
        for n in sizes:
            rows.append(m.forward_portion(_idx(tok[at:at + n]), at, range(n))[0])
            at += n
        while at < len(tok):
            rows.append(m.decode_given_token(_idx(tok[at:at + 1]), at).clone())
            at += 1
        _check(torch.cat(rows), want, dtype)
    assert m.device_flags() == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_prompts(dtype):
    """Portions long enough for every form of the recurrence, one after the other, and decoding after them."""
    name = "wide"
    m = _model(name, dtype)
    tok = _tokens(name, 420, seed=11)
    want = _want(name, tok)
    m.setup_caches(1, 424)
    m.setup_decode(1)
    for sizes in ([420], [300, 100], [7, 260, 20, 3], [129, 256]):
        rows, at = [], 0
        for n in sizes:
            rows.append(m.forward_portion(_idx(tok[at:at + n]), at, range(n))[0])
            at += n
        while at < len(tok):
            rows.append(m.decode_given_token(_idx(tok[at:at + 1]), at).clone())
            at += 1
        _check(torch.cat(rows), want, dtype)
    assert m.device_flags() == 0


@pytest.mark.parametrize("name", ["shared", "odd", "wide"])
def test_decoding_from_the_first_token_on(name):
    """Long decoding without any prompt: position 0 itself through the decode step, several rounds of every ring."""
    m = _model(name, F32)
    tok = _tokens(name, 150)
    m.setup_caches(1, 160)
    m.setup_decode(1)
    rows = [m.decode_given_token(_idx(tok[i:i + 1]), i).clone() for i in range(len(tok))]
    _check(torch.cat(rows), _want(name, tok), F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["shared", "wide"])
def test_batches_equal_their_rows_alone(name, dtype):
    m = _model(name, dtype)
    seqs = [_tokens(name, 120, seed=s) for s in (1, 2, 3)]
    idx = torch.tensor(seqs, device=DEV)
    m.setup_caches(3, 128)
    m.setup_decode(3)
    rows = [m.forward_portion(idx[:, :70], 0, range(70)), m.forward_portion(idx[:, 70:97], 70, range(27))]
    rows += [m.decode_given_token(idx[:, i:i + 1], i).clone().unsqueeze(1) for i in range(97, 120)]
    got = torch.cat(rows, 1)
    for b, s in enumerate(seqs):
        _check(got[b], _want(name, s), dtype)
    # fewer sequences than the caches have room for
    part = m.forward_portion(idx[1:2, :50], 0, range(50))
    _check(part[0], _want(name, seqs[1])[:50], dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["shared", "odd"])
def test_a_slot_is_used_again(name, dtype):
    """Sequences one after the other in one slot, longer before shorter and shorter before longer."""
    m = _model(name, dtype)
    s = TraceSession(m, 160)
    for n, cut, seed in ((150, 149, 0), (23, 9, 5), (1, 1, 6), (97, 60, 7), (6, 2, 8)):
        tok = _tokens(name, n, seed)
        rows = [s.run("r%d" % seed, tok[:cut], range(cut))] + [s.run("r%d" % seed, [t], [0]) for t in tok[cut:]]
        rows = [r.clone() for r in rows]
        s.end("r%d" % seed)
        _check(torch.cat(rows), _want(name, tok), dtype)


@pytest.mark.parametrize("name", ["shared", "plain", "wide"])
def test_greedy_generation(name):
    """The framework's generate(): every token is the argmax of the logits of what came before it, with the
    graph and without, whole prompt and in portions."""
    m = _model(name, F32)
    prompt = torch.tensor([_tokens(name, 45, seed=3), _tokens(name, 45, seed=4)])
    seq, stats = generate(m, prompt, 30)
    assert seq.shape == (2, 75) and stats["decode_only_tokens"] == 58
    m.max_seq_length = -1
    assert torch.equal(generate(m, prompt, 30, use_graph=False, prefill_chunk=16)[0], seq)
    for b in range(2):
        logits = _want(name, seq[b].tolist())
        top2 = logits[44:74].topk(2).values
        clear = top2[:, 0] - top2[:, 1] > 1e-3 * logits.std()
        assert (logits[44:74].argmax(-1)[clear] == seq[b, 45:].cpu()[clear]).all() and clear.sum() > 20


@pytest.mark.parametrize("window,pairs", [(50, [(99, 50), (99, 49), (120, 71), (120, 70), (63, 63), (49, 0), (50, 0)]),
                                          (64, [(127, 64), (127, 63), (64, 0), (63, 0)]),
                                          (1, [(9, 9), (9, 8)])])
def test_keys_at_the_windows_edge_show_in_the_logits(window, pairs):
    """One attention layer, one query-key pair made to stand out in the unrotated elements: the key's token decides
    the query's logits exactly when the window holds it - in a prompt, in a late portion, and decoded."""
    cfg = config([attention(heads=2, kv_heads=1, dim=32, window=window, rot_dims=16, scale=0.3, softcap=20.0, ff=0)],
                 width=64, vocab=40, scale=1.0)
    w = orc.random_weights(cfg, 4)
    # token 38 asks, token 39 answers: their normed embeddings meet in one unrotated element of q and k
    w["embed"] = (0.3 * torch.randn(40, 64, generator=torch.Generator().manual_seed(2))).to(BF16)
    w["embed"][38] = torch.tensor([1.0, -1.0]).repeat(32).to(BF16)
    w["embed"][39] = torch.tensor([1.0, 1.0, -1.0, -1.0]).repeat(16).to(BF16)
    w["l0.norm1"] = torch.ones(64, dtype=BF16)
    ask, answer = torch.tensor([1.0, -1.0]).repeat(32) / 8, torch.tensor([1.0, 1.0, -1.0, -1.0]).repeat(16) / 8
    for h in range(2):
        w["l0.mix.q"][32 * h + 20] = ask.to(BF16)
    w["l0.mix.k"][20] = answer.to(BF16)
    w["l0.mix.sink"] = torch.tensor([2.0, 3.0]).to(BF16)
    for dtype in (F32, BF16):
        model = build_model(cfg, {k: tuple(v.shape) for k, v in w.items()}, dtype, DEV)
        model.load_tensors(w)
        model.setup_caches(1, 144)
        model.setup_decode(1)
        for i, j in pairs:
            tok = torch.randint(0, 38, (i + 1,), generator=torch.Generator().manual_seed(i * 131 + j)).tolist()
            tok[i] = 38
            tok[j] = 39
            want = orc.forward(tok, w, cfg)[-1:]
            gone = list(tok)
            gone[j] = 7
            moved = (orc.forward(gone, w, cfg)[-1:] - want).pow(2).mean().sqrt() / want.std()
            assert (moved > 0.05) if i - j < window else (moved == 0), (i, j, float(moved))
            _check(model.forward_portion(_idx(tok), 0)[0], want, dtype)
            if i > 2:
                model.forward_portion(_idx(tok[:i - 1]), 0, ())
                _check(model.forward_portion(_idx(tok[i - 1:]), i - 1)[0], want, dtype)
                model.forward_portion(_idx(tok[:i]), 0, ())
                _check(model.decode_given_token(_idx(tok[i:]), i), want, dtype)


def test_the_first_tokens_and_a_far_token_reach_the_memory():
    """A memory layer whose input gate opens for one token only: that token, first or far back, decides later
    outputs - whole, in portions and decoded."""
    cfg = config([memory(heads=2, dim=16, vdim=16, gate_cap=10.0, ff=0)], width=64, vocab=40, scale=1.0)
    w = orc.random_weights(cfg, 5)
    w["embed"][39] = torch.tensor([1.0, 1.0, -1.0, -1.0]).repeat(16).to(BF16)
    w["l0.norm1"] = torch.ones(64, dtype=BF16)
    opens = torch.tensor([1.0, 1.0, -1.0, -1.0]).repeat(16) / 8
    w["l0.mix.i"], w["l0.mix.i.b"] = opens.expand(2, 64).contiguous().to(BF16), torch.full((2,), -4.0).to(BF16)
    w["l0.mix.f"], w["l0.mix.f.b"] = torch.zeros(2, 64).to(BF16), torch.full((2,), 9.0).to(BF16)
    for dtype in (F32, BF16):
        m = build_model(cfg, {k: tuple(v.shape) for k, v in w.items()}, dtype, DEV)
        m.load_tensors(w)
        m.setup_caches(1, 144)
        m.setup_decode(1)
        for at in (0, 1, 63, 64, 70):
            tok = torch.randint(0, 38, (140,), generator=torch.Generator().manual_seed(at)).tolist()
            tok[at] = 39
            want = orc.forward(tok, w, cfg)
            gone = list(tok)
            gone[at] = 3
            other = orc.forward(gone, w, cfg)
            assert (other[-1] - want[-1]).pow(2).mean().sqrt() > 0.1 * want.std()
            for cut in (140, at + 1, 100):
                rows = [m.forward_portion(_idx(tok[:cut]), 0, range(cut))[0]]
                rows += [m.decode_given_token(_idx(tok[i:i + 1]), i).clone() for i in range(cut, 140)]
                _check(torch.cat(rows), want, dtype)


def test_sizes_the_fast_kernels_do_not_take_still_run_in_bf16():
    cfg = config([attention(heads=2, kv_heads=2, dim=136, rot_dims=4, window=33, ff=0), memory(heads=2, dim=20, vdim=12, ff=0)], width=60)
    w = orc.random_weights(cfg, 8)
    m = build_model(cfg, {k: tuple(v.shape) for k, v in w.items()}, BF16, DEV)
    m.load_tensors(w)
    m.setup_caches(1, 104)
    tok = torch.randint(0, cfg["vocab"], (100,), generator=torch.Generator().manual_seed(0)).tolist()
    _check(m.forward_portion(_idx(tok), 0, range(100))[0], orc.forward(tok, w, cfg), BF16)


def test_a_token_outside_the_vocabulary_raises_the_status_flag():
    m = _model("plain", F32)
    m.setup_caches(1, 16)
    m.forward_portion(_idx([1, 2, CONFIGS["plain"]["vocab"]]), 0)
    assert m.device_flags() != 0


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_runner_as_a_process(dtype, tmp_path):
    name = "shared"
    cfg, folder, out = CONFIGS[name], tmp_path / "model", tmp_path / "out"
    folder.mkdir(), out.mkdir()
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(folder / "model.safetensors"), _weights(name))
    a, b = _tokens(name, 61, seed=1), _tokens(name, 33, seed=2)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:40], want=[0, 39])], end=[]),
             dict(step=1, entries=[dict(id="a", tokens=a[40:60], want=[])], end=[]),
             dict(step=2, entries=[dict(id="a", tokens=a[60:], want=[0])], end=["a"]),
             dict(step=3, entries=[dict(id="b", tokens=b, want=list(range(33)))], end=["b"])]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True,
                       text=True, timeout=300, env=dict(os.environ, PATH=os.path.dirname(sys.executable) + ":" + os.environ["PATH"]))
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    got = {i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").copy()).view(-1, cfg["vocab"]) for i in (0, 2, 3)}
    assert not (out / "1.f32").exists()
    wa, wb = _want(name, a), _want(name, b)
    dt = getattr(torch, dtype)
    _check(got[0], wa[[0, 39]], dt), _check(got[2], wa[60:], dt), _check(got[3], wb, dt)


def test_generation_from_the_command_line(tmp_path):
    """Same tokens as generate() in this process; two prompts as a batch."""
    name = "shared"
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS[name]))
    write_safetensors(str(tmp_path / "model.safetensors"), _weights(name))
    prompts = [_tokens(name, 30, seed=1), _tokens(name, 30, seed=2)]
    want, _ = generate(_model(name, F32), torch.tensor(prompts), 8)
    text = ";".join(",".join(map(str, p)) for p in prompts)
    r = subprocess.run([sys.executable, "-m", "socket_b200.generate", "--model", str(tmp_path), "--tokens", text, "--new", "8",
                        "--dtype", "float32", "--prefill-chunk", "13"], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [[int(t) for t in line.split(",")] for line in r.stdout.split()] == want[:, 30:].tolist()
