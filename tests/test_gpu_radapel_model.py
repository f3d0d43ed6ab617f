"""The Radapel decoder as a whole, against the plain implementation: prompts, token-by-token decoding,
portions, batches, slots that are used again, greedy generation, and trace replay."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import radapel_oracle as orc
from tests.radapel_util import CONFIGS, attention, config, latent, mamba
from socket_b200.decoder import generate
from socket_b200.registry import build_model, write_safetensors
from socket_b200.trace import TraceSession

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F32, BF16 = torch.float32, torch.bfloat16
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# rms of the logit error over the rms of the logits: (median, largest) over the positions.  The weights of
# these tests make scores large, so that in bf16 a few positions amplify rounding; faults show in fp32.
TOL = {F32: (2e-5, 4e-5), BF16: (6e-2, 3e-1)}

_plain = {}


def _weights(name):
    return orc.random_weights(CONFIGS[name], 17, bias_rows=14)


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
    before, at and after chunk borders, then single tokens through the captured step."""
    m = _model(name, dtype)
    tok = _tokens(name, 150)
    want = _want(name, tok)
    m.setup_caches(1, 160)
    m.setup_decode(1)
    for sizes in ([2] * 30, [40, 40, 40], [39, 2, 38, 41], [1, 5, 33, 64, 7], [23, 2, 100]):
        rows, at = [], 0
        for n in sizes:
            rows.append(m.forward_portion(_idx(tok[at:at + n]), at, range(n))[0])
            at += n
        while at < len(tok):
            rows.append(m.decode_given_token(_idx(tok[at:at + 1]), at).clone())
            at += 1
        _check(torch.cat(rows), want, dtype)
    assert m.device_flags() == 0


@pytest.mark.parametrize("name", ["looped", "wide"])
def test_decoding_from_the_first_token_on(name):
    """Long decoding without any prompt: position 0 itself through the decode step."""
    m = _model(name, F32)
    tok = _tokens(name, 150)
    m.setup_caches(1, 160)
    m.setup_decode(1)
    rows = [m.decode_given_token(_idx(tok[i:i + 1]), i).clone() for i in range(len(tok))]
    _check(torch.cat(rows), _want(name, tok), F32)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_batches_equal_their_rows_alone(dtype):
    name = "wide"
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


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["looped", "odd"])
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
    with pytest.raises(RuntimeError, match="before"):
        s.run("a", [1], [])
        s.run("b", [1], [])


@pytest.mark.parametrize("name", ["looped", "plain", "wide"])
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


def test_far_keys_and_borders_show_in_the_logits():
    """One layer each, a single query-key pair made to stand out: the key's token decides the query's logits
    exactly when the mask lets it be seen - for a key just inside and just outside the chunk, and for the
    first token under the sink - in a prompt, and decoded."""
    for layer, pairs in ((attention(heads=2, kv_heads=1, dim=32, vdim=32, chunk=50, mlp=False), [(99, 50), (99, 49), (100, 99), (50, 50)]),
                         (latent(heads=2, dim=32, rot_dim=16, vdim=32, kv_rank=48, mlp=False), [(130, 0), (64, 63), (128, 64)])):
        cfg = config([layer], width=64, vocab=40, scale=1.0)
        w = orc.random_weights(cfg, 4)
        m = layer["mixer"]
        # token 38 asks, token 39 answers: their (normed) embeddings meet in one direction of q and k
        emb = torch.zeros(64)
        emb[:32] = 1.0
        w["embed"] = (0.3 * torch.randn(40, 64, generator=torch.Generator().manual_seed(2))).to(BF16)
        w["embed"][38], w["embed"][39] = emb.to(BF16), (emb.flip(0) * 1.5).to(BF16)
        w["l0.norm1"] = torch.ones(64, dtype=BF16)
        ask, answer = torch.zeros(64), torch.zeros(64)
        ask[:32], answer[32:] = 0.4, 0.4
        q, kname = w["l0.mix.q"], "l0.mix.k" if layer["type"] == "attention" else "l0.mix.uk"
        if layer["type"] == "attention":
            q[0], w[kname][0] = ask.to(BF16), answer.to(BF16)
        else:
            w["l0.mix.dkv"][0], w[kname][0], q[0] = answer.to(BF16), 0, ask.to(BF16)
            w[kname][0, 0] = 2.0
        for dtype in (F32, BF16):
            model = build_model(cfg, {k: tuple(v.shape) for k, v in w.items()}, dtype, DEV)
            model.load_tensors(w)
            model.setup_caches(1, 144)
            model.setup_decode(1)
            for i, j in pairs:
                tok = torch.randint(0, 38, (i + 1,), generator=torch.Generator().manual_seed(i * 131 + j)).tolist()
                tok[j] = 39
                tok[i] = 38
                if i == j:
                    tok[i] = 39
                want = orc.forward(tok, w, cfg)[-1:]
                gone = list(tok)
                gone[j] = 7
                moved = (orc.forward(gone, w, cfg)[-1:] - want).pow(2).mean().sqrt() / want.std()
                seen = m.get("mask") is None or i // m["mask"]["size"] == j // m["mask"]["size"]
                assert bool(moved > 0.1) == seen, (i, j, float(moved))
                _check(model.forward_portion(_idx(tok), 0)[0], want, dtype)
                if i > 0:
                    model.forward_portion(_idx(tok[:i]), 0, ())
                    _check(model.decode_given_token(_idx(tok[i:]), i), want, dtype)


def test_sizes_the_fast_kernels_do_not_take_still_run_in_bf16():
    cfg = config([attention(heads=2, kv_heads=2, dim=20, vdim=136, chunk=33, mlp=False), mamba(heads=2, vdim=12, state=20, groups=1)], width=60)
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
    name = "looped"
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
    name = "looped"
    (tmp_path / "config.json").write_text(json.dumps(CONFIGS[name]))
    write_safetensors(str(tmp_path / "model.safetensors"), _weights(name))
    prompts = [_tokens(name, 30, seed=1), _tokens(name, 30, seed=2)]
    want, _ = generate(_model(name, F32), torch.tensor(prompts), 8)
    text = ";".join(",".join(map(str, p)) for p in prompts)
    r = subprocess.run([sys.executable, "-m", "socket_b200.generate", "--model", str(tmp_path), "--tokens", text, "--new", "8",
                        "--dtype", "float32", "--prefill-chunk", "13"], capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [[int(t) for t in line.split(",")] for line in r.stdout.split()] == want[:, 30:].tolist()
