"""Host-side checks of the Timalorn decoder that need no GPU: configuration, shared tensors, weight loading,
rotary frequencies, and the plain implementation against properties that follow from the definitions."""
import json
import math

import pytest
import torch

from oracle import timalorn_oracle as orc
from socket_b200 import block_ops
from socket_b200.mixers import YarnScaling, rotary_angles, rotary_frequencies
from socket_b200.registry import ARCHITECTURES, build_model, libraries_of, load_model, write_safetensors
from socket_b200.timalorn import TimalornConfig
from tests.timalorn_util import CONFIGS, attention, config, memory

D64 = torch.float64


def _rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=D64)


# ------------------------------------------------------------------------------- configuration, weights
def test_registry_and_library():
    assert "Timalorn" in ARCHITECTURES and libraries_of(CONFIGS["plain"]) == ("blocks",)


def test_owners_of_shared_tensors():
    cfg = TimalornConfig.from_dict(CONFIGS["shared"])
    assert cfg.owners == (0, 1, 0, 3, 1, 5)
    assert TimalornConfig.from_dict(CONFIGS["plain"]).owners == (2, 1, 2)
    chain = config([attention(), attention(weights_of=0), attention(weights_of=1)])
    assert TimalornConfig.from_dict(chain).owners == (0, 0, 0) and orc.owner(chain, 2) == 0


def test_bad_configurations_are_refused():
    for bad, what in ((dict(attention(), type="other"), "mixer"),
                      (dict(attention(), mlp={"kind": "sparse", "ff": 8}), "feed-forward"),
                      (dict(attention(), mixer=dict(attention()["mixer"], vdim=16)), "keys"),
                      (attention(weights_of=0), "weights_of")):
        with pytest.raises(ValueError, match=what):
            TimalornConfig.from_dict(config([bad, memory()]))
    with pytest.raises(ValueError, match="differ"):
        TimalornConfig.from_dict(config([attention(), attention(window=8, weights_of=0)]))
    with pytest.raises(ValueError, match="weights_of"):
        TimalornConfig.from_dict(config([memory(weights_of=1), memory(weights_of=0)]))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_weights_load_from_a_model_folder(name, tmp_path):
    cfg = CONFIGS[name]
    w = orc.random_weights(cfg, 3)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    model = load_model(str(tmp_path), torch.float32, "cpu")
    own = model.tensors()
    assert {k: tuple(v.shape) for k, v in own.items()} == orc.tensor_shapes(cfg)
    for k, v in own.items():
        assert torch.equal(v, w[k].float()), k
    # every element of a fused matrix is some tensor's or stays zero
    for i, layer in model.layers.items():
        mine = {k.split(".", 1)[1]: v for k, v in w.items() if k.startswith(f"l{i}.")}
        big = [v for k, v in mine.items() if k in ("mix.q", "mix.k", "mix.v", "mix.g", "mlp.gate", "mlp.up")]
        assert int((layer.w_in != 0).sum()) == sum(int((t != 0).sum()) for t in big)
        big = [v for k, v in mine.items() if k in ("mix.o", "mlp.down")]
        assert int((layer.w_out != 0).sum()) == sum(int((t != 0).sum()) for t in big)
    for bad in ({k: v for k, v in w.items() if k != "head"}, dict(w, other=w["head"]), dict(w, head=w["head"][:-1])):
        with pytest.raises(ValueError):
            model.load_tensors(bad)


def test_layers_that_share_tensors_have_caches_of_their_own():
    m = build_model(CONFIGS["shared"], dtype=torch.float32, device="cpu")
    assert len(m.runs) == 6 and len(m.layers) == 4
    caches = [m.layer_of(r).mixer.make_cache(1, 16, torch.float32, "cpu") for r in m.runs]
    assert m.layer_of(m.runs[0]) is m.layer_of(m.runs[2]) and caches[0].rows.data_ptr() != caches[2].rows.data_ptr()
    assert m.layer_of(m.runs[1]) is m.layer_of(m.runs[4]) and caches[1].S.data_ptr() != caches[4].S.data_ptr()
    assert caches[0].angles.data_ptr() == caches[2].angles.data_ptr()
    assert caches[0].rows.shape == (1, 16, 2, 32) and caches[5].rows.shape[1] == 9     # no more rows than the window


def test_operators_refuse_cpu_tensors():
    z = torch.zeros
    with pytest.raises(RuntimeError, match="CUDA"):
        block_ops.rotary_rows(z(1, 2, 8), z(1, 1, 8), z(4, 2, 2), 4, z(1, 4, 1, 12), B=1, S=1)
    with pytest.raises(RuntimeError, match="CUDA"):
        block_ops.glu_silu(z(2, 8), z(2, 8))


# ------------------------------------------------------------------------------- rotary frequencies
@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [
    (8, 3000.0, 3.0, 48, 5.0, 0.6), (64, 10000.0, 8.0, 2048, 32.0, 1.0), (2, 500.0, 2.0, 64, 4.0, 1.0),
    (128, 1e6, 40.0, 4096, 32.0, 1.0), (16, 100.0, 4.0, 16, 30.0, 20.0), (10, 777.0, 1.0, 100, 2.0, 2.0)])
def test_rotary_frequencies(dims, base, factor, original, fast, slow):
    s = dict(factor=factor, original=original, fast=fast, slow=slow)
    want = orc.rotary_frequencies(dims, base, s)
    got = rotary_frequencies(dims, base, YarnScaling(factor, original, fast, slow))
    torch.testing.assert_close(got, torch.tensor(want, dtype=D64), rtol=1e-12, atol=0)
    plain = [base ** (-2 * i / dims) for i in range(dims // 2)]
    assert all(p / factor * (1 - 1e-12) <= f <= p * (1 + 1e-12) for f, p in zip(want, plain))
    a = rotary_angles(3000, dims, base, "cpu", YarnScaling(factor, original, fast, slow))
    gain = 0.1 * math.log(factor) + 1
    for p in (0, 1, 2999):
        for i, f in enumerate(want):
            assert abs(float(a[p, i, 0]) - gain * math.cos(p * f)) < 1e-6 and abs(float(a[p, i, 1]) - gain * math.sin(p * f)) < 1e-6


def test_frequencies_are_kept_blended_and_stretched():
    """Over a wide band all three kinds occur: fast pairs as they are, slow ones divided by the factor."""
    s = dict(factor=16.0, original=4096, fast=32.0, slow=1.0)
    f = orc.rotary_frequencies(128, 10000.0, s)
    ratio = [a / 10000.0 ** (-2 * i / 128) for i, a in enumerate(f)]
    assert abs(ratio[0] - 1) < 1e-12 and abs(ratio[-1] - 1 / 16) < 1e-12 and any(0.1 < r < 0.9 for r in ratio)
    assert all(a >= b - 1e-12 for a, b in zip(ratio, ratio[1:]))


# ------------------------------------------------------------------------------- the plain implementation
def test_plain_rotation_depends_on_distance_only():
    rot = attention()["mixer"]["rot"]
    q, k = _rand(24, seed=1), _rand(24, seed=2)
    at = lambda x, p: orc.rotate_halves(x, p, rot)  # noqa: E731
    torch.testing.assert_close(at(q, 40) @ at(k, 33), at(q, 7) @ at(k, 0))
    assert not torch.allclose(at(q, 40) @ at(k, 33), at(q, 8) @ at(k, 0))
    assert torch.equal(at(q, 5)[8:], q[8:])


def test_plain_attention_sees_its_window_only():
    cfg = config([attention(window=6, ff=0)], width=40)
    w = orc.random_weights(cfg, 1)
    tok = torch.randint(0, cfg["vocab"], (20,), generator=torch.Generator().manual_seed(1)).tolist()
    full = orc.forward(tok, w, cfg)
    for j in (0, 5, 11):
        other = list(tok)
        other[j] = (tok[j] + 1) % cfg["vocab"]
        changed = (orc.forward(other, w, cfg) - full).abs().amax(-1) > 0
        assert changed.tolist() == [j <= i < j + 6 for i in range(20)]


def test_plain_sink_takes_weight_only():
    v, s, sink = _rand(4, 3, seed=1), _rand(4, seed=2), torch.tensor(1.3, dtype=D64)
    f = torch.exp(s).sum() / (torch.exp(s).sum() + math.exp(1.3))
    torch.testing.assert_close(orc.attend(s, v, sink), orc.attend(s, v) * f)


def test_plain_memory_carries_its_state_and_equals_its_unstabilised_form():
    S, N, P = 13, 5, 4
    q, k, v = _rand(S, N, seed=1), _rand(S, N, seed=2), _rand(S, P, seed=3)
    i, f = 2 * _rand(S, seed=4), orc.log_sigmoid(2 * _rand(S, seed=5))
    o, (st, n, m) = orc.matrix_memory(q, k, v, i, f)
    o1, s1 = orc.matrix_memory(q[:6], k[:6], v[:6], i[:6], f[:6])
    o2, (st2, n2, m2) = orc.matrix_memory(q[6:], k[6:], v[6:], i[6:], f[6:], s1)
    torch.testing.assert_close(torch.cat([o1, o2]), o)
    torch.testing.assert_close((st2, n2, m2), (st, n, m))
    # sums weighted by exp(i_s + f_{s+1} + .. + f_t); the denominator's floor is 1 in these units
    for t in range(S):
        wts = torch.stack([torch.exp(i[s] + f[s + 1:t + 1].sum()) for s in range(t + 1)])
        num = (wts[:, None] * v[:t + 1] * (k[:t + 1] @ q[t])[:, None]).sum(0)
        den = (wts * (k[:t + 1] @ q[t])).sum().abs().clamp(min=1.0)
        torch.testing.assert_close(o[t], num / den, rtol=1e-4, atol=1e-5)       # the 1e-6 beside the floor


def test_plain_parallel_layer_has_one_norm():
    cfg = config([memory()])
    w = {k: v.to(D64) for k, v in orc.random_weights(cfg, 2).items()}
    sub = {k[3:]: v for k, v in w.items() if k.startswith("l0.")}
    x = _rand(5, 80)
    h = orc.layer_norm(x, sub["norm1"], 3e-5)
    mix = orc.mlstm(h, {k[4:]: v for k, v in sub.items() if k.startswith("mix.")}, cfg["layers"][0]["mixer"], 3e-5)
    ff = orc.feed_forward(h, {k[4:]: v for k, v in sub.items() if k.startswith("mlp.")})
    torch.testing.assert_close(orc.layer(x, sub, cfg["layers"][0], 3e-5), x + mix + ff)
    assert abs(float((h / sub["norm1"]).mean())) < 1e-12
