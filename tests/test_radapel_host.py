"""Host-side checks of the Radapel decoder that need no GPU: configuration and layer order, weight
loading, the distance buckets, the checkpoint reader, the block library's binding, and the plain
implementation against properties that follow from the definitions."""
import json
import math
import os
import re

import pytest
import torch

from oracle import radapel_oracle as orc
from socket_b200 import _lib, block_ops, build
from socket_b200.mixers import distance_buckets, rotary_angles
from socket_b200.radapel import RadapelConfig, layer_runs
from socket_b200.registry import (ARCHITECTURES, build_model, libraries_of, load_model, read_safetensors,
                                  write_safetensors)
from tests.radapel_util import CONFIGS, attention, config, latent, mamba

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ------------------------------------------------------------------------------- library
def test_block_library_exports_every_declared_symbol():
    text = open(os.path.join(ROOT, "include", "socket_b200_blocks.h")).read()
    names = sorted(set(re.findall(r"SK_API[^;(]*?\b(skb_\w+)\s*\(", text)))
    lib = _lib.blocks()
    assert len(names) >= 15 and sorted(_lib.BLOCK_SIGNATURES) == names
    for n in names:
        assert hasattr(lib, n), n
    assert lib.skb_abi_version() == 1


@pytest.mark.parametrize("struct,cls", [("sk_residual_params", _lib.ResidualParams), ("sk_attn_params", _lib.AttnParams),
                                        ("sk_rotary_rows_params", _lib.RotaryRowsParams), ("sk_mlstm_params", _lib.MlstmParams),
                                        ("sk_latent_params", _lib.LatentParams), ("sk_ssm_params", _lib.SsmParams)])
def test_block_structs_match_the_header(struct, cls):
    text = open(os.path.join(ROOT, "include", "socket_b200_blocks.h")).read()
    body = text[text.index(f"typedef struct {struct} {{"):text.index(f"}} {struct};")]
    body = re.sub(r"/\*.*?\*/", "", body, flags=re.S)
    fields = [re.findall(r"(\w+)\s*$", name.strip())[0]
              for decl in body.split("{", 1)[1].split(";") if decl.strip() for name in decl.split(",")]
    assert fields == [f[0] for f in cls._fields_]


def test_block_operators_refuse_bad_arguments_and_cpu_tensors():
    with pytest.raises(RuntimeError, match="CUDA"):
        block_ops.embed_rows(torch.zeros(3, dtype=torch.long), torch.zeros(4, 8), 1.0)
    p = _lib.AttnParams()
    lib = _lib.blocks()
    import ctypes
    assert lib.skb_attn(ctypes.byref(p), None) == -1 and b"null pointer" in lib.skb_last_error()
    p.q = p.k = p.v = p.out = 1 << 20
    p.dtype, p.B, p.S, p.H, p.G, p.dqk, p.dv, p.kv_rows = _lib.SK_BF16, 1, 4, 6, 4, 64, 64, 64
    assert lib.skb_attn(ctypes.byref(p), None) == -1 and b"multiple" in lib.skb_last_error()
    p.G, p.start = 3, 61
    assert lib.skb_attn(ctypes.byref(p), None) == -1 and b"positions up to 64" in lib.skb_last_error()


def test_a_model_compiles_only_its_own_library():
    assert libraries_of({"architecture": "Radapel"}) == ("blocks",) and libraries_of({"architecture": "Transformer"}) == ("step",)
    step = {os.path.basename(s) for s in build._sources("step")}
    blocks = {os.path.basename(s) for s in build._sources("blocks")}
    assert step & blocks == {"host.cu"} and {s + ".cu" for s in build.BLOCK_SOURCES} <= blocks
    with pytest.raises(ValueError, match="unknown architecture"):
        libraries_of({"architecture": "none such"})


# ------------------------------------------------------------------------------- configuration, weights
def test_layer_order_of_a_loop():
    runs = layer_runs(RadapelConfig.from_dict(CONFIGS["looped"]))
    assert [r.layer for r in runs] == [0, 1, 2, 3, 1, 2, 3, 1, 2, 3, 4]
    assert [r.new_pass for r in runs] == [None, 0, None, None, 1, None, None, 2, None, None, None]
    assert [(r.layer, r.new_pass) for r in runs] == [(i, t if f else None) for i, t, f in orc.layer_order(CONFIGS["looped"])]
    assert [r.layer for r in layer_runs(RadapelConfig.from_dict(CONFIGS["plain"]))] == [0, 1, 2]


def test_bad_configurations_are_refused():
    with pytest.raises(ValueError, match="mixer"):
        RadapelConfig.from_dict(config([dict(attention(), type="other")]))
    with pytest.raises(ValueError, match="feed-forward"):
        RadapelConfig.from_dict(config([dict(attention(), mlp={"kind": "sparse", "ff": 8, "limit": 1.0})]))
    with pytest.raises(ValueError, match="loop"):
        RadapelConfig.from_dict(config([attention(), mamba()], loop=(1, 3, 2)))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_weights_load_from_a_model_folder(name, tmp_path):
    cfg = CONFIGS[name]
    w = orc.random_weights(cfg, 3, bias_rows=10)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), w)
    model = load_model(str(tmp_path), torch.float32, "cpu")
    own = model.tensors()
    assert {k: tuple(v.shape) for k, v in own.items()} == orc.tensor_shapes(cfg, bias_rows=10)
    for k, v in own.items():
        assert torch.equal(v, w[k].float()), k
    # derived buffers: a cache row's expansion is the keys and values of its latent
    for i, e in enumerate(cfg["layers"]):
        if e["type"] == "latent_attention":
            m, mix = e["mixer"], model.layers[i].mixer
            row = torch.zeros(mix.row)
            row[:m["kv_rank"] + m["rot_dim"]] = torch.randn(m["kv_rank"] + m["rot_dim"])
            kv = mix.expand @ row
            c, rot = row[:m["kv_rank"]], row[m["kv_rank"]:m["kv_rank"] + m["rot_dim"]]
            uk = (w[f"l{i}.mix.uk"].float() @ c).view(m["heads"], m["dim"])
            want = torch.cat([torch.cat([uk, rot.expand(m["heads"], -1)], 1).reshape(-1), w[f"l{i}.mix.uv"].float() @ c])
            torch.testing.assert_close(kv, want)
        elif e["type"] == "attention":
            m, mix = e["mixer"], model.layers[i].mixer
            for n in range(0, mix.bias.shape[1]):
                row = orc.distance_bucket(n, 10, m["bias_max"])
                assert torch.equal(mix.bias[:, n], w[f"l{i}.mix.rel"].float()[row])
    # missing, additional and misshapen tensors are refused
    for bad in ({k: v for k, v in w.items() if k != "head"}, dict(w, other=w["head"]), dict(w, head=w["head"][:-1])):
        with pytest.raises(ValueError):
            model.load_tensors(bad)


def test_safetensors_round_trip(tmp_path):
    path = str(tmp_path / "a.safetensors")
    t = {"a": torch.randn(3, 5).to(torch.bfloat16), "b": torch.arange(7, dtype=torch.int32), "c": torch.randn(2, 2, 2),
         "d": torch.zeros(0, 4)}
    write_safetensors(path, t)
    got = read_safetensors(path)
    assert all(torch.equal(got[k], v) and got[k].dtype == v.dtype for k, v in t.items()) and set(got) == set(t)
    raw = open(path, "rb").read()
    open(path, "wb").write(raw[:-1])
    with pytest.raises(ValueError):
        read_safetensors(path)


def test_the_frameworks_transformer_is_in_the_same_registry(tmp_path):
    from socket_b200.model import ModelArgs, Transformer
    cfg = dict(architecture="Transformer", block_size=64, vocab_size=64, n_layer=1, n_head=2, n_local_heads=1, dim=256,
               intermediate_size=64)
    a = Transformer(ModelArgs(**{k: v for k, v in cfg.items() if k != "architecture"})).init_random(1)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), a.state_dict())
    b = load_model(str(tmp_path), torch.float32, "cpu")
    prompt = torch.arange(9).view(1, 9)
    for m in (a, b):
        m.setup_caches(1, 16)
    assert torch.equal(a.prefill(prompt), b.prefill(prompt))
    # logits at chosen places of a portion: the last one is what prefill returns
    some = b.forward_portion(prompt, 0, [2, 8])
    torch.testing.assert_close(some[:, 1], a.prefill(prompt))
    assert set(ARCHITECTURES) >= {"Radapel", "Transformer"}


def test_positions_outside_the_caches_are_refused():
    m = build_model(CONFIGS["plain"], dtype=torch.float32, device="cpu")
    m.max_batch_size, m.max_seq_length = 1, 8
    with pytest.raises(RuntimeError, match="outside the caches"):
        m.forward_portion(torch.zeros(1, 5, dtype=torch.long), 4)


# ------------------------------------------------------------------------------- distance buckets, angles
@pytest.mark.parametrize("rows,far", [(16, 50), (16, 128), (10, 160), (9, 77), (32, 1000), (6, 4.5), (8, 9), (20, 6)])
def test_distance_buckets(rows, far):
    top = max(math.ceil(far), rows)
    got = distance_buckets(top, rows, far).tolist()
    half = rows // 2
    assert got[:half] == list(range(half)) and got[-1] == rows - 1
    assert all(b - a >= 0 for a, b in zip(got, got[1:]))
    assert got == [orc.distance_bucket(n, rows, far) for n in range(top + 1)]
    for n in range(half, top + 1):                     # the edge rule in exact integers where it is one
        if isinstance(far, int) and far > half:
            k = 0
            while half + k < rows - 1 and n ** (rows - half) * half ** (k + 1) >= far ** (k + 1) * half ** (rows - half):
                k += 1
            assert got[n] == half + k, n
    assert orc.distance_bucket(50 * top, rows, far) == rows - 1


def test_rotary_angles_stay_exact_far_out():
    a = rotary_angles(5000, 8, 777.0, "cpu")
    for p in (0, 1, 4999):
        for i in range(4):
            ang = p * 777.0 ** (-2 * i / 8)
            assert abs(float(a[p, i, 0]) - math.cos(ang)) < 1e-6 and abs(float(a[p, i, 1]) - math.sin(ang)) < 1e-6


# ------------------------------------------------------------------------------- the plain implementation
def test_plain_state_space_carries_its_state():
    g = torch.Generator().manual_seed(0)
    S, H, P, G, N = 11, 4, 3, 2, 5
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)  # noqa: E731
    x, B, C, dt, A, D = r(S, H, P), r(S, G, N), r(S, G, N), r(S, H).abs(), r(H), r(H)
    y, st = orc.state_space(x, B, C, dt, A, D)
    y1, s1 = orc.state_space(x[:4], B[:4], C[:4], dt[:4], A, D)
    y2, s2 = orc.state_space(x[4:], B[4:], C[4:], dt[4:], A, D, s1)
    torch.testing.assert_close(torch.cat([y1, y2]), y)
    torch.testing.assert_close(s2, st)


def test_plain_attention_sees_its_chunk_only():
    cfg = config([attention(chunk=6, mlp=False)], width=40)
    w = orc.random_weights(cfg, 1)
    tok = torch.randint(0, cfg["vocab"], (15,), generator=torch.Generator().manual_seed(1)).tolist()
    full = orc.forward(tok, w, cfg)
    other = list(tok)
    other[5] = (tok[5] + 1) % cfg["vocab"]             # the last token of chunk 0
    changed = (orc.forward(other, w, cfg) - full).abs().amax(-1) > 0
    assert changed.tolist() == [i == 5 for i in range(15)]
    other = list(tok)
    other[6] = (tok[6] + 1) % cfg["vocab"]             # the first of chunk 1
    changed = (orc.forward(other, w, cfg) - full).abs().amax(-1) > 0
    assert changed.tolist() == [6 <= i < 12 for i in range(15)]


def test_plain_sink_takes_weight_only():
    v = torch.randn(4, 3, dtype=torch.float64)
    s = torch.randn(4, dtype=torch.float64)
    a, b = orc.softmax_attend(s, v), orc.softmax_attend(s, v, 1.3)
    f = torch.exp(s).sum() / (torch.exp(s).sum() + math.exp(1.3))
    torch.testing.assert_close(b, a * f)


def test_plain_latent_attention_depends_on_distance_only():
    m = latent(mlp=False)["mixer"]
    q, k = torch.randn(8, dtype=torch.float64), torch.randn(8, dtype=torch.float64)
    at = lambda x, p: orc.rotate_pairs(x, p, m["rot"]["dims"], m["rot"]["base"])  # noqa: E731
    torch.testing.assert_close(at(q, 40) @ at(k, 33), at(q, 7) @ at(k, 0))


def test_prompt_parsing_of_the_command_line():
    from socket_b200.generate import parse_prompts
    assert parse_prompts("5,17,3") == [[5, 17, 3]] and parse_prompts("1,2;3,4") == [[1, 2], [3, 4]]
    for bad in ("", "1,2;3"):
        with pytest.raises(ValueError):
            parse_prompts(bad)
