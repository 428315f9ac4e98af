"""Dogotar without a GPU: the configuration reader, the parts list and tensor names, the cache needs, and the plain
implementation's own consistency where the design says two forms are the same."""

import json
import math

import pytest
import torch

import dogotar_models as dm
import plain_dogotar as plain


def test_config_reader_takes_every_key_and_refuses_what_is_missing():
    from prefixserve_b200.config import DogotarConfig, UnsupportedModelError
    raw = dm.CONFIGS["mixed"]
    cfg = DogotarConfig.from_dicts(raw)
    assert (cfg.vocab, cfg.width, cfg.norm_eps) == (131, 40, 4e-3)
    assert [l.mixer.kind for l in cfg.layers] == ["attention", "parallel", "attention", "parallel", "attention", "attention"]
    assert [l.ff for l in cfg.layers] == [30, 26, None, None, 17, 24] and cfg.value_source() == 2
    a = cfg.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.reach, a.v_mix) == (6, 3, 12, 5, 0.3, 4.0, 20, False)
    assert (a.rot.base, a.rot.dims, a.rot.factor) == (300.0, 6, 2.0)
    assert cfg.layers[2].mixer.softcap is None and cfg.layers[2].mixer.reach is None and cfg.layers[2].mixer.rot.factor is None
    assert cfg.layers[4].mixer.rot is None
    p = cfg.layers[1].mixer
    assert (p.left_scale, p.right_scale, p.left.reach, p.left.softcap) == (1.2, 0.6, 21, 7.0)
    assert (p.right.heads, p.right.dim, p.right.vdim, p.right.gate_cap) == (3, 12, 5, 3.0)
    assert cfg.to_config_json() == raw  # what is written is what was read
    for drop in (("vocab",), ("width",), ("norm", "eps"), ("layers", 0, "mixer", "scale"), ("layers", 0, "mixer", "rot", "base"),
                 ("layers", 0, "mixer", "rot", "scaling", "factor"), ("layers", 1, "mixer", "left"), ("layers", 1, "mixer", "left_scale"),
                 ("layers", 1, "mixer", "right", "gate_cap"), ("layers", 1, "mixer", "right_scale"), ("layers", 0, "mlp", "ff"),
                 ("layers", 0, "mlp", "kind"), ("layers", 3, "type"), ("layers", 3, "mixer", "left", "heads")):
        broken = json.loads(json.dumps(raw))
        at = broken
        for k in drop[:-1]:
            at = at[k]
        del at[drop[-1]]
        with pytest.raises(UnsupportedModelError):
            DogotarConfig.from_dicts(broken)
    for path, value in ((("layers", 0, "mixer", "kv_heads"), 4), (("layers", 0, "type"), "other"), (("layers", 0, "mixer", "rot", "dims"), 5),
                        (("layers", 0, "mixer", "rot", "dims"), 14), (("layers", 0, "mixer", "softcap"), 0.0), (("layers", 0, "mlp", "kind"), "moe"),
                        (("layers", 1, "mixer", "right", "gate_cap"), -1.0), (("layers", 0, "mixer", "mask", "size"), 0),
                        (("layers", 5, "mixer", "vdim"), 4), (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0), (("layers",), [])):
        broken = json.loads(json.dumps(raw))
        at = broken
        for k in path[:-1]:
            at = at[k]
        at[path[-1]] = value
        with pytest.raises(UnsupportedModelError):
            DogotarConfig.from_dicts(broken)


def test_every_tensor_of_a_checkpoint_has_a_part_and_the_cache_holds_what_the_masks_need(tmp_path):
    from prefixserve_b200 import architectures  # noqa: F401
    from prefixserve_b200.config.registry import read_model_folder
    from prefixserve_b200.parts.model import build_model
    for which, cfg in dm.CONFIGS.items():
        weights = dm.tensors(cfg, seed=1)
        arch, typed = read_model_folder(dm.write_folder(tmp_path / which, cfg, weights))
        spec = arch.to_spec(typed)
        model = build_model(spec)
        wanted = {arch.tensor_name(path): tuple(ps.shape) for path, ps in model.param_table().items()}
        assert wanted == {k: tuple(v.shape) for k, v in weights.items()}, which
        first = next((i for i, l in enumerate(cfg["layers"]) if l["mixer"].get("v_mix")), None)
        for i, (lay, need) in enumerate(zip(cfg["layers"], model.cache_needs())):
            m = lay["mixer"]
            a = m if lay["type"] == "attention" else m["left"]
            size = (a.get("mask") or {}).get("size")
            assert need.paged.planes == 1 and need.paged.num_kv_heads == a["kv_heads"] and need.paged.head_dim == a["dim"] + a["vdim"]
            if lay["type"] == "attention":
                assert (need.paged.window, need.paged.chunk, need.state) == (size, None, None)
                assert spec.layers[i].mixer["value_mix"] == (None if not m.get("v_mix") else "source" if i == first else "mixed")
            else:
                b = m["right"]
                held = b["heads"] * (b["dim"] * b["vdim"] + b["dim"] * -(-b["vdim"] // 128) + -(-b["vdim"] // 128))
                assert (need.paged.window, need.paged.chunk) == (None, size) and held <= need.state.shape[0] <= held + 3


def test_what_a_layer_has_no_use_for_may_be_left_in_a_checkpoint_but_nothing_else(tmp_path):
    from prefixserve_b200 import architectures  # noqa: F401
    from prefixserve_b200.config.registry import get_architecture, read_model_folder
    arch, typed = read_model_folder(dm.write_folder(tmp_path / "m", dm.CONFIGS["mixed"], {}))
    assert arch is get_architecture("Dogotar")
    assert arch.ignorable(typed, "l2.norm2") and arch.ignorable(typed, "l3.norm2.b") and arch.ignorable(typed, "l0.mix.vmix")
    assert not arch.ignorable(typed, "l4.mix.vmix")
    assert not arch.ignorable(typed, "l0.norm2") and not arch.ignorable(typed, "l2.norm1") and not arch.ignorable(typed, "l9.norm2")


def test_joined_outputs_put_matrices_side_by_side_with_gaps():
    """The block's one matrix holds every sublayer's columns where their rows go, zeros in between, and the parts let go of
    theirs; sublayers that offer no rows are refused."""
    from prefixserve_b200.config.presets import preset
    from prefixserve_b200.config.registry import get_architecture
    from prefixserve_b200.config.spec import LayerSpec, part
    from prefixserve_b200.parts import Block
    from prefixserve_b200.weights.random_init import random_tensors
    cfg = preset("dogotar-tiny")
    spec = get_architecture("Dogotar").to_spec(cfg)
    g = torch.Generator().manual_seed(0)
    mem = part("matrix_memory", hidden_size=20, num_heads=1, dim=6, vdim=5, gate_cap=3.0, eps=1e-4)
    att = part("head_norm_attention", hidden_size=20, num_heads=3, num_kv_heads=1, dim=4, vdim=7, scale=0.5, eps=1e-4)
    norm = part("layer", size=20, eps=1e-4)
    block = Block(LayerSpec(part("side_by_side_sum", hidden_size=20, branches=(att, mem)), part("mlp", hidden_size=20, intermediate_size=9), norm, norm,
                            arrangement="parallel_rows"))
    w = {}
    for name, p in block.named_parts():
        w[name] = random_tensors(p.param_specs(), 3, std=1.0, dtype=torch.float32)
        p.load(w[name], compute_dtype=torch.float32, device=torch.device("cpu"))
    block.join_outputs()
    assert block.row_columns == [(0, 29), (32, 41)] and block.w_out.shape == (20, 48)
    assert torch.equal(block.w_out[:, :21], w["mixer"]["left.o_proj"]) and torch.equal(block.w_out[:, 24:29], w["mixer"]["right.o_proj"])
    assert torch.equal(block.w_out[:, 32:41], w["ffn"]["down_proj"])
    assert float(block.w_out[:, 21:24].abs().max()) == 0 and float(block.w_out[:, 41:].abs().max()) == 0
    assert block.mixer.w_o is None and block.ffn.w_down is None
    assert all(l.arrangement == "parallel_rows" for l in spec.layers)
    other = Block(LayerSpec(att, part("gated_mlp", hidden_size=20, intermediate_size=8), norm, norm, arrangement="parallel_rows"))
    with pytest.raises(ValueError):
        other.join_outputs()


def test_linear_scaling_of_the_frequencies():
    from prefixserve_b200.parts.position import rope_amplitude, rope_inverse_frequencies
    plain_f, scaled = rope_inverse_frequencies(12, 700.0, None), rope_inverse_frequencies(12, 700.0, {"kind": "linear", "factor": 2.5})
    assert torch.allclose(scaled * 2.5, plain_f) and rope_amplitude({"kind": "linear", "factor": 2.5}) == 1.0
    x = torch.randn(5, 2, 12, generator=torch.Generator().manual_seed(0), dtype=torch.float64)
    angle = 3 * float(scaled[1])
    y = plain.rotate(x, 12, 700.0, 2.5)[3, 0]
    assert torch.allclose(y[1], x[3, 0, 1] * math.cos(angle) - x[3, 0, 7] * math.sin(angle), atol=1e-6)
    assert torch.equal(plain.rotate(x, 4, 700.0, 2.5)[..., 4:], x[..., 4:])


def test_matrix_memory_of_the_plain_model_in_its_attention_form():
    """Weights from sums of log gates, without the running exponent (which only sets the floor of the normalizer); cut in two."""
    g = torch.Generator().manual_seed(0)
    n, H, d, dv = 11, 2, 3, 4
    q, k = (torch.randn(n, H, d, generator=g, dtype=torch.float64) for _ in range(2))
    v = torch.randn(n, H, dv, generator=g, dtype=torch.float64)
    i, f = 3 * torch.randn(n, H, generator=g, dtype=torch.float64), torch.nn.functional.logsigmoid(torch.randn(n, H, generator=g, dtype=torch.float64))
    o = plain.matrix_memory(q, k, v, i, f)
    for t in range(n):
        w = torch.stack([torch.exp(i[j] + f[j + 1: t + 1].sum(0)) * (q[t] * k[j]).sum(-1) for j in range(t + 1)])
        m = torch.zeros(H, dtype=torch.float64)
        for j in range(t + 1):
            m = torch.maximum(f[j] + m, i[j])
        den = torch.maximum(w.sum(0).abs(), torch.ones(H, dtype=torch.float64)) + 1e-6 * torch.exp(m)
        want = torch.einsum("jh,jhv->hv", w, v[: t + 1]) / den[:, None]
        assert torch.allclose(o[t], want, atol=1e-12)


def test_masks_layer_norm_cap_and_gelu_of_the_plain_model():
    m = plain.in_window(9, 4)
    assert m[8].tolist() == [False] * 5 + [True] * 4 and m[2].tolist() == [True] * 3 + [False] * 6
    c = plain.in_chunk(9, 4)
    assert c[3].tolist() == [True] * 4 + [False] * 5 and c[4].tolist() == [False] * 4 + [True] + [False] * 4 and c[7].tolist() == [False] * 4 + [True] * 4 + [False]
    assert torch.equal(plain.in_window(5, None), torch.tril(torch.ones(5, 5, dtype=torch.bool))) and torch.equal(plain.in_chunk(5, None), plain.in_window(5, None))
    x = torch.tensor([[1.0, 5.0, -3.0, 9.0]], dtype=torch.float64)
    one, zero = torch.ones(4, dtype=torch.float64), torch.zeros(4, dtype=torch.float64)
    assert torch.allclose(plain.layer_norm(x, 2 * one, zero + 1, 1e-5), 2 * torch.nn.functional.layer_norm(x, (4,), eps=1e-5) + 1)
    assert torch.allclose(plain.gelu_tanh(x), torch.nn.functional.gelu(x, approximate="tanh"))
    assert torch.allclose(plain.soft_cap(torch.tensor([0.01, 1e6, -1e6], dtype=torch.float64), 5.0), torch.tensor([5 * math.tanh(0.002), 5.0, -5.0], dtype=torch.float64))
    assert torch.equal(plain.mix_values(one, zero, 0.25), 0.75 * one)


def test_random_weights_of_the_presets_describe_themselves(tmp_path):
    from prefixserve_b200.config.presets import preset
    from prefixserve_b200.config.registry import read_model_folder
    from prefixserve_b200.weights import write_random_model
    cfg = preset("dogotar-tiny")
    _, back = read_model_folder(write_random_model(tmp_path / "m", cfg, 0, dtype=torch.bfloat16))
    assert back == cfg
    for name in ("dogotar-2048", "dogotar-4096"):
        assert preset(name).to_config_json()["width"] == int(name.split("-")[1])
