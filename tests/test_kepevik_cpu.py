"""CPU tests of the Kepevik design: configuration, layout, tensor names, the state row, and the plain implementation's own
consistency (tests/plain_kepevik.py is the oracle of the GPU tests)."""
import copy
import math

import pytest
import torch

import plain_kepevik as P
from kepevik_tiny import CONFIGS, make_weights, random_config
from tiny import random_tokens

from llm_b200.config.model_config import ConfigError, parse_config
from llm_b200.csrc import ops
from llm_b200.engine.model import Model, collect_parameters


def f64(*shape, seed=[0]):
    seed[0] += 1
    return torch.randn(*shape, dtype=torch.float64, generator=torch.Generator().manual_seed(seed[0]))


def test_config_reads_every_size_and_constant():
    cfg, _ = CONFIGS["A"]
    arch, c = parse_config(cfg)
    assert arch.name == "Kepevik" and c.width == 64 and c.vocab == 200 and c.embedding_scale == 2.0 and c.norm_eps == 1e-5
    assert [l["type"] for l in c.layers] == ["mlstm", "parallel", "mlstm"]
    assert c.layers[0]["mixer"] == {"heads": 2, "dim": 16, "vdim": 24, "gate_cap": 6.0}
    par = c.layers[1]["mixer"]
    assert par["left"] == {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 16, "scale": 0.3, "rot_dims": 8, "rot_base": 10000.0}
    assert par["right"] == {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 8, "conv": 3}
    assert (par["left_scale"], par["right_scale"]) == (0.7, 0.9)
    assert c.layers[0]["mlp"] == {"kind": "dense", "ff": 40}
    assert c.layers[1]["mlp"] == {"kind": "moe", "ff": 24, "experts": 6, "identity": 2, "top": 2, "shared": 32}


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "type"), "conv"), (("layers", 0, "mixer", "dim"), 0), (("layers", 0, "mixer", "gate_cap"), 0.0),
    (("layers", 0, "mixer", "vdim"), -1), (("layers", 1, "mixer", "left", "kv_heads"), 3), (("layers", 1, "mixer", "left", "vdim"), 8),
    (("layers", 1, "mixer", "left", "rot", "dims"), 7), (("layers", 1, "mixer", "left", "rot", "dims"), 18),
    (("layers", 1, "mixer", "left", "rot", "base"), 0.0), (("layers", 1, "mixer", "right", "kv_heads"), 3),
    (("layers", 1, "mixer", "right", "conv"), 17), (("layers", 1, "mixer", "right", "conv"), 0), (("layers", 1, "mixer", "left_scale"), "x"),
    (("layers", 1, "mlp", "kind"), "sparse"), (("layers", 1, "mlp", "expert", "ff"), 0), (("layers", 1, "mlp", "router", "top"), 9),
    (("layers", 1, "mlp", "router", "identity"), -1), (("layers", 1, "mlp", "router", "experts"), 300), (("layers", 1, "mlp", "shared", "ff"), 0),
    (("layers", 0, "mlp", "ff"), 0), (("layers", 0, "mlp"), 3), (("width",), -1), (("norm", "eps"), "x"), (("embedding", "scale"), "x")])
def test_config_errors_name_the_key(path, value):
    cfg = copy.deepcopy(CONFIGS["A"][0])
    at = cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError):
        parse_config(cfg)


@pytest.mark.parametrize("missing", ["embedding", "norm", "layers", "width", "vocab"])
def test_config_requires_its_keys(missing):
    cfg = copy.deepcopy(CONFIGS["B"][0])
    del cfg[missing]
    with pytest.raises(ConfigError):
        parse_config(cfg)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_tensor_names_and_shapes_are_those_of_the_weights(name):
    cfg, _ = CONFIGS[name]
    w = make_weights(cfg, seed=1)
    want = collect_parameters(cfg)
    assert sorted(want) == sorted(w)
    for n, info in want.items():
        assert info.fits(w[n].shape), (n, info.shape, tuple(w[n].shape))


def test_layout_caches_and_state_rows():
    cfg, _ = CONFIGS["B"]
    arch, c = parse_config(cfg)
    spec = arch.build_spec(c)
    assert [l.block for l in spec.layers] == ["sandwich"] * 4 and spec.order == (0, 1, 2, 3)
    model = Model(spec, torch.float32, torch.device("cpu"))
    # the attention's keys and values: two page sets of equal heads and sizes; the mlstm layers keep no keys
    assert len(model.cache_instances) == 2 and len(model.state_needs) == 4 and model.group_keys == [("full", None, 0)]
    need = model.blocks[0].mixer.cache_need()
    assert (need.kind, need.num_kv_heads, need.head_dim, need.value_dim, need.values) == ("full", 2, 64, 64, True)
    # delta rule: three inputs of the convolution over [q | k | v], then S
    assert model.state_needs[0].shape == (3 * (2 * 64 + 4 * 32) + 4 * 64 * 32,)
    # mlstm: S, then n and m once per block of 64 value columns
    assert model.state_needs[1].shape == (4 * 32 * 72 + 4 * 2 * 32 + 4 * 2,)
    assert model.state_needs[3].shape == (2 * 64 * 128 + 2 * 2 * 64 + 2 * 2,)


@pytest.mark.parametrize("heads,dim,vdim", [(1, 1, 1), (3, 7, 67), (2, 64, 64), (5, 10, 129)])
def test_state_row_of_the_matrix_memory_has_room_for_its_parts(heads, dim, vdim):
    n_off, m_off, size = ops.mlstm_state(heads, dim, vdim)
    blocks = -(-vdim // 64)
    assert n_off >= heads * dim * vdim and m_off >= n_off + heads * blocks * dim and size >= m_off + heads * blocks
    assert n_off % 4 == m_off % 4 == size % 4 == 0


def test_stacked_input_product_of_the_delta_rule_splits_as_its_parts():
    """Ranks off the grid of 8: zero rows pad them, and the second factors have zero columns there."""
    from llm_b200.parts.base import build_part
    from llm_b200.models.spec import PartSpec
    W, H, G, D, V, ra, rg = 24, 3, 1, 6, 5, 5, 9
    part = build_part("mixer", PartSpec("gated_delta", {
        "hidden_size": W, "num_heads": H, "num_qk_heads": G, "head_dim": D, "value_dim": V, "taps": 2, "eps": 1e-6,
        "channel_decay": True, "low_rank_gate": True}, "x"), torch.float32, torch.device("cpu"))
    sizes = {"a1": (ra, W), "a2": (H * D, ra), "g1": (rg, W), "g2": (H * V, rg)}
    w = {n: torch.randn(sizes.get(n[2:], info.shape)) for n, info in part.parameters().items()}
    part.bind(w)
    h = torch.randn(4, W)
    proj = h @ part.w_in.T
    assert proj.shape[1] % 8 == 0 and all(s.start % 8 == 0 for s in part.cols.values())
    qkv = torch.cat([w["x.q"], w["x.k"], w["x.v"]])
    assert torch.allclose(proj[:, :part.conv_channels], h @ qkv.T, atol=1e-5)
    assert torch.allclose(proj[:, part.cols["b"]], h @ w["x.b"].T, atol=1e-5)
    assert torch.allclose(proj[:, part.cols["a1"]] @ part.w_a2.T, h @ w["x.a1"].T @ w["x.a2"].T, atol=1e-4)
    assert torch.allclose(proj[:, part.cols["g1"]] @ part.w_g2.T, h @ w["x.g1"].T @ w["x.g2"].T, atol=1e-4)
    w["x.a2"] = torch.randn(H * D, ra + 1)
    with pytest.raises(ValueError):
        part.bind(w)


def test_plain_matrix_memory_agrees_with_its_closed_form():
    """The running-maximum recurrence against sums written out over all earlier tokens without one."""
    T, H, D, V = 11, 2, 5, 3
    q, k, v = f64(T, H, D), f64(T, H, D), f64(T, H, V)
    i, f = 3 * f64(T, H), P.log_sigmoid(f64(T, H))
    got = P.mlstm_scan(q, k, v, i, f)
    F = f.cumsum(0)
    for t in range(T):
        for h in range(H):
            wgt = torch.exp(i[:t + 1, h] + F[t, h] - F[:t + 1, h])
            s = (k[:t + 1, h] @ q[t, h]) * wgt
            m = max(float(F[t, h]), float((i[:t + 1, h] + F[t, h] - F[:t + 1, h]).max()))
            want = (s.unsqueeze(1) * v[:t + 1, h]).sum(0) / (max(abs(float(s.sum())), 1.0) + 1e-6 * math.exp(m))
            assert torch.allclose(got[t, h], want, rtol=1e-9, atol=1e-12)


def test_plain_delta_rule_decays_each_channel_on_its_own():
    """No key ever written again: what is read back is the first value through the decays of the channels it was written along."""
    T, D, V = 6, 4, 3
    k, q = torch.zeros(T, 1, D, dtype=torch.float64), f64(T, 1, D)
    k[0, 0] = f64(D)
    v, decay = f64(T, 1, V), torch.rand(T, 1, D, dtype=torch.float64)
    out = P.delta_scan(q, k, v, torch.full((T, 1), 0.7, dtype=torch.float64), decay)
    for t in range(T):
        reach = decay[1:t + 1, 0].prod(dim=0) * k[0, 0]
        assert torch.allclose(out[t, 0], (reach @ q[t, 0]) * 0.7 * v[0, 0])


def test_plain_rotation_turns_halves_against_each_other():
    x = f64(9, 2, 10)
    y = P.rotate_halves(x, 6, 50.0)
    assert torch.allclose(y[..., 6:], x[..., 6:]) and torch.allclose(y[0], x[0])
    for i in range(3):
        a = 7 * 50.0 ** (-2.0 * i / 6)
        assert torch.allclose(y[7, 1, i], x[7, 1, i] * math.cos(a) - x[7, 1, i + 3] * math.sin(a))
        assert torch.allclose(y[7, 1, i + 3], x[7, 1, i + 3] * math.cos(a) + x[7, 1, i] * math.sin(a))


def test_plain_router_counts_identity_experts_in_the_softmax_and_passes_their_input():
    h = f64(5, 4)
    p = {"router": torch.zeros(3, 4, dtype=torch.float64), "correction": torch.tensor([0.0, -5.0, 1.0], dtype=torch.float64)}
    ids, wts, _ = P.route(h, p, {"experts": 2, "identity": 1, "top": 1})
    assert ids.flatten().tolist() == [2] * 5 and torch.allclose(wts, torch.full((5, 1), 1 / 3, dtype=torch.float64))
    mlp = {"router": {"experts": 2, "identity": 1, "top": 1}}
    assert torch.allclose(P.moe_ff(h, p, mlp), h / 3)


@pytest.mark.parametrize("seed", range(8))
def test_random_configurations_parse_and_name_their_tensors(seed):
    cfg = random_config(3000 + seed)
    w = make_weights(cfg, seed=seed)
    assert sorted(collect_parameters(cfg)) == sorted(w)
    logits = P.forward(cfg, {k: v.double() for k, v in w.items()}, random_tokens(17, cfg["vocab"], seed))
    assert logits.shape == (17, cfg["vocab"]) and bool(torch.isfinite(logits).all())
