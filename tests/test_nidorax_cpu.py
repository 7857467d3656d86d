"""CPU tests of the Nidorax design: configuration, layout, tensor names, caches and states, frequencies, and the plain
implementation's own consistency (tests/plain_nidorax.py is the oracle of the GPU tests)."""
import copy
import math

import pytest
import torch

import plain_nidorax as P
from nidorax_tiny import CONFIGS, make_weights, random_config, yarn
from tiny import random_tokens

from llm_b200.config.model_config import ConfigError, parse_config
from llm_b200.engine.model import Model, collect_parameters


def test_config_reads_every_size_and_constant():
    cfg, _ = CONFIGS["A"]
    arch, c = parse_config(cfg)
    assert arch.name == "Nidorax" and (c.width, c.vocab, c.postln_alpha, c.norm_eps) == (72, 210, 1.5, 1e-5)
    assert [l["type"] for l in c.layers] == ["lightning"] + ["latent_attention"] * 4
    assert c.layers[0]["mixer"] == {"heads": 3, "dim": 16, "vdim": 24, "decay": (0.4, 0.9, 0.995)}
    m = c.layers[1]["mixer"]
    assert (m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"]) == (3, 16, 8, 12, 24, 0.3)
    assert (m["rot_dims"], m["rot_base"], m["rot_scaling"]) == (8, 5e4, {"factor": 8.0, "original": 256.0, "fast": 32.0, "slow": 1.0})
    assert [l["mixer"].get("kv_from") for l in c.layers] == [None, None, 1, None, 1]
    assert c.layers[0]["mlp"] == {"kind": "moe", "ff": 24, "experts": 6, "top": 2, "groups": 3, "keep": 2} and c.layers[2]["mlp"] is None


@pytest.mark.parametrize("path,value", [
    (("layers", 0, "type"), "attention"), (("layers", 0, "mixer", "dim"), 0), (("layers", 0, "mixer", "decay"), [0.1, 0.2]),
    (("layers", 0, "mixer", "decay"), [0.1, 0.2, 1.5]), (("layers", 0, "mixer", "decay"), [0.1, 0.2, "x"]),
    (("layers", 1, "mixer", "rot_dim"), 7), (("layers", 1, "mixer", "rot", "dims"), 10), (("layers", 1, "mixer", "rot", "scaling"), 4),
    (("layers", 1, "mixer", "rot", "scaling"), {"factor": 2.0}), (("layers", 1, "mixer", "rot", "scaling", "factor"), 0.0),
    (("layers", 1, "mixer", "scale"), "x"), (("layers", 2, "mixer", "kv_from"), 0), (("layers", 2, "mixer", "kv_from"), 3),
    (("layers", 4, "mixer", "kv_from"), 2), (("layers", 2, "mixer", "kv_rank"), 25), (("layers", 2, "mixer", "rot", "base"), 10.0),
    (("layers", 0, "mlp", "kind"), "dense"), (("layers", 0, "mlp", "router", "top"), 5), (("layers", 0, "mlp", "router", "groups", "count"), 4),
    (("layers", 0, "mlp", "router", "groups", "keep"), 4), (("layers", 0, "mlp", "expert", "ff"), 0), (("width",), -1),
    (("norm", "eps"), "x"), (("postln_alpha",), None)])
def test_config_errors_name_the_key(path, value):
    cfg = copy.deepcopy(CONFIGS["A"][0])
    at = cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError):
        parse_config(cfg)


@pytest.mark.parametrize("missing", ["postln_alpha", "norm", "layers", "width", "vocab"])
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


def test_layout_caches_and_states():
    arch, c = parse_config(CONFIGS["A"][0])
    spec = arch.build_spec(c)
    assert [l.block for l in spec.layers] == ["postnorm"] * 5 and [l.cache_of for l in spec.layers] == [None, None, 1, None, 1]
    assert all(l.params == {"alpha": 1.5} for l in spec.layers) and spec.head.params["tied_to"] == "embed"
    model = Model(spec, torch.float32, torch.device("cpu"))
    # two layers keep latents (one page group, one vector per token, no value pages); three read them
    assert len(model.cache_instances) == 2 and len(model.group_keys) == 1
    assert [(o.cache_instance, o.owns_cache) for o in model.occurrences] == [(None, True), (0, True), (0, False), (1, True), (0, False)]
    need = model.blocks[1].mixer.cache_need()
    assert (need.kind, need.num_kv_heads, need.head_dim, need.values) == ("full", 1, 24 + 8, False)
    assert [s.shape for s in model.state_needs] == [(3 * 16 * 24,)]
    # bfloat16 rows are padded to a width that the tensor-core kernels take
    model = Model(spec, torch.bfloat16, torch.device("cpu"))
    assert model.blocks[1].mixer.row_width == 64 and Model(parse_config(CONFIGS["B"][0])[0].build_spec(parse_config(CONFIGS["B"][0])[1]),
                                                          torch.bfloat16, torch.device("cpu")).blocks[0].mixer.row_width == 128


def test_a_model_of_recurrences_keeps_no_cache():
    arch, c = parse_config(CONFIGS["E"][0])
    model = Model(arch.build_spec(c), torch.float32, torch.device("cpu"))
    assert not model.cache_instances and len(model.state_needs) == 2


@pytest.mark.parametrize("dims,base,scaling", [(8, 1e4, yarn(4.0, 64, 16.0, 2.0)), (64, 5e5, yarn(40.0, 4096)), (2, 10.0, yarn(2.0, 50)),
                                               (32, 1e4, yarn(1.0, 2048)), (12, 100.0, yarn(8.0, 16, 32.0, 4.0)), (16, 1e4, None)])
def test_frequencies_and_their_factor_on_cos_and_sin(dims, base, scaling):
    from llm_b200.parts.position import PairRotary
    part = PairRotary(dims, base, scaling, layout="halves", scaling_kind="yarn")
    freqs, amp = P.yarn(dims, base, scaling)
    assert torch.allclose(torch.from_numpy(part.host_frequencies()).double(), torch.tensor(freqs, dtype=torch.float64), rtol=1e-6, atol=0)
    assert abs(part.amplitude - amp) < 1e-12


def test_frequencies_over_the_three_ranges():
    """Fast pairs keep their frequency, slow pairs are divided by the factor, and the ramp lies between."""
    freqs, amp = P.yarn(64, 1e4, yarn(16.0, 1024))
    plain = [1e4 ** (-2.0 * i / 64) for i in range(32)]
    ratio = [f / p for f, p in zip(freqs, plain)]
    assert ratio[0] == 1.0 and abs(ratio[-1] - 1 / 16) < 1e-12 and all(a >= b - 1e-12 for a, b in zip(ratio, ratio[1:]))
    assert any(1 / 16 + 1e-6 < r < 1 - 1e-6 for r in ratio) and abs(amp - (0.1 * math.log(16.0) + 1.0)) < 1e-12


def test_unknown_scaling_is_an_error():
    from llm_b200.parts.position import PairRotary
    with pytest.raises(ValueError):
        PairRotary(8, 1e4, yarn(2.0, 50), scaling_kind="linear")
    with pytest.raises(ValueError):
        PairRotary(8, 1e4, {"factor": 2.0, "original": 50, "fast": 32.0}, scaling_kind="yarn")


# ---- the plain implementation against itself -------------------------------------------------------------
def test_plain_recurrence_agrees_with_the_sum_over_earlier_tokens():
    torch.manual_seed(0)
    T, H, D, V = 12, 3, 5, 4
    f64 = lambda *s: torch.randn(*s, dtype=torch.float64)
    q, k, v, decay = f64(T, H, D), f64(T, H, D), f64(T, H, V), [0.0, 0.7, 1.0]
    got, _ = P.lightning_recurrence(q, k, v, decay)
    for h in range(H):
        for t in range(T):
            want = sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert torch.allclose(got[t, h], want, rtol=1e-10, atol=1e-10)


def test_plain_scores_depend_on_distance_alone():
    """Turning queries and keys by their positions leaves a score that only the distance enters."""
    torch.manual_seed(1)
    freqs, amp = P.yarn(8, 1e4, yarn(4.0, 64))
    q, k = torch.randn(8, dtype=torch.float64), torch.randn(8, dtype=torch.float64)
    at = lambda x, p: P.rotate_halves(x.unsqueeze(0), torch.tensor([p]), freqs, amp)[0]
    assert abs(float(at(q, 30) @ at(k, 11)) - float(at(q, 219) @ at(k, 200))) < 1e-10
    assert abs(float(at(q, 5) @ at(k, 5)) - amp * amp * float(q @ k)) < 1e-10


def test_router_strikes_out_groups_and_renormalises():
    """An expert outside the kept groups cannot be chosen whatever its score; negative choice scores inside still can; the
    weights are the scores without the correction and sum to one."""
    x = torch.zeros(1, 4, dtype=torch.float64)
    p = {"router": torch.zeros(6, 4, dtype=torch.float64), "correction": torch.tensor([-0.5, -0.9, 0.3, -2.0, 0.2, 0.1], dtype=torch.float64)}
    ids, w, _ = P.route(x, p, {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}})
    assert ids[0].tolist() == [2, 4, 5] and torch.allclose(w, torch.full((1, 3), 1 / 3, dtype=torch.float64))
    ids, _, _ = P.route(x, p, {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}})
    assert ids[0].tolist() == [2, 3]
    p["router"][1, 0], x[0, 0] = 1.0, 2.0
    ids, w, _ = P.route(x, p, {"experts": 6, "top": 6, "groups": {"count": 1, "keep": 1}})
    assert sorted(ids[0].tolist()) == list(range(6)) and abs(float(w.sum()) - 1) < 1e-12


def test_stored_norm_weight_of_zero_is_a_gain_of_one():
    x = torch.randn(3, 16, dtype=torch.float64)
    assert torch.allclose(P.centred_norm(x, torch.zeros(16, dtype=torch.float64), 1e-6), P.rms_unit(x, 1e-6))
    from llm_b200.parts.norm import RMSNorm
    part = RMSNorm(16, 1e-6, weight_name="", centred=True, prefix="n", dtype=torch.float32, device=torch.device("cpu"))
    part.bind({"n": torch.full((16,), 0.25)})
    assert torch.equal(part.gain, torch.full((16,), 1.25))


@pytest.mark.parametrize("seed", range(10))
def test_random_configurations_parse_and_name_their_tensors(seed):
    cfg = random_config(3000 + seed, large=seed % 2 == 1)
    w = make_weights(cfg, seed=seed)
    assert sorted(collect_parameters(cfg)) == sorted(w)
    if seed % 2 == 0:
        logits = P.forward(cfg, {k: v.double() for k, v in w.items()}, random_tokens(17, cfg["vocab"], seed))
        assert logits.shape == (17, cfg["vocab"]) and bool(torch.isfinite(logits).all())
