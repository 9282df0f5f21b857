"""Zetavik without a GPU: configuration and registry, parts and their constants, expected tensors, cache and state needs,
refusals, the random-weights mode, and the plain implementation's pieces by hand."""
import copy
import json
import math

import pytest
import torch

import plain_zetavik as P
from zetavik_configs import CONFIGS, SEEDS, dense, lat, layer, lin, make_weights, model, moe, random_tokens, row_error, ssm, tensor_shapes


def spec_of(cfg):
    from dlgo_b200.config import config_from_dict
    return config_from_dict(cfg).architecture_spec()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_expected_tensors_are_the_design_s(name):
    from dlgo_b200.engine.model import CausalLM
    m = CausalLM(spec_of(CONFIGS[name]))
    got = {n: tuple(ps.shape) for n, ps in m.expected_tensors().items()}
    assert got == tensor_shapes(CONFIGS[name])


def test_registry_and_round_trip():
    from dlgo_b200.config import ZetavikConfig, config_from_dict, registered_architectures
    assert "Zetavik" in registered_architectures()
    for cfg in CONFIGS.values():
        c = config_from_dict(cfg)
        assert isinstance(c, ZetavikConfig)
        assert config_from_dict(json.loads(json.dumps(c.to_dict()))) == c


def test_parts_carry_the_file_s_constants():
    spec = spec_of(CONFIGS["P"])
    assert [l.block for l in spec.layers] == ["parallel_prenorm"] * 4
    assert all(set(l.norms) == {"mixer_norm"} and l.norms["mixer_norm"].kind == "layernorm" for l in spec.layers)
    assert spec.head.params["tied_to"] == "embed" and spec.final_norm.kind == "layernorm"
    l0, l1, l2, l3 = spec.layers
    a = l0.mixer.params
    assert l0.mixer.kind == "latent_attention" and (a["q_rank"], a["kv_rank"], a["rope_dim"], a["qk_dim"], a["v_dim"]) == (28, 40, 8, 24, 20)
    assert a["head_gate"] and a["scale"] == 0.25
    pe = spec.position_encodings[a["position_encoding"]].params
    assert pe["rotary_dim"] == 8 and pe["theta"] == 500.0 and pe.get("pairing", "split_half") == "split_half"
    f = l0.ffn.params
    assert (f["weight_scale"], f["group_count"], f["group_keep"], f["shared_size"], f["top"]) == (1.5, 3, 2, 24, 3)
    assert f["score"] == "softmax" and not f["renormalize"] and f["gated"]
    s = l1.mixer.params
    assert l1.mixer.kind == "mamba2" and l1.ffn is None
    assert (s["num_heads"], s["v_dim"], s["state_size"], s["num_groups"], s["conv_taps"], s["norm_groups"]) == (6, 12, 24, 3, 3, 3)
    assert l2.mixer.kind == "lightning_attention" and l2.mixer.params["decay"] == (0.99, 0.93) and l2.ffn.kind == "relu2_mlp"
    assert l3.mixer.params["eps"] == 1e-5 and spec_of(CONFIGS["Q"]).layers[0].mixer.params["eps"] == 1e-6
    # absent groups and shared expert: one group, none
    f = spec_of(CONFIGS["Q"]).layers[0].ffn.params
    assert (f["group_count"], f["group_keep"], f["shared_size"], f["weight_scale"]) == (1, 1, None, 0.7)


def test_cache_and_state_needs():
    from dlgo_b200.engine.model import CausalLM
    needs, borrows, states = CausalLM(spec_of(CONFIGS["P"])).cache_needs()
    assert borrows == [None] * 4 and needs[1] is None and needs[2] is None and needs[3] is None
    assert (needs[0].planes, needs[0].head_dim, needs[0].num_kv_heads, needs[0].window) == (1, 48, 1, None)   # latent 40 + rotated 8
    assert set(states) == {1, 2, 3}
    assert states[1].shape == (6 * 24 * 12 + 2 * (6 * 12 + 2 * 3 * 24),)
    assert states[2].shape == (2, 32, 40)
    assert states[3].shape == (3 * 20 * 10 + 4 * (3 * 10 + 2 * 20),)
    # a row is rounded up to whole 16 bytes; one tap keeps no inputs
    needs, _, states = CausalLM(spec_of(CONFIGS["Q"])).cache_needs()
    assert states[0].shape == (36,)                                  # 1 x 5 x 7 = 35
    assert (needs[1].head_dim, needs[3].head_dim) == (13, 28)


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "mamba", "type"),
    (("layers", 1, "mixer", "groups"), 4, "groups"),
    (("layers", 1, "mixer", "norm_groups"), 7, "norm_groups"),
    (("layers", 1, "mixer", "conv"), 0, "conv"),
    (("layers", 1, "mixer", "state"), None, "state"),
    (("layers", 0, "mixer", "rot_dim"), 7, "rot_dim"),
    (("layers", 0, "mixer", "rot"), None, "rot"),
    (("layers", 0, "mixer", "rot", "dims"), 6, "rot"),
    (("layers", 0, "mixer", "q_rank"), 0, "q_rank"),
    (("layers", 2, "mixer", "decay"), [0.5], "decay"),
    (("layers", 0, "mlp", "router", "top"), 5, "top"),
    (("layers", 0, "mlp", "router", "groups", "count"), 4, "groups"),
    (("layers", 0, "mlp", "router", "groups", "keep"), 4, "groups"),
    (("layers", 0, "mlp", "shared", "ff"), 0, "ff"),
    (("layers", 0, "mlp", "kind"), "glu", "kind"),
    (("layers", 2, "mlp", "ff"), -1, "ff"),
    (("norm",), None, "norm"),
    (("width",), 0, "width"),
    (("layers",), [], "layers"),
])
def test_refused_configurations_name_the_key(path, value, word):
    from dlgo_b200.config import ConfigError, config_from_dict
    cfg = copy.deepcopy(CONFIGS["P"])
    at = cfg
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        config_from_dict(cfg)


def test_refused_parts():
    from dlgo_b200.parts import BLOCKS, MIXERS
    from dlgo_b200.config.spec import PartSpec
    base = dict(hidden_size=8, num_heads=4, v_dim=4, state_size=8, num_groups=2, conv_taps=4, norm_groups=2, eps=1e-5)
    MIXERS.build(PartSpec("mamba2", base))
    for bad in (dict(num_groups=3), dict(norm_groups=3), dict(state_size=513), dict(conv_taps=0)):
        with pytest.raises(ValueError):
            MIXERS.build(PartSpec("mamba2", dict(base, **bad)))
    with pytest.raises(ValueError):
        BLOCKS.build(PartSpec("parallel_prenorm", dict(mixer=None, ffn=None, norms={"mixer_norm": object()})))


def test_random_weights_mode(tmp_path):
    from dlgo_b200.config import config_from_dict
    from dlgo_b200.weights import write_random_model
    a = write_random_model(config_from_dict(CONFIGS["Q"]), 7, str(tmp_path / "a"))
    cfg, w = P.read_model(a)
    assert cfg["layers"][0]["mixer"] == CONFIGS["Q"]["layers"][0]["mixer"]
    assert {n: tuple(t.shape) for n, t in w.items()} == tensor_shapes(CONFIGS["Q"])
    assert torch.isfinite(P.forward(cfg, w, [1, 2, 3])).all()


# ------------------------------------------------------------------ the plain implementation by hand
def test_plain_norms():
    u = torch.tensor([[1.0, 3.0]])
    assert torch.allclose(P.layer_norm(u, torch.tensor([2.0, 5.0]), 0.0), torch.tensor([[-2.0, 5.0]]))
    assert torch.allclose(P.layer_norm(u, torch.ones(2), 3.0), torch.tensor([[-0.5, 0.5]]))
    y, z = torch.tensor([[2.0, -1.0, 4.0, 3.0]]), torch.tensor([[0.0, 1.0, -1.0, 2.0]])
    u = (y * z * torch.sigmoid(z))[0]
    want = torch.cat([u[:2] / ((u[:2] ** 2).mean() + 0.1).sqrt(), u[2:] / ((u[2:] ** 2).mean() + 0.1).sqrt()]) * 3.0
    assert torch.allclose(P.gate_then_group_norm(y, z, torch.full((4,), 3.0), 2, 0.1)[0], want)


def test_plain_convolution_and_recurrence():
    u = torch.tensor([[1.0], [10.0], [100.0]])
    y = P.short_conv(u, torch.tensor([[2.0, 3.0]]), torch.tensor([0.5]))
    assert y[:, 0].tolist() == [3.5, 32.5, 320.5]                    # the last tap is the current token's
    # two heads of one value, two groups of one state row: head h reads group h
    x = torch.tensor([[[1.0], [2.0]], [[3.0], [-1.0]]])
    B = torch.tensor([[[1.0], [0.5]], [[2.0], [4.0]]])
    C = torch.tensor([[[1.0], [1.0]], [[10.0], [1.0]]])
    dt = torch.tensor([[0.1, 1.0], [0.2, 2.0]])
    A, D = torch.tensor([1.0, 0.5]), torch.tensor([7.0, 0.0])
    y, S = P.state_space_recurrence(x, B, C, dt, A, D)
    s0, s1 = 0.1 * 1 * 1, 1.0 * 0.5 * 2
    assert math.isclose(float(y[0, 0, 0]), s0 + 7, rel_tol=1e-6) and math.isclose(float(y[0, 1, 0]), s1, rel_tol=1e-6)
    s0 = s0 * math.exp(-0.2) + 0.2 * 2 * 3
    s1 = s1 * math.exp(-1.0) + 2.0 * 4 * -1
    assert math.isclose(float(y[1, 0, 0]), 10 * s0 + 21, rel_tol=1e-5) and math.isclose(float(y[1, 1, 0]), s1, rel_tol=1e-5)
    assert torch.allclose(S.flatten(), torch.tensor([s0, s1]))


def test_plain_rotation_pairs_halves():
    t = torch.zeros(2, 1, 4)
    t[1, 0] = torch.tensor([1.0, 0.0, 0.0, 2.0])
    r = P.rotate_halves(t, 100.0)
    c0, s0, c1, s1 = math.cos(1), math.sin(1), math.cos(0.1), math.sin(0.1)
    assert torch.allclose(r[1, 0], torch.tensor([c0, -2 * s1, s0, 2 * c1]), atol=1e-6)


def test_plain_router():
    h = torch.eye(6)[:1]
    router = torch.zeros(6, 6)
    router[:, 0] = torch.tensor([3.0, 0.0, 2.9, 2.8, 1.0, 2.95])
    s = torch.softmax(router[:, 0], 0)
    idx, wt = P.route(h, router, {"experts": 6, "top": 3, "scale": 2.0})
    assert idx[0].tolist() == [0, 5, 2] and torch.allclose(wt[0], 2 * s[[0, 5, 2]])
    # three groups of two, the best by their largest: (3.0), (2.9), (2.95): the middle one is out
    idx, wt = P.route(h, router, {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}})
    assert idx[0].tolist() == [0, 5, 4] and torch.allclose(wt[0], s[[0, 5, 4]])


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_plain_model_is_causal_and_every_tensor_counts(name):
    cfg = CONFIGS[name]
    w = {k: v.double() for k, v in make_weights(cfg, SEEDS[name]).items()}
    tokens = random_tokens(24, cfg["vocab"], 3)
    ref = P.forward(cfg, w, tokens)
    other = P.forward(cfg, w, tokens[:12] + [(t + 1) % cfg["vocab"] for t in tokens[12:]])
    assert torch.allclose(ref[:12], other[:12], atol=1e-9) and not torch.allclose(ref[12:], other[12:], atol=1e-3)
    for n in w:
        if n == "embed" or ".mlp.e" in n:
            continue
        w2 = dict(w)
        w2[n] = torch.roll(w[n], 1, 0) if w[n].shape[0] > 1 else 0.5 * w[n]
        moved = float(row_error(P.forward(cfg, w2, tokens), ref).max())
        # (one expert: its router has nothing to choose)
        one = n.endswith("router") and w[n].shape[0] == 1
        assert (moved == 0) if one else (moved > 1e-5), (n, moved)
