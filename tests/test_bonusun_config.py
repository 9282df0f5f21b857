"""Bonusun without a GPU: configuration and registry, parts and their constants, the run order, expected tensors, cache and
state needs, refusals, the random-weights mode, and the plain implementation's pieces by hand."""
import copy
import json
import math

import pytest
import torch

import plain_bonusun as P
from bonusun_configs import CONFIGS, SEEDS, make_weights, random_tokens, row_error, tensor_shapes


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
    from dlgo_b200.config import BonusunConfig, config_from_dict, registered_architectures
    assert "Bonusun" in registered_architectures()
    for cfg in CONFIGS.values():
        c = config_from_dict(cfg)
        assert isinstance(c, BonusunConfig)
        assert config_from_dict(json.loads(json.dumps(c.to_dict()))) == c


def test_run_order_repeats_the_span():
    assert [e.layer for e in spec_of(CONFIGS["P"]).order] == [0, 1, 2, 1, 2, 3]
    assert [e.layer for e in spec_of(CONFIGS["Q"]).order] == [0, 1, 2, 3, 4]
    assert [e.layer for e in spec_of(CONFIGS["R"]).order] == [0, 1, 2, 3, 2, 3, 4]
    assert all(e.cache_of is None for e in spec_of(CONFIGS["R"]).order)
    cfg = dict(CONFIGS["P"], loop={"start": 0, "stop": 4, "times": 3})
    assert [e.layer for e in spec_of(cfg).order] == [0, 1, 2, 3] * 3
    cfg = dict(CONFIGS["P"], loop={"start": 3, "stop": 4, "times": 1})
    assert [e.layer for e in spec_of(cfg).order] == [0, 1, 2, 3]


def test_parts_carry_the_file_s_constants():
    spec = spec_of(CONFIGS["P"])
    assert spec.streams == 2 and spec.final_norm.params["bias_name"] == ".b" and spec.head.params["tied_to"] is None
    assert all(l.block == "hyper_prenorm" for l in spec.layers)
    assert all(c.params["result_scale"] == 0.6 for l in spec.layers for c in l.connections.values())
    l0, l1, l2, l3 = spec.layers
    assert l0.mixer.kind == "rglru" and {k: l0.mixer.params[k] for k in ("width", "parts", "conv_taps", "rate")} == \
        {"width": 60, "parts": 3, "conv_taps": 4, "rate": 8.0}
    f = l0.ffn.params
    assert (f["group_count"], f["group_keep"], f["group_top"], f["top"], f["weight_scale"]) == (3, 2, 2, 3, 1.7)
    assert f["score"] == "sigmoid" and f["renormalize"] and f["correction"] and f["shared_gate"]
    assert f["clamp"] == (1.5, 1.702, 1.0) and f["shared_clamp"] == (0.8, 1.702, 1.0) and f["shared_size"] == 24
    (_, a, fa), (_, b, fb) = l1.mixer.params["mixers"]
    assert (a.kind, b.kind, fa, fb) == ("headnorm_attention", "matrix_memory", 0.7, 1.3)
    assert (a.params["qk_dim"], a.params["v_dim"], a.params["num_heads"], a.params["num_kv_heads"], a.params["scale"]) == (24, 40, 6, 2, 0.3)
    assert a.params["sink"] and a.params["window"] is None and b.params["gate_cap"] == 6.0
    pe = spec.position_encodings[a.params["position_encoding"]].params
    assert pe["rotary_dim"] == 12 and pe["theta"] == 5000.0 and pe["scaling"]["factor"] == 4.0
    assert l1.ffn.kind == "two_matrix_mlp" and l1.ffn.params["activation"] == "gelu_tanh"
    assert l2.ffn is None and set(l2.connections) == {"mixer_conn"} and l2.mixer.params["window"] == 37
    assert spec.position_encodings[l2.mixer.params["position_encoding"]].params["scaling"] is None
    assert l3.mixer.params["position_encoding"] is None and l3.mixer.params["window"] is None
    assert l3.ffn.params["shared_size"] is None and l3.ffn.params["shared_clamp"] is None
    assert spec_of(CONFIGS["Q"]).layers[0].mixer.params["mixers"][1][1].params["eps"] == 1e-6


def test_linear_scaling_of_frequencies():
    from dlgo_b200.parts.rope import rotary_frequencies
    plain = rotary_frequencies(12, 5000.0, None)
    assert rotary_frequencies(12, 5000.0, {"rope_type": "linear", "factor": 4.0}) == [f / 4.0 for f in plain]


def test_cache_and_state_needs():
    from dlgo_b200.engine.model import CausalLM
    needs, borrows, states = CausalLM(spec_of(CONFIGS["P"])).cache_needs()
    assert borrows == [None] * 6 and needs[0] is None
    assert [(n.num_kv_heads, n.head_dim, n.window) for n in needs[1:]] == [(2, 40, None), (2, 24, 37), (2, 40, None), (2, 24, 37), (1, 28, None)] \
        or [(n.num_kv_heads, n.window) for n in needs[1:]] == [(2, None), (2, 37), (2, None), (2, 37), (1, None)]
    assert all(n.head_dim >= h for n, h in zip(needs[1:], (40, 24, 40, 24, 28)))
    assert set(states) == {0, 1, 3}
    assert states[0].shape == (60 * (1 + 4),)                                     # S and an input per tap
    n = 3 * (16 * 20 + 16 + 1)
    assert states[1].shape == states[3].shape == (n + -n % 4,)                    # S, n and m per head, whole 16 bytes
    # every pass of the loop has a place of its own
    assert len(CausalLM(spec_of(CONFIGS["R"])).cache_needs()[2]) == 6


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "lru", "type"),
    (("layers", 0, "mixer", "blocks"), 7, "blocks"),
    (("layers", 0, "mixer", "conv"), 0, "conv"),
    (("layers", 1, "mixer", "left", "kv_heads"), 4, "kv_heads"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 7, "rot.dims"),
    (("layers", 1, "mixer", "left", "rot", "dims"), 26, "rot.dims"),
    (("layers", 1, "mixer", "left", "rot", "scaling", "factor"), 0, "factor"),
    (("layers", 1, "mixer", "left", "scale"), None, "scale"),
    (("layers", 1, "mixer", "right", "gate_cap"), -1.0, "gate_cap"),
    (("layers", 1, "mixer", "right"), None, "right"),
    (("layers", 1, "mixer", "right_scale"), None, "right_scale"),
    (("layers", 2, "mixer", "mask", "size"), 0, "size"),
    (("layers", 2, "mixer", "vdim"), None, "vdim"),
    (("layers", 0, "mlp", "router", "top"), 5, "top"),
    (("layers", 0, "mlp", "router", "groups", "count"), 4, "groups"),
    (("layers", 0, "mlp", "router", "groups", "keep"), 4, "groups"),
    (("layers", 0, "mlp", "expert", "limit"), 0, "limit"),
    (("layers", 0, "mlp", "shared", "limit"), None, "limit"),
    (("layers", 0, "mlp", "kind"), "glu", "kind"),
    (("layers", 1, "mlp", "ff"), -1, "ff"),
    (("loop", "stop"), 9, "loop"),
    (("loop", "times"), 0, "loop"),
    (("streams",), 9, "streams"),
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
    from dlgo_b200.config.spec import PartSpec
    from dlgo_b200.parts import FEED_FORWARDS, MIXERS
    unit = dict(hidden_size=8, width=12, parts=3, conv_taps=4)
    MIXERS.build(PartSpec("rglru", unit))
    memory = dict(hidden_size=8, num_heads=2, qk_dim=4, v_dim=4, gate_cap=1.0, eps=1e-5)
    MIXERS.build(PartSpec("matrix_memory", memory))
    experts = dict(hidden_size=8, intermediate_size=8, num_experts=4, top=2, gated=True, activation="silu", group_top=2)
    FEED_FORWARDS.build(PartSpec("routed_experts", experts))
    for reg, kind, base, bad in ((MIXERS, "rglru", unit, dict(parts=5)), (MIXERS, "rglru", unit, dict(conv_taps=0)),
                                 (MIXERS, "matrix_memory", memory, dict(gate_cap=0.0)),
                                 (MIXERS, "matrix_memory", memory, dict(qk_dim=513)),
                                 (FEED_FORWARDS, "routed_experts", experts, dict(group_top=3)),
                                 (FEED_FORWARDS, "routed_experts", experts, dict(gated=False, clamp=(1.0, 1.0, 0.0))),
                                 (FEED_FORWARDS, "two_matrix_mlp", dict(hidden_size=8, intermediate_size=8), dict(activation="exp"))):
        with pytest.raises(ValueError):
            reg.build(PartSpec(kind, dict(base, **bad)))


def test_random_weights_mode(tmp_path):
    from dlgo_b200.config import config_from_dict
    from dlgo_b200.weights import write_random_model
    a = write_random_model(config_from_dict(CONFIGS["Q"]), 7, str(tmp_path / "a"))
    cfg, w = P.read_model(a)
    assert cfg["layers"][4]["mixer"] == CONFIGS["Q"]["layers"][4]["mixer"]
    assert {n: tuple(t.shape) for n, t in w.items()} == tensor_shapes(CONFIGS["Q"])
    assert torch.isfinite(P.forward(cfg, w, [1, 2, 3])).all()


# ------------------------------------------------------------------ the plain implementation by hand
def test_plain_norm_and_streams():
    u = torch.tensor([[1.0, 3.0]])
    assert torch.allclose(P.layer_norm(u, torch.tensor([2.0, 5.0]), torch.tensor([0.5, 0.0]), 0.0), torch.tensor([[-1.5, 5.0]]))
    X = torch.tensor([[[1.0]], [[10.0]]])
    w = {"c.in": torch.tensor([2.0, 3.0]), "c.out": torch.tensor([1.0, -1.0]), "c.mix": torch.tensor([[1.0, 4.0], [0.0, 2.0]])}
    seen = []
    Y = P.through_streams(X, w, "c.", 0.5, lambda u: seen.append(u) or u * 10)
    assert seen[0].item() == 32.0
    assert Y.flatten().tolist() == [1.0 + 160.0, 4.0 + 20.0 - 160.0]       # mix is [from, to]


def test_plain_attention_window_and_sink():
    q = k = torch.zeros(4, 1, 1)
    v = torch.tensor([1.0, 2.0, 4.0, 8.0]).view(4, 1, 1)
    o = P.attend(q, k, v, 1.0, torch.tensor([0.0]), 2).flatten()             # the sink weighs as much as a key
    assert torch.allclose(o, torch.tensor([1 / 2, 3 / 3, 6 / 3, 12 / 3]))
    o = P.attend(q, k, v, 1.0, torch.tensor([math.log(6.0)]), None).flatten()
    assert torch.allclose(o, torch.tensor([1 / 7, 3 / 8, 7 / 9, 15 / 10]))


def test_plain_rotation_of_the_first_entries():
    t = torch.zeros(2, 1, 6)
    t[1, 0] = torch.tensor([1.0, 0.0, 0.0, 2.0, 5.0, 6.0])
    r = P.rotate_halves(t, {"base": 100.0, "dims": 4, "scaling": {"factor": 2.0}})
    c0, s0, c1, s1 = math.cos(0.5), math.sin(0.5), math.cos(0.05), math.sin(0.05)
    assert torch.allclose(r[1, 0], torch.tensor([c0, -2 * s1, s0, 2 * c1, 5.0, 6.0]), atol=1e-6)


def test_plain_matrix_memory():
    q, k, v = torch.tensor([[[2.0]], [[1.0]]]), torch.tensor([[[1.0]], [[3.0]]]), torch.tensor([[[5.0]], [[7.0]]])
    i, f = torch.tensor([[-2.0], [1.0]]), torch.tensor([[-0.5], [-0.1]])
    o, (S, n, m) = P.matrix_memory(q, k, v, i, f)
    m1 = -0.5                                                                # max(-0.5 + 0, -2)
    s1, n1 = math.exp(-2 - m1) * 5, math.exp(-2 - m1)
    assert math.isclose(float(o[0, 0, 0]), 2 * s1 / (max(2 * n1, math.exp(-m1)) + 1e-6), rel_tol=1e-6)
    s2, n2 = math.exp(-0.1 + m1 - 1) * s1 + 21, math.exp(-0.1 + m1 - 1) * n1 + 3
    assert math.isclose(float(o[1, 0, 0]), s2 / (max(n2, math.exp(-1.0)) + 1e-6), rel_tol=1e-6)
    assert torch.allclose(torch.stack([S[0, 0, 0], n[0, 0], m[0]]), torch.tensor([s2, n2, 1.0]))


def test_plain_recurrent_unit():
    x = torch.tensor([[1.0], [10.0]])
    assert P.causal_conv(x, torch.tensor([[2.0, 3.0]]), torch.tensor([0.5]))[:, 0].tolist() == [3.5, 32.5]
    u, r, i, lam = torch.tensor([[2.0], [3.0]]), torch.tensor([[0.5], [0.25]]), torch.tensor([[1.0], [0.5]]), torch.tensor([0.0])
    S = P.gated_recurrence(u, r, i, lam)
    a0, a1 = math.exp(-4 * math.log(2)), math.exp(-2 * math.log(2))
    s0 = math.sqrt(1 - a0 * a0) * 2.0
    assert torch.allclose(S.flatten(), torch.tensor([s0, a1 * s0 + math.sqrt(1 - a1 * a1) * 0.5 * 3.0]))
    w = torch.tensor([[[1.0, 2.0], [0.0, 1.0]], [[3.0, 0.0], [0.0, 0.5]]])
    assert P.block_linear(torch.tensor([[1.0, 10.0, 2.0, 4.0]]), w, torch.zeros(2, 2))[0].tolist() == [21.0, 10.0, 6.0, 2.0]


def test_plain_router_and_expert():
    h = torch.eye(6)[:1]
    router, corr = torch.zeros(6, 6), torch.tensor([-2.0, -2.0, -1.0, -2.5, -1.9, -1.2])
    router[:, 0] = torch.tensor([3.0, 0.0, 0.0, 2.8, 1.0, -1.0])
    s = torch.sigmoid(router[:, 0])
    idx, wt = P.route(h, router, corr, {"experts": 6, "top": 2, "scale": 2.0})
    assert idx[0].tolist() == [2, 5] and torch.allclose(wt[0], 2 * s[[2, 5]] / s[[2, 5]].sum())
    # groups of two, scored by the sum of both
    c = s + corr
    keep = int(c.view(3, 2).sum(1).argmax())
    for kept in (1, 2):
        idx, _ = P.route(h, router, corr, {"experts": 6, "top": 2 * kept, "scale": 1.0, "groups": {"count": 3, "keep": kept}})
        assert {2 * keep, 2 * keep + 1} <= set(idx[0].tolist()) and len(set(e // 2 for e in idx[0].tolist())) == kept
    y = P.clamped_expert(torch.tensor([[1.0]]), torch.tensor([[9.0], [-9.0]]), torch.tensor([[-5.0], [0.5]]), torch.tensor([[1.0, 1.0]]), 2.0)
    g = 2.0 / (1 + math.exp(-3.404)) * (-2.0 + 1) + -9.0 / (1 + math.exp(1.702 * 9)) * 1.5
    assert math.isclose(float(y), g, rel_tol=1e-5)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_plain_model_is_causal_and_every_tensor_counts(name):
    cfg = CONFIGS[name]
    w = {k: v.double() for k, v in make_weights(cfg, SEEDS[name]).items()}
    tokens = random_tokens(24, cfg["vocab"], 3)
    ref = P.forward(cfg, w, tokens)
    other = P.forward(cfg, w, tokens[:12] + [(t + 1) % cfg["vocab"] for t in tokens[12:]])
    assert torch.allclose(ref[:12], other[:12], atol=1e-9) and not torch.allclose(ref[12:], other[12:], atol=1e-3)
    for n in w:
        # (what a layer norm takes out again: the scale of one stream, or of streams that are still equal)
        if n == "embed" or ".mlp.e" in n or (n.endswith(".in") and (cfg["streams"] == 1 or n == "l0.hc1.in")):
            continue
        w2 = dict(w)
        w2[n] = w[n].clone()
        w2[n][0] *= 5.0 if n.endswith("correction") else 1.5
        moved = float(row_error(P.forward(cfg, w2, tokens), ref).max())
        # (one expert: its router has nothing to choose, and its weight is 1)
        one = (n.endswith("router") or n.endswith("correction")) and w[n].shape[0] == 1
        assert (moved < 1e-9) if one else (moved > 1e-6), (n, moved)
