"""Small Zetavik configurations with weights of a useful size, and helpers that run the engine and the plain
implementation on them.  The configurations differ from one another in every size and in the order of their layers, and
include values that are 1 (one head, one group, one tap, one expert, one chosen, a factor of one) or absent (no groups
of experts, no shared expert, a layer without feed-forward) and values that models often make equal but that need not be
(state rows and value columns, key and value sizes, groups of heads and of the norm, the two latents)."""
from __future__ import annotations

import functools
import json
import os
from typing import Dict, Sequence, Tuple

import torch

from bazurax_configs import RowCheck, assert_rows, random_tokens, row_error      # noqa: F401  (shared test helpers)


def ssm(heads, vdim, state, groups=1, conv=4, norm_groups=1):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base=10000.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
            "scale": scale, "rot": {"base": base, "dims": rot_dim}}


def lin(heads, dim, vdim, decay):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, scale=1.0, groups=None, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp=None):
    kind = "mamba2" if "state" in mixer else ("latent_attention" if "kv_rank" in mixer else "lightning")
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def model(vocab, width, layers, eps=1e-5):
    return {"architecture": "Zetavik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


CONFIGS: Dict[str, dict] = {
    # latent attention first; state rows that are no multiple of 16; three groups of heads; convolutions of three and
    # of five taps; a layer without feed-forward; top 3 of 6 in groups of two
    "P": model(150, 72, [
        layer(lat(3, 24, 8, 20, 28, 40, 0.25, 500.0), moe(40, 6, 3, 1.5, (3, 2), 24)),
        layer(ssm(6, 12, 24, 3, 3, 3)),
        layer(lin(2, 32, 40, (0.99, 0.93)), dense(56)),
        layer(ssm(3, 10, 20, 1, 5, 5), dense(88))]),
    # one head everywhere it can be, one tap, sizes that are multiples of nothing; one expert of which one is chosen;
    # as many groups as experts; two latent layers whose cache rows differ; width 46
    "Q": model(97, 46, [
        layer(ssm(1, 7, 5, 1, 1, 1), moe(24, 1, 1, 0.7)),
        layer(lat(1, 8, 4, 40, 33, 9, 0.4, 100.0)),
        layer(lin(1, 20, 12, (0.97,)), moe(18, 5, 2, 1.0, (5, 3))),
        layer(lat(2, 10, 6, 8, 12, 22, 0.35, 3000.0), moe(16, 4, 1, 3.0, (2, 1), 10)),
        layer(ssm(5, 6, 33, 5, 2, 2), dense(30))], eps=1e-6),
    # sizes that the tensor-core kernels take in bfloat16: latent heads of 64 and 128 numbers, states of 64 and 128
    # rows, linear attention of 64 and 128; wide experts; width 128
    "R": model(260, 128, [
        layer(ssm(4, 64, 64, 2, 4, 4), moe(64, 8, 3, 2.5, (4, 2), 96)),
        layer(lat(4, 32, 32, 64, 80, 96, 0.15, 1e6), dense(192)),
        layer(lin(3, 64, 32, (0.96875, 0.998, 0.9)), moe(64, 8, 2, 0.5, (2, 2))),
        layer(ssm(2, 36, 128, 1, 4, 1), dense(96)),
        layer(lat(2, 64, 64, 128, 128, 128, 0.1), moe(48, 12, 4, 1.0, (3, 2), 64)),
        layer(lin(2, 128, 64, (0.99, 0.5)))], eps=1e-6),
}
SEEDS = {"P": 51, "Q": 52, "R": 53}


def tensor_shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of a configuration's tensors, from the design's description (not from the package)."""
    d, V = cfg["width"], cfg["vocab"]
    s: Dict[str, Tuple[int, ...]] = {"embed": (V, d), "final.norm": (d,)}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        s[p + "norm1"] = (d,)
        H, dv, x = m["heads"], m["vdim"], p + "mix."
        if L["type"] == "mamba2":
            inner, gn = H * dv, m["groups"] * m["state"]
            C = inner + 2 * gn
            s.update({x + "in": (inner + C + H, d), x + "conv": (C, m["conv"]), x + "conv.b": (C,), x + "dt_bias": (H,),
                      x + "A_log": (H,), x + "D": (H,), x + "norm": (inner,), x + "o": (d, inner)})
        elif L["type"] == "lightning":
            n = m["dim"]
            s.update({x + "q": (H * n, d), x + "k": (H * n, d), x + "v": (H * dv, d), x + "g": (H * dv, d),
                      x + "norm": (H * dv,), x + "o": (d, H * dv)})
        else:
            n, r, R, Q = m["dim"], m["rot_dim"], m["kv_rank"], m["q_rank"]
            s.update({x + "dq": (Q, d), x + "dq.norm": (Q,), x + "uq": (H * (n + r), Q), x + "dkv": (R + r, d),
                      x + "dkv.norm": (R,), x + "uk": (H * n, R), x + "uv": (H * dv, R), x + "g": (H, d),
                      x + "o": (d, H * dv)})
        mlp, y = L["mlp"], p + "mlp."
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            s.update({y + "up": (mlp["ff"], d), y + "down": (d, mlp["ff"])})
            continue
        E, forms = mlp["router"]["experts"], [(f"e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        s[y + "router"] = (E, d)
        if "shared" in mlp:
            forms.append(("shared.", mlp["shared"]["ff"]))
        for q, f in forms:
            s.update({y + q + "gate": (f, d), y + q + "up": (f, d), y + q + "down": (d, f)})
    return s


def make_weights(cfg: dict, seed: int, sharpen: float = 3.0, mild: bool = False) -> Dict[str, torch.Tensor]:
    """Weights (bfloat16): matrices ~ N(0, 1/in), the embedding N(0, 1), norm weights around 1, taps of visible size on
    every position, biases of visible size, decays from a few tokens to hundreds.  The queries' second matrix is
    multiplied by ``sharpen`` so that the softmax is far from uniform and a wrong, missing or extra key moves the logits;
    routers are scaled up so that choices are not near ties.  ``mild`` (whole models in bfloat16): flatter softmaxes and
    routers, and experts whose results are smaller, so that a router's near tie that rounding tips the other way stays
    one row's affair instead of colouring, through that position's keys and states, every later row of its sequence
    (float32 runs carry the sharp cases)."""
    if mild:
        sharpen = 1.5
    g = torch.Generator().manual_seed(seed)
    w = {}
    shapes = tensor_shapes(cfg)
    for name in sorted(shapes):
        shape = shapes[name]
        r = torch.randn(shape, generator=g)
        if name == "embed":
            t = r
        elif name.endswith(".conv"):
            t = 0.4 * r
            t[:, -1] += 1.0
        elif name.endswith(".conv.b"):
            t = 0.3 * r
        elif name.endswith(".A_log"):
            t = torch.rand(shape, generator=g) * 4.0 - 3.5
        elif name.endswith(".dt_bias"):
            t = -1.0 + r
        elif name.endswith(".D"):
            t = 0.5 + 0.5 * r
        elif "norm" in name:
            t = 1.0 + 0.2 * r
        elif name.endswith(".router"):
            t = (1.0 if mild else 3.0) * r / shape[1] ** 0.5
        elif mild and ".mlp.e" in name and name.endswith(".down"):
            t = 0.25 * r / shape[1] ** 0.5
        elif name.endswith("mix.uq"):
            t = sharpen * r / shape[1] ** 0.5
        else:
            t = r / shape[1] ** 0.5
        w[name] = t.to(torch.bfloat16)
    return w


def config_of(cfg: dict):
    from dlgo_b200.config.zetavik import ZetavikConfig
    return ZetavikConfig.from_dict(cfg)


def write_model(name: str, out_dir: str, sharpen: float = 3.0, mild: bool = False) -> str:
    from dlgo_b200.weights import save_tensors
    os.makedirs(out_dir, exist_ok=True)
    with open(os.path.join(out_dir, "config.json"), "w") as f:
        json.dump(CONFIGS[name], f)
    save_tensors(os.path.join(out_dir, "model.safetensors"), make_weights(CONFIGS[name], SEEDS[name], sharpen, mild=mild))
    return out_dir


@functools.lru_cache(maxsize=64)
def _plain_cached(model_dir: str, tokens: tuple) -> torch.Tensor:
    import plain_zetavik as P
    cfg, w = P.read_model(model_dir, torch.float64)
    return P.forward(cfg, w, list(tokens)).to(torch.float32)


def plain_logits(model_dir: str, tokens: Sequence[int]) -> torch.Tensor:
    """Logits [T, vocab] of the plain implementation (float64 arithmetic) for one whole sequence."""
    return _plain_cached(model_dir, tuple(int(t) for t in tokens))
