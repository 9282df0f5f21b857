"""Small Bonusun configurations with weights of a useful size, and helpers that run the engine and the plain
implementation on them.  The configurations differ from one another in every size and in the order of their layers, and
include values that are 1 (one stream, one head, one kv head, one tap, one part, one expert, one chosen, a window of one)
or absent (no rotation, no scaling, no mask, no groups of experts, no shared expert, no loop, a layer without feed-forward)
and values that models often make equal but that need not be (key and value sizes, heads and kv heads, rotated and whole
heads, the limits of the experts and of the shared one, the recurrence's width and the model's)."""
from __future__ import annotations

import functools
import json
import os
from typing import Dict, Sequence, Tuple

import torch

from bazurax_configs import RowCheck, assert_rows, random_tokens, row_error      # noqa: F401  (shared test helpers)


def att(heads, kv, dim, vdim, scale, rot=0, base=10000.0, factor=None, window=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if factor:
            m["rot"]["scaling"] = {"factor": factor}
    if window:
        m["mask"] = {"size": window}
    return m


def mem(heads, dim, vdim, cap=15.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def par(left, right, left_scale=1.0, right_scale=1.0):
    return {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def rec(width, blocks, conv):
    return {"width": width, "blocks": blocks, "conv": conv}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, limit=2.0, scale=1.0, groups=None, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "scale": scale}}
    if groups:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def layer(mixer, mlp=None):
    kind = "parallel" if "left" in mixer else ("rglru" if "blocks" in mixer else "attention")
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def model(vocab, width, layers, streams=2, mult=0.8, loop=None, eps=1e-5):
    cfg = {"architecture": "Bonusun", "vocab": vocab, "width": width, "streams": streams, "residual_mult": mult,
           "norm": {"eps": eps}, "layers": layers}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


CONFIGS: Dict[str, dict] = {
    # the recurrent unit first; a loop over the middle; values wider and narrower than keys; three query heads per kv head;
    # half of a head turns; a layer without feed-forward, one without rotation
    "P": model(150, 72, [
        layer(rec(60, 3, 4), moe(40, 6, 3, 1.5, 1.7, (3, 2), (24, 0.8))),
        layer(par(att(6, 2, 24, 40, 0.3, 12, 5000.0, 4.0), mem(3, 16, 20, 6.0), 0.7, 1.3), dense(88)),
        layer(att(4, 2, 24, 16, 0.25, 24, 300.0, window=37)),
        layer(att(2, 1, 20, 28, 0.3), moe(16, 4, 1, 1.0, 0.6, (2, 1)))], streams=2, mult=0.6, loop=(1, 3, 2)),
    # one of everything: streams, heads, parts, taps, experts; a window of one and one longer than a page; sizes that are
    # multiples of nothing; no loop
    "Q": model(97, 46, [
        layer(par(att(1, 1, 10, 7, 0.4, 10, 100.0), mem(1, 7, 5, 2.0), 1.0, 1.0), moe(24, 1, 1, 0.9, 2.0, None, (10, 3.0))),
        layer(rec(33, 1, 1)),
        layer(att(3, 3, 12, 20, 0.35, 4, 1e6, 2.0, window=1), dense(30)),
        layer(rec(50, 5, 6), moe(18, 6, 4, 5.0, 1.0, (3, 2))),
        layer(par(att(5, 1, 8, 8, 0.5, window=70), mem(2, 33, 12, 30.0), 0.4, 1.6), dense(51))], streams=1, mult=1.0, eps=1e-6),
    # sizes that the tensor-core kernels take in bfloat16: heads of 64 and 128 (also stretched to them), memories of 32, 64
    # and 128, parts of 64 and 32 channels, experts of 64 and 96
    "R": model(260, 128, [
        layer(att(4, 2, 64, 48, 0.125, 64, 250000.0, window=64), moe(64, 8, 2, 2.0, 2.5, (4, 3), (96, 1.0))),
        layer(par(att(3, 1, 48, 64, 0.15, 32, 1e5, 8.0), mem(2, 64, 64, 15.0), 1.2, 0.9), dense(192)),
        layer(rec(256, 4, 3), dense(96)),
        layer(par(att(2, 2, 96, 128, 0.1, 96, 1e4, window=129), mem(3, 32, 72, 4.0), 0.8, 0.5), moe(96, 12, 4, 1.0, 1.0, (3, 2))),
        layer(rec(96, 3, 2))], streams=4, mult=0.5, loop=(2, 4, 2), eps=1e-6),
}
SEEDS = {"P": 61, "Q": 62, "R": 63}


def tensor_shapes(cfg: dict) -> Dict[str, Tuple[int, ...]]:
    """Names and shapes of a configuration's tensors, from the design's description (not from the package)."""
    d, V, n_s = cfg["width"], cfg["vocab"], cfg["streams"]
    s: Dict[str, Tuple[int, ...]] = {"embed": (V, d), "head": (V, d), "final.norm": (d,), "final.norm.b": (d,)}

    def attention(p, m):
        H, G, n, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        s.update({p + "q": (H * n, d), p + "k": (G * n, d), p + "v": (G * v, d), p + "q.norm": (n,), p + "k.norm": (n,),
                  p + "sink": (H,), p + "o": (d, H * v)})

    for i, L in enumerate(cfg["layers"]):
        p, m, x = f"l{i}.", L["mixer"], f"l{i}.mix."
        for q in (1, 2) if L["mlp"] is not None else (1,):
            s.update({p + f"norm{q}": (d,), p + f"norm{q}.b": (d,), p + f"hc{q}.in": (n_s,), p + f"hc{q}.out": (n_s,),
                      p + f"hc{q}.mix": (n_s, n_s)})
        if L["type"] == "attention":
            attention(x, m)
        elif L["type"] == "rglru":
            w, b = m["width"], m["blocks"]
            s.update({x + "y": (w, d), x + "y.b": (w,), x + "x": (w, d), x + "x.b": (w,), x + "conv": (w, m["conv"]),
                      x + "conv.b": (w,), x + "ra": (b, w // b, w // b), x + "ra.b": (b, w // b),
                      x + "ri": (b, w // b, w // b), x + "ri.b": (b, w // b), x + "lam": (w,), x + "o": (d, w)})
        else:
            attention(x + "left.", m["left"])
            r, x = m["right"], x + "right."
            H, n, v = r["heads"], r["dim"], r["vdim"]
            s.update({x + "q": (H * n, d), x + "k": (H * n, d), x + "v": (H * v, d), x + "g": (H * v, d), x + "o": (d, H * v),
                      x + "norm": (H * v,), x + "i": (H, d), x + "i.b": (H,), x + "f": (H, d), x + "f.b": (H,)})
        mlp, y = L["mlp"], p + "mlp."
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            s.update({y + "up": (mlp["ff"], d), y + "down": (d, mlp["ff"])})
            continue
        E = mlp["router"]["experts"]
        forms = [(f"e{e}.", mlp["expert"]["ff"]) for e in range(E)]
        s.update({y + "router": (E, d), y + "correction": (E,)})
        if "shared" in mlp:
            forms.append(("shared.", mlp["shared"]["ff"]))
            s[y + "shared.sg"] = (1, d)
        for q, f in forms:
            s.update({y + q + "gate": (f, d), y + q + "up": (f, d), y + q + "down": (d, f)})
    return s


def make_weights(cfg: dict, seed: int, sharpen: float = 2.5, mild: bool = False) -> Dict[str, torch.Tensor]:
    """Weights (bfloat16): matrices ~ N(0, 1/in), the embedding N(0, 1), norm weights around 1 and biases of visible size,
    connections that mix the streams, sinks around the scores, corrections that make choice scores negative, forget gates
    from a few tokens to hundreds.  The queries' norm weight is multiplied by ``sharpen`` so that the softmax is far from
    uniform and a wrong, missing or extra key moves the logits; gates of experts are large enough to meet their limits.
    ``mild`` (whole models in bfloat16): flatter softmaxes and routers and smaller experts' results, so that a router's
    near tie that rounding tips the other way stays one row's affair."""
    if mild:
        sharpen = 1.3
    g = torch.Generator().manual_seed(seed)
    w = {}
    shapes = tensor_shapes(cfg)
    n_s = cfg["streams"]
    for name in sorted(shapes):
        shape = shapes[name]
        r = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = r
        elif last == "in":
            t = 1.0 / n_s + 0.3 * r
        elif last == "out":
            t = 1.0 + 0.3 * r
        elif name.endswith(".mix"):
            t = torch.eye(n_s) * 0.8 + 0.3 * r / n_s
        elif name.endswith(".q.norm"):
            t = sharpen * (1.0 + 0.2 * r)
        elif "norm" in name:
            t = 0.2 * r if last == "b" else 1.0 + 0.2 * r
        elif last == "sink":
            t = 1.0 + r
        elif last == "correction":
            t = -0.6 + 0.15 * r
        elif name.endswith(".f.b"):
            t = 3.0 + 2.0 * r
        elif name.endswith(".conv"):
            t = 0.4 * r
            t[:, -1] += 1.0
        elif last == "lam":
            t = -4.0 + 2.0 * r
        elif last == "b":
            t = 0.4 * r
        elif last == "router":
            t = (1.0 if mild else 3.0) * r / shape[1] ** 0.5
        elif mild and ".mlp.e" in name and last == "down":
            t = 0.25 * r / shape[1] ** 0.5
        elif last in ("ra", "ri", "gate"):
            t = 1.5 * r / shape[-1] ** 0.5
        else:
            t = r / shape[-1] ** 0.5
        w[name] = t.to(torch.bfloat16)
    return w


def config_of(cfg: dict):
    from dlgo_b200.config.bonusun import BonusunConfig
    return BonusunConfig.from_dict(cfg)


def write_model(name: str, out_dir: str, sharpen: float = 2.5, mild: bool = False) -> str:
    from dlgo_b200.weights import save_tensors
    os.makedirs(out_dir, exist_ok=True)
    with open(os.path.join(out_dir, "config.json"), "w") as f:
        json.dump(CONFIGS[name], f)
    save_tensors(os.path.join(out_dir, "model.safetensors"), make_weights(CONFIGS[name], SEEDS[name], sharpen, mild=mild))
    return out_dir


@functools.lru_cache(maxsize=64)
def _plain_cached(model_dir: str, tokens: tuple) -> torch.Tensor:
    import plain_bonusun as P
    cfg, w = P.read_model(model_dir, torch.float64)
    return P.forward(cfg, w, list(tokens)).to(torch.float32)


def plain_logits(model_dir: str, tokens: Sequence[int]) -> torch.Tensor:
    """Logits [T, vocab] of the plain implementation (float64 arithmetic) for one whole sequence."""
    return _plain_cached(model_dir, tuple(int(t) for t in tokens))
