"""A plain, slow implementation of the Bonusun design, one function per mechanism, written from its equations only.
It shares no code with the package: it reads config.json and the safetensors file itself and computes whole sequences
on the CPU with torch in float32 or float64.

Notation: h is a sublayer's input [T, width]; X are the residual streams [s, T, width]; w the tensors by name.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional, Tuple

import torch

_DT = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "F64": torch.float64}


def read_model(model_dir: str, dtype: torch.dtype = torch.float64) -> Tuple[dict, Dict[str, torch.Tensor]]:
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(model_dir, "model.safetensors"), "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        head = json.loads(f.read(n))
        blob = f.read()
    w = {}
    for name, info in head.items():
        if name == "__metadata__":
            continue
        a, b = info["data_offsets"]
        t = torch.frombuffer(bytearray(blob[a:b]), dtype=_DT[info["dtype"]]).reshape(info["shape"])
        w[name] = t.to(dtype) if t.is_floating_point() else t
    return cfg, w


def run_order(cfg: dict) -> List[int]:
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b, times = loop["start"], loop["stop"], loop["times"]
    return list(range(a)) + list(range(a, b)) * times + list(range(b, n))


# ------------------------------------------------------------------------------ norms and small functions
def layer_norm(x, weight, bias, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight + bias


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


# ------------------------------------------------------------------------------ attention
def rotate_halves(t: torch.Tensor, rot: dict, first: int = 0) -> torch.Tensor:
    """t [T, heads, dim], row p at position first + p: of the first rot.dims entries, i turns with i + dims/2."""
    T, r = t.shape[0], rot["dims"]
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    f = torch.tensor([rot["base"] ** (-2.0 * i / r) / factor for i in range(r // 2)], dtype=torch.float64)
    ang = torch.arange(first, first + T, dtype=torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(ang).to(t.dtype)[:, None, :], torch.sin(ang).to(t.dtype)[:, None, :]
    u, v = t[..., :r // 2], t[..., r // 2:r]
    return torch.cat([u * c - v * s, v * c + u * s, t[..., r:]], dim=-1)


def attend(q, k, v, scale, sink, window: Optional[int]):
    """q [T, H, d], k [T, G, d], v [T, G, dv], sink [H] -> [T, H, dv]; the softmax's denominator also holds exp(sink)."""
    T, H = q.shape[:2]
    n = H // k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(n, 1)) * scale
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) if window is None else (j <= i) & (i - j < window)
    s = s.masked_fill(~seen[None], float("-inf"))
    s = torch.cat([s, sink.to(s.dtype)[:, None, None].expand(H, T, 1)], dim=-1)
    p = torch.softmax(s, dim=-1)[..., :T]
    return torch.einsum("hij,jhd->ihd", p, v.repeat_interleave(n, 1))


def attention(h, w, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = over_rms((h @ w[p + "q"].T).view(T, H, d), eps) * w[p + "q.norm"]
    k = over_rms((h @ w[p + "k"].T).view(T, G, d), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).view(T, G, dv)
    if m.get("rot"):
        q, k = rotate_halves(q, m["rot"]), rotate_halves(k, m["rot"])
    window = m["mask"]["size"] if m.get("mask") else None
    return attend(q, k, v, m["scale"], w[p + "sink"], window).reshape(T, H * dv) @ w[p + "o"].T


# ------------------------------------------------------------------------------ matrix memory
def matrix_memory(q, k, v, i, f, state=None):
    """q, k [T, H, d], v [T, H, dv], log gates i, f [T, H]; token by token.  Returns (o [T, H, dv], (S, n, m))."""
    T, H, d = q.shape
    dv = v.shape[-1]
    if state is None:
        state = (q.new_zeros(H, d, dv), q.new_zeros(H, d), q.new_zeros(H))
    S, n, m = state
    out = []
    for t in range(T):
        top = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - top), torch.exp(i[t] - top)
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        m = top
        num = torch.einsum("hd,hde->he", q[t], S)
        den = torch.maximum((q[t] * n).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(num / den[:, None])
    return torch.stack(out), (S, n, m)


def mlstm(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, dv)
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = -softplus(-cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    o, _ = matrix_memory(q, k, v, i, f)
    o = over_rms(o, eps).reshape(T, H * dv) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def parallel(h, w, p, m, eps):
    return (m["left_scale"] * attention(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * mlstm(h, w, p + "right.", m["right"], eps))


# ------------------------------------------------------------------------------ gated linear recurrence
def causal_conv(x, taps, bias):
    """x [T, c], taps [c, n] (the last column is the current token's)."""
    n = taps.shape[1]
    padded = torch.cat([x.new_zeros(n - 1, x.shape[1]), x])
    return sum(padded[j:j + x.shape[0]] * taps[:, j] for j in range(n)) + bias


def block_linear(u, weight, bias):
    """u [T, b * n], weight [b, n, n] as [out, in] per part, bias [b, n]."""
    b, n, _ = weight.shape
    return (torch.einsum("tbi,boi->tbo", u.view(-1, b, n), weight) + bias).reshape(u.shape)


def gated_recurrence(u, r, i, lam, state=None):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with log a = -8 r softplus(lam); returns all S_t [T, c]."""
    S = u.new_zeros(u.shape[1]) if state is None else state
    log_a = -8 * r * softplus(lam)
    a, b = torch.exp(log_a), torch.sqrt(-torch.expm1(2 * log_a))
    out = []
    for t in range(u.shape[0]):
        S = a[t] * S + b[t] * i[t] * u[t]
        out.append(S)
    return torch.stack(out)


def rglru(h, w, p, m, eps):
    y = gelu_tanh(h @ w[p + "y"].T + w[p + "y.b"])
    u = causal_conv(h @ w[p + "x"].T + w[p + "x.b"], w[p + "conv"], w[p + "conv.b"])
    r = torch.sigmoid(block_linear(u, w[p + "ra"], w[p + "ra.b"]))
    i = torch.sigmoid(block_linear(u, w[p + "ri"], w[p + "ri.b"]))
    return (gated_recurrence(u, r, i, w[p + "lam"]) * y) @ w[p + "o"].T


# ------------------------------------------------------------------------------ feed-forwards
def clamped_expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ down.T


def route(h, router, correction, r):
    """Chosen experts [T, top] and their weights."""
    s = torch.sigmoid(h @ router.T)
    c = s + correction
    T, E = s.shape
    g = r.get("groups")
    if g:
        size = E // g["count"]
        best = torch.topk(c.view(T, g["count"], size), min(2, size), dim=-1).values.sum(-1)
        keep = torch.topk(best, g["keep"], dim=-1).indices
        ok = torch.zeros(T, g["count"], dtype=torch.bool).scatter(1, keep, True)
        c = c.masked_fill(~ok.repeat_interleave(size, dim=1), float("-inf"))
    idx = torch.topk(c, r["top"], dim=-1).indices
    wt = s.gather(1, idx)
    return idx, wt / (wt.sum(-1, keepdim=True) + 1e-20) * r["scale"]


def experts(h, w, p, mlp):
    idx, wt = route(h, w[p + "router"], w[p + "correction"], mlp["router"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, k = (idx == e).nonzero(as_tuple=True)
        if len(t):
            q = f"{p}e{e}."
            out[t] += wt[t, k][:, None] * clamped_expert(h[t], w[q + "gate"], w[q + "up"], w[q + "down"],
                                                         mlp["expert"]["limit"])
    if mlp.get("shared"):
        q = p + "shared."
        out = out + torch.sigmoid(h @ w[q + "sg"].T) * clamped_expert(h, w[q + "gate"], w[q + "up"], w[q + "down"],
                                                                      mlp["shared"]["limit"])
    return out


def feed_forward(h, w, p, mlp):
    if mlp["kind"] == "dense":
        return gelu_tanh(h @ w[p + "up"].T) @ w[p + "down"].T
    return experts(h, w, p, mlp)


# ------------------------------------------------------------------------------ the whole model
def through_streams(X, w, p, mult, sublayer):
    """One sublayer on the streams X [s, T, d]: reads sum_s in[s] X_s, returns the streams it leaves."""
    y = sublayer(torch.einsum("s,std->td", w[p + "in"], X))
    return torch.einsum("st,sxd->txd", w[p + "mix"], X) + mult * w[p + "out"][:, None, None] * y


MIXERS = {"attention": attention, "parallel": parallel, "rglru": rglru}


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the streams' sum after every layer run."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    e = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    X = e[None].repeat(cfg["streams"], 1, 1)
    for i in run_order(cfg):
        L, p = cfg["layers"][i], f"l{i}."

        def mix(u):
            n = layer_norm(u, w[p + "norm1"], w[p + "norm1.b"], eps)
            return MIXERS[L["type"]](n, w, p + "mix.", L["mixer"], eps)

        def ff(u):
            return feed_forward(layer_norm(u, w[p + "norm2"], w[p + "norm2.b"], eps), w, p + "mlp.", L["mlp"])

        X = through_streams(X, w, p + "hc1.", mult, mix)
        if L.get("mlp") is not None:
            X = through_streams(X, w, p + "hc2.", mult, ff)
        if layers_out is not None:
            layers_out.append(X.sum(0))
    return layer_norm(X.sum(0), w["final.norm"], w["final.norm.b"], eps) @ w["head"].T


def greedy_generate(cfg: dict, w: Dict[str, torch.Tensor], prompt, n: int) -> List[int]:
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(forward(cfg, w, tokens)[-1].argmax()))
    return tokens[len(prompt):]
