"""A plain, slow implementation of the Zetavik design, one function per mechanism, written from its equations only.
It shares no code with the package: it reads config.json and the safetensors file itself and computes whole sequences
on the CPU with torch in float32 or float64.

Notation: x_0 = E[token]; a layer turns x into  x + (mixer(n) + ff(n))  with ONE  n = LN(x)  for both (a layer
without feed-forward: x + mixer(n)); logits = E LN_final(x).

    LN(u)  = (u - mean u) / sqrt(mean (u - mean u)^2 + e) * w
    RMS(u) = u / sqrt(mean u^2 + e)
"""
from __future__ import annotations

import json
import os
import struct
from typing import Dict, List, Optional, Tuple

import torch

_DT = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "F64": torch.float64}


def read_model(model_dir: str, dtype: torch.dtype = torch.float32) -> Tuple[dict, Dict[str, torch.Tensor]]:
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


def layer_norm(u: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    c = u - u.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * weight


def rms_norm(u: torch.Tensor, weight: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    r = u / torch.sqrt((u * u).mean(-1, keepdim=True) + eps)
    return r if weight is None else r * weight


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------ state-space mixer
def short_conv(u: torch.Tensor, taps: torch.Tensor, bias: torch.Tensor) -> torch.Tensor:
    """u [T, C] over time, taps [C, n]: y_t = bias + sum_j taps[:, j] * u_(t - n + 1 + j), zeros before the start."""
    T, C = u.shape
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, C, dtype=u.dtype), u], dim=0)
    y = bias.expand(T, C).clone()
    for j in range(n):
        y = y + taps[:, j] * padded[j:j + T]
    return y


def state_space_recurrence(x, B, C, dt, A, D, S0=None):
    """x [T, H, P], B, C [T, G, N], dt [T, H], A [H] (positive), D [H]:
    S_t = exp(-A dt_t) S_(t-1) + dt_t B_t x_t^T,  y_t = S_t^T C_t + D x_t;  head h reads group h // (H / G).
    Returns (y [T, H, P], the last S [H, N, P])."""
    T, H, P = x.shape
    G, N = B.shape[1], B.shape[2]
    per = H // G
    S = torch.zeros(H, N, P, dtype=x.dtype) if S0 is None else S0.clone()
    y = torch.zeros_like(x)
    for t in range(T):
        Bt, Ct = B[t].repeat_interleave(per, dim=0), C[t].repeat_interleave(per, dim=0)
        S = torch.exp(-A * dt[t])[:, None, None] * S + (dt[t][:, None] * Bt)[:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnp,hn->hp", S, Ct) + D[:, None] * x[t]
    return y, S


def gate_then_group_norm(y, z, weight, groups, eps):
    """RMS norm of y * silu(z) in ``groups`` equal parts of a row, then the weight."""
    u = y * silu(z)
    T, n = u.shape
    return rms_norm(u.view(T, groups, n // groups), None, eps).reshape(T, n) * weight


def mamba2(h, w, p, m, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ w[p + "in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    xbc = silu(short_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=-1)
    dt = torch.nn.functional.softplus(dt + w[p + "dt_bias"], threshold=1e9)
    y, _ = state_space_recurrence(x.view(T, H, P), B.view(T, G, N), C.view(T, G, N), dt, torch.exp(w[p + "A_log"]),
                                  w[p + "D"])
    return gate_then_group_norm(y.reshape(T, inner), z, w[p + "norm"], m["norm_groups"], eps) @ w[p + "o"].T


# ------------------------------------------------------------------------------ linear attention
def decayed_linear_attention(q, k, v, decay):
    """S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t;  q, k [T, H, d], v [T, H, dv], decay [H]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o


def lightning(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, k, v = silu(h @ w[p + "q"].T), silu(h @ w[p + "k"].T), silu(h @ w[p + "v"].T)
    o = decayed_linear_attention(q.view(T, H, d), k.view(T, H, d), v.view(T, H, dv),
                                 torch.tensor(m["decay"], dtype=h.dtype)).reshape(T, H * dv)
    return (rms_norm(o, w[p + "norm"], eps) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------------------ latent attention
def rotate_halves(t: torch.Tensor, base: float, first: int = 0) -> torch.Tensor:
    """t [T, heads, r], row p at position first + p: entry i turns with entry i + r/2 by (first + p) * base^(-2i/r)."""
    T, r = t.shape[0], t.shape[-1]
    f = torch.tensor([base ** (-2.0 * i / r) for i in range(r // 2)], dtype=torch.float64)
    ang = torch.arange(first, first + T, dtype=torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(ang).to(t.dtype)[:, None, :], torch.sin(ang).to(t.dtype)[:, None, :]
    u, v = t[..., :r // 2], t[..., r // 2:]
    return torch.cat([u * c - v * s, v * c + u * s], dim=-1)


def causal_attend(q, k, v, scale):
    """q, k [T, H, d], v [T, H, dv] -> [T, H, dv]."""
    T = q.shape[0]
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~torch.tril(torch.ones(T, T, dtype=torch.bool))[None], float("-inf"))
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, dim=-1), v)


def latent_attention(h, w, p, m, eps):
    T = h.shape[0]
    H, d, r, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).view(T, H, d + r)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :R], w[p + "dkv.norm"], eps)
    base = m["rot"]["base"]
    q = torch.cat([q[..., :d], rotate_halves(q[..., d:], base)], -1)
    kr = rotate_halves(down[:, None, R:], base).expand(T, H, r)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, d), kr], -1)
    o = causal_attend(q, k, (c @ w[p + "uv"].T).view(T, H, dv), m["scale"])
    o = o * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[p + "o"].T


# ------------------------------------------------------------------------------ feed-forwards
def gated_ff(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(h, router, r):
    """Chosen experts [T, top] and their weights: softmax over all, the best groups by their largest score, the
    largest scores within them, as they are, times the router's scale."""
    s = torch.softmax(h.to(torch.float32 if h.dtype != torch.float64 else torch.float64) @ router.T, dim=-1)
    T, E = s.shape
    c = s.clone()
    g = r.get("groups")
    if g:
        best = s.view(T, g["count"], E // g["count"]).max(-1).values
        keep = torch.topk(best, g["keep"], dim=-1).indices
        ok = torch.zeros(T, g["count"], dtype=torch.bool).scatter(1, keep, True)
        c = c.masked_fill(~ok.repeat_interleave(E // g["count"], dim=1), -1.0)
    idx = torch.topk(c, r["top"], dim=-1).indices
    return idx, s.gather(1, idx) * r.get("scale", 1.0)


def experts(h, w, p, mlp):
    idx, wt = route(h, w[p + "router"], mlp["router"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, k = (idx == e).nonzero(as_tuple=True)
        if len(t):
            q = f"{p}e{e}."
            out[t] += wt[t, k][:, None] * gated_ff(h[t], w[q + "gate"], w[q + "up"], w[q + "down"])
    if mlp.get("shared"):
        q = p + "shared."
        out = out + gated_ff(h, w[q + "gate"], w[q + "up"], w[q + "down"])
    return out


def feed_forward(h, w, p, mlp):
    if mlp["kind"] == "dense":
        return torch.relu(h @ w[p + "up"].T).square() @ w[p + "down"].T
    return experts(h, w, p, mlp)


# ------------------------------------------------------------------------------ the whole model
MIXERS = {"mamba2": mamba2, "latent_attention": latent_attention, "lightning": lightning}


def forward(cfg: dict, w: Dict[str, torch.Tensor], tokens, layers_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layers_out`` collects the residual stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        n = layer_norm(x, w[p + "norm1"], eps)
        y = MIXERS[L["type"]](n, w, p + "mix.", L["mixer"], eps)
        if L.get("mlp") is not None:
            y = y + feed_forward(n, w, p + "mlp.", L["mlp"])
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, w["final.norm"], eps) @ w["embed"].T


def greedy_generate(cfg: dict, w: Dict[str, torch.Tensor], prompt, n: int) -> List[int]:
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(forward(cfg, w, tokens)[-1].argmax()))
    return tokens[len(prompt):]
