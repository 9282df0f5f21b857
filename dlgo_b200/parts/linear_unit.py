"""A recurrent block around a real-gated linear recurrent unit (Griffin) over a fixed-size state.

With h the mixer's input, two branches of ``width`` channels:

    y = gelu(Wy h + by)                                          (tanh form)
    u = bc + causal convolution over time of (Wx h + bx)         per channel, ``conv_taps`` taps, no activation
    r = sigmoid(Ra[p] u_p + br),  i = sigmoid(Ri[p] u_p + bi)    for each of ``parts`` equal parts u_p of u
    log a = -rate * r * softplus(lam)
    S_t = a S_(t-1) + sqrt(1 - a^2) * i * u                      per channel, S = 0 before the first token
    result = Wo (S * y) * out_scale

The state of a sequence is S followed by the convolution's last inputs (an entry per tap, the input of position p in
entry p mod taps), fp32, zero when the slot is taken; no position is cached.  The projections' results, the convolution,
the gates' sums, the decay and the recurrence are fp32 in every precision; in bfloat16 prompts u enters the gates'
contraction rounded (and y leaves its contraction finished, in bfloat16).
"""
from __future__ import annotations

import os
from typing import Any, Callable, Dict, Mapping, Optional

import torch

from ..csrc import kernels as K
from .base import Mixer, ParamSpec, PositionEncoding, StateNeed
from .linear import ADD_F32, STORE_F32, Linear
from .registry import MIXERS

_NAMES = {"y": "y_proj.weight", "y_bias": "y_proj.bias", "x": "x_proj.weight", "x_bias": "x_proj.bias", "conv": "conv.weight",
          "conv_bias": "conv.bias", "r": "r_gate.weight", "r_bias": "r_gate.bias", "i": "i_gate.weight",
          "i_bias": "i_gate.bias", "decay": "decay", "out": "o_proj.weight"}
CONV_TILE = 16                                                       # tokens of a block of the convolution
SEGMENT = int(os.environ.get("DLGO_RGLRU_SEGMENT", 0))               # tokens of a segment of the recurrence (0: see segment)
SCAN_BLOCKS = int(os.environ.get("DLGO_RGLRU_BLOCKS", 1184))         # blocks of the recurrence on the GPU at once: eight per SM
TC_MIN_TOKENS = 64                                                   # prompt steps whose gates run on the tensor cores


def segment(tokens: int, width: int) -> int:
    """Tokens of a segment: as many segments as run at the same time, of at least 16 tokens."""
    if SEGMENT > 0:
        return SEGMENT
    segments = max(1, SCAN_BLOCKS // -(-width // 128))
    return max(16, -(-tokens // (8 * segments)) * 8)


class RealGatedLinearUnit(Mixer):
    """``rate``: the constant factor of the decay's logarithm.  ``names``: tensor names below the part's prefix."""

    def __init__(self, hidden_size: int, width: int, parts: int, conv_taps: int, rate: float = 8.0, out_scale: float = 1.0,
                 names: Optional[Mapping[str, str]] = None):
        super().__init__(hidden_size=hidden_size, width=width, parts=parts, conv_taps=conv_taps, rate=rate,
                         out_scale=out_scale, names=names)
        if min(hidden_size, width, parts, conv_taps) <= 0 or not rate > 0:
            raise ValueError("sizes and rate must be positive")
        if width % parts:
            raise ValueError(f"parts ({parts}) must divide width ({width})")
        if out_scale != 1.0:
            raise ValueError("this mixer carries no factor on its result")
        self.hidden_size, self.width, self.parts = int(hidden_size), int(width), int(parts)
        self.shape = K.RglruShape(self.width, self.parts, int(conv_taps), float(rate))
        self.names = dict(_NAMES)
        self.names.update(names or {})
        self.w_in: Optional[Linear] = None        # rows y | x
        self.w_y: Optional[Linear] = None         # the same rows as contractions of their own (prompts)
        self.w_x: Optional[Linear] = None
        self.wo: Optional[Linear] = None
        self.w_gates: Optional[torch.Tensor] = None      # [parts, 2 B, B]
        self.b_y = self.b_x = self.taps = self.b_conv = self.b_r = self.b_i = self.lam = None
        self.x_col = 0

    def param_specs(self) -> Dict[str, ParamSpec]:
        n, d, w, p = self.names, self.hidden_size, self.width, self.parts
        b = w // p
        return {
            n["y"]: ParamSpec((w, d)), n["y_bias"]: ParamSpec((w,)), n["x"]: ParamSpec((w, d)), n["x_bias"]: ParamSpec((w,)),
            n["conv"]: ParamSpec((w, self.shape.taps), "last_one_plus_normal"), n["conv_bias"]: ParamSpec((w,)),
            n["r"]: ParamSpec((p, b, b)), n["r_bias"]: ParamSpec((p, b)), n["i"]: ParamSpec((p, b, b)),
            n["i_bias"]: ParamSpec((p, b)), n["decay"]: ParamSpec((w,)), n["out"]: ParamSpec((d, w)),
        }

    def state_need(self) -> StateNeed:
        return StateNeed((self.shape.state_floats(),), torch.float32)

    def load(self, get: Callable[[str], torch.Tensor], runtime: Any) -> None:
        n, w = self.names, self.width
        rows = [runtime.compute_copy(get(n[k])) for k in ("y", "x")]
        if w % 8:                                 # (x starts on a whole 16 bytes of a result's row)
            rows.insert(1, torch.zeros((-w % 8, self.hidden_size), dtype=rows[0].dtype, device=rows[0].device))
        self.x_col = w + -w % 8
        self.w_in = Linear(torch.cat(rows, dim=0).contiguous(), runtime)
        self.w_y, self.w_x = Linear(self.w_in.weight[:w], runtime), Linear(self.w_in.weight[self.x_col:], runtime)
        self.wo = Linear(get(n["out"]), runtime)
        self.w_gates = torch.cat([runtime.compute_copy(get(n["r"])), runtime.compute_copy(get(n["i"]))], dim=1).contiguous()
        self.b_y, self.b_x, self.taps, self.b_conv, self.b_r, self.b_i, self.lam = (
            get(n[k]).to(torch.float32).reshape(-1).contiguous() for k in
            ("y_bias", "x_bias", "conv", "conv_bias", "r_bias", "i_bias", "decay"))

    def _gate_logits(self, u: torch.Tensor, rows: Optional[torch.Tensor]) -> torch.Tensor:
        """[T * parts, 2 B] fp32: a part's rows of both matrices times its part of u (a grouped contraction whose groups
        are the parts, every one with all tokens)."""
        T, B = u.shape[0], self.width // self.parts
        z = torch.empty((T * self.parts, 2 * B), dtype=torch.float32, device=u.device)
        a = rows if rows is not None else u.view(T * self.parts, B)
        K.moe_gemm(K.part_plan(self.parts, T, K.MOE_FEW_ROWS if T <= 64 else K.MOE_TILE_ROWS, u.device), a, self.w_gates, z,
                   1, True, K.ACT_NONE)
        return z

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx: Any, cache: Any,
                state: Optional[torch.Tensor], positions: Mapping[str, PositionEncoding]) -> None:
        if state is None:
            raise RuntimeError("a recurrent unit needs its state")
        T, w, s = ctx.n_tokens, self.width, self.shape
        act = self.wo.weight.dtype
        st = state if state.dim() == 2 else state.view(state.shape[0], -1)
        if ctx.decode:
            a = K.rglru_step(self.w_in(x, STORE_F32), self.x_col, self.b_y, self.b_x, self.taps, self.b_conv, self.w_gates,
                             self.b_r, self.b_i, self.lam, ctx.token_pos, ctx.seq_slot, st, s)
            self.wo(a, ADD_F32, residual)
            return
        # bfloat16 prompts: the gates, and a segment's walk from zero behind them, in one launch on the tensor cores
        on_tc = T >= TC_MIN_TOKENS and K.rglru_gates_tc_takes(act, w // self.parts)
        if act == torch.bfloat16 and T >= TC_MIN_TOKENS:
            y, by = self.w_y.bias_act(x, self.b_y, K.ACT_GELU_TANH), None
            xs = self.w_x(x, STORE_F32)
        else:
            proj = self.w_in(x, STORE_F32)
            y, by, xs = proj[:, :w], self.b_y, proj[:, self.x_col:self.x_col + w]
        tiles, n_tiles, _ = ctx.tiles(CONV_TILE)
        u, rows = K.rglru_conv(xs, self.b_x, self.taps, self.b_conv, tiles, n_tiles, ctx.token_seq, ctx.token_pos,
                               ctx.seq_slot, st, s, None if act == torch.float32 else act, on_tc, f32=not on_tc)
        tiles, n_tiles, _ = ctx.tiles(K.RGLRU_TC_SEGMENT if on_tc else segment(T, w))
        direct = not on_tc and n_tiles == ctx.n_seqs
        scratch = None if direct else ctx.scratch("rglru_segments", n_tiles * 3 * w)
        if on_tc:
            z = K.rglru_gates_tc(rows, self.w_gates, self.b_r, self.b_i, self.lam, tiles, n_tiles, T, scratch, s)
        else:
            z = self._gate_logits(u, rows)
        a = K.rglru_scan(z, u, self.b_r, self.b_i, self.lam, y, by, xs, self.b_x, tiles, n_tiles, direct, ctx.token_seq,
                         ctx.token_pos, ctx.seq_slot, st, scratch, s, act, prepared=on_tc)
        self.wo(a, ADD_F32, residual)


MIXERS.register("rglru", RealGatedLinearUnit)
