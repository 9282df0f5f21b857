"""State-space mixing with a scalar decay per head and token (Mamba-2's recurrence) over a fixed-size state.

With h the mixer's input, one projection gives [z | x | B | C | dt] (``heads * v_dim`` numbers for z and x,
``groups * state`` for B and C, one per head for dt):

    x, B, C <- silu(causal convolution over time, per channel, with a bias)
    d = softplus(dt + dt_bias)                                  per head
    S_t = exp(-exp(A_log) d) S_(t-1) + d B_t x_t^T              S [state, v_dim] per head
    y_t = S_t^T C_t + D x_t                                     head h reads B and C of group h // (heads / groups)
    result = Wo (rms over each of ``norm_groups`` parts of (y * silu(z)), times ``norm``)

The state of a sequence is S for every head followed by the last ``conv_taps - 1`` inputs of the convolution, fp32, zero
when the slot is taken; no position is cached.  The projection's result and everything up to the norm are fp32 in every
precision, but that a bfloat16 run's prompts take x, B and C as bfloat16 behind their silu and run the recurrence's
products on the tensor cores.
"""
from __future__ import annotations

import os
from typing import Any, Callable, Dict, Mapping, Optional

import torch

from ..csrc import kernels as K
from .base import Mixer, ParamSpec, PositionEncoding, StateNeed
from .linear import ADD_F32, STORE_F32, Linear, stack_rows
from .registry import MIXERS

_NAMES = {"in": "in_proj.weight", "conv": "conv.weight", "conv_bias": "conv.bias", "dt_bias": "dt_bias", "decay": "A_log",
          "skip": "D", "norm": "norm.weight", "out": "out_proj.weight"}
SEGMENT = int(os.environ.get("DLGO_SSD_SEGMENT", 128))   # tokens of a segment where a prompt's segments run side by side
TC_SEGMENT = int(os.environ.get("DLGO_SSD_TC_SEGMENT", 0))   # ... on the tensor cores (0: see tc_segment)
TC_BLOCKS = 444                                          # blocks of the tensor-core recurrence on the GPU at once: three per SM
TC_MIN_TOKENS = int(os.environ.get("DLGO_SSD_TC_MIN_TOKENS", 64))   # prompt steps that run there (0: never)
CONV_TILE = 16                                           # tokens of a block of the convolution
_WHOLE_SEQUENCE = 1 << 30


def tc_segment(tokens: int, heads: int, v_dim: int) -> int:
    """Tokens of a segment on the tensor cores: whole chunks of 64, as many segments as run at the same time (one more
    would be a second wave of blocks)."""
    if TC_SEGMENT > 0:
        return TC_SEGMENT
    segments = max(1, TC_BLOCKS // (heads * -(-v_dim // 64)))
    return -(-tokens // (64 * segments)) * 64


class StateSpaceMixer(Mixer):
    """``names``: tensor names below the part's prefix."""

    def __init__(self, hidden_size: int, num_heads: int, v_dim: int, state_size: int, num_groups: int, conv_taps: int,
                 norm_groups: int, eps: float, names: Optional[Mapping[str, str]] = None):
        super().__init__(hidden_size=hidden_size, num_heads=num_heads, v_dim=v_dim, state_size=state_size,
                         num_groups=num_groups, conv_taps=conv_taps, norm_groups=norm_groups, eps=eps, names=names)
        if min(hidden_size, num_heads, v_dim, state_size, num_groups, conv_taps, norm_groups) <= 0:
            raise ValueError("sizes must be positive")
        if num_heads % num_groups:
            raise ValueError(f"num_groups ({num_groups}) must divide num_heads ({num_heads})")
        if (num_heads * v_dim) % norm_groups:
            raise ValueError(f"norm_groups ({norm_groups}) must divide num_heads * v_dim ({num_heads * v_dim})")
        if state_size > K.SSD_MAX_STATE:
            raise ValueError(f"state_size must be at most {K.SSD_MAX_STATE}, got {state_size}")
        self.hidden_size = int(hidden_size)
        self.shape = K.SsdShape(int(num_heads), int(num_groups), int(state_size), int(v_dim), int(conv_taps))
        self.norm_groups, self.eps = int(norm_groups), float(eps)
        self.names = dict(_NAMES)
        self.names.update(names or {})
        self.w_in: Optional[Linear] = None        # rows z | x | B | C | dt
        self.wo: Optional[Linear] = None
        self.taps = self.conv_bias = self.dt_bias = self.a_log = self.skip = self.norm = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        n, d, s = self.names, self.hidden_size, self.shape
        return {
            n["in"]: ParamSpec((s.columns, d)), n["conv"]: ParamSpec((s.channels, s.taps), "last_one_plus_normal"),
            n["conv_bias"]: ParamSpec((s.channels,)), n["dt_bias"]: ParamSpec((s.heads,)), n["decay"]: ParamSpec((s.heads,)),
            n["skip"]: ParamSpec((s.heads,), "one_plus_normal"), n["norm"]: ParamSpec((s.inner,), "one_plus_normal"),
            n["out"]: ParamSpec((d, s.inner)),
        }

    def state_need(self) -> StateNeed:
        return StateNeed((self.shape.state_floats(),), torch.float32)

    def load(self, get: Callable[[str], torch.Tensor], runtime: Any) -> None:
        n = self.names
        self.w_in = Linear(stack_rows([runtime.compute_copy(get(n["in"]))]), runtime)
        self.wo = Linear(get(n["out"]), runtime)
        # what enters the recurrence is 32-bit in every precision
        self.taps, self.conv_bias, self.dt_bias, self.a_log, self.skip, self.norm = (
            get(n[k]).to(torch.float32).contiguous() for k in ("conv", "conv_bias", "dt_bias", "decay", "skip", "norm"))

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx: Any, cache: Any,
                state: Optional[torch.Tensor], positions: Mapping[str, PositionEncoding]) -> None:
        if state is None:
            raise RuntimeError("state-space mixing needs its state")
        s = self.shape
        proj = self.w_in(x, STORE_F32)                      # [T, columns (+ padding)] fp32
        if ctx.decode:
            y = K.ssd_step(proj, self.taps, self.conv_bias, self.dt_bias, self.a_log, self.skip, ctx.seq_slot, state, s)
        else:
            on_tc = 0 < TC_MIN_TOKENS <= ctx.n_tokens and K.ssd_chunks_takes(self.wo.weight.dtype, s.state, s.v_dim)
            tiles, n_tiles, _ = ctx.tiles(CONV_TILE)
            xbc, steps = K.ssd_conv(proj, self.taps, self.conv_bias, self.dt_bias, self.a_log, tiles, n_tiles,
                                    ctx.token_seq, ctx.seq_slot, state, s,
                                    out_dtype=torch.bfloat16 if on_tc else torch.float32, log_decay=on_tc)
            tiles, n_tiles, _ = ctx.tiles(tc_segment(ctx.n_tokens, s.heads, s.v_dim) if on_tc else SEGMENT)
            direct = n_tiles == ctx.n_seqs
            scratch = None if direct else ctx.scratch("ssd_segments", K.ssd_scratch_floats(n_tiles, s))
            if on_tc:
                bc = s.groups * s.state
                y = K.ssd_chunks(xbc, 0, s.inner, s.inner + bc, steps, None, self.skip, tiles, n_tiles, direct, ctx.seq_slot,
                                 state, scratch, s.heads, s.groups, s.state, s.v_dim)
            else:
                y = K.ssd_segments(xbc, steps, self.skip, tiles, n_tiles, direct, ctx.seq_slot, state, scratch, s)
        seqs, n_seqs, _ = ctx.tiles(1 if ctx.decode else _WHOLE_SEQUENCE)
        a = K.ssd_gate_norm(y, proj, self.norm, self.norm_groups, self.eps, self.wo.weight.dtype, seqs, n_seqs,
                            ctx.seq_slot, state, s)
        self.wo(a, ADD_F32, residual)


MIXERS.register("mamba2", StateSpaceMixer)
