"""Matrix memory with exponential gates (mLSTM) over a fixed-size state.

With h the mixer's input, per head ``q = Wq h * dim^(-1/2)``, ``k = Wk h`` (``qk_dim`` numbers), ``v = Wv h``
(``v_dim``), and two log gates

    i = cap tanh((w_i . h + b_i) / cap)                       f = logsigmoid(cap tanh((w_f . h + b_f) / cap))

and from S = 0, n = 0, m = 0 (``cap``: ``gate_cap``)

    m_t = max(f + m_(t-1), i)
    S_t = exp(f + m_(t-1) - m_t) S_(t-1) + exp(i - m_t) k v^T           n_t the same with k alone
    o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6)
    result = Wo (o / rms(o) per head * norm * sigmoid(Wg h)) * out_scale

The state of a sequence is S [heads, qk_dim, v_dim], n [heads, qk_dim] and m [heads], fp32, zero when the slot is taken;
no position is cached.  The projection's result and everything up to the gated norm are fp32 in every precision, but that
a bfloat16 run's prompts take q, k and v as bfloat16 and run the recurrence's products on the tensor cores (once m is
known, the recurrence has a decay and a step per head and token like state-space mixing; n is the same on v = 1).
"""
from __future__ import annotations

from typing import Any, Callable, Dict, Mapping, Optional

import torch

from ..csrc import kernels as K
from .base import Mixer, ParamSpec, PositionEncoding, StateNeed
from .linear import ADD_F32, STORE, STORE_F32, Linear, stack_rows
from .registry import MIXERS
from .state_space import SEGMENT, TC_MIN_TOKENS, tc_segment

_NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "gate": "g_proj.weight", "out": "o_proj.weight",
          "norm": "norm.weight", "input_gate": "i_gate.weight", "input_gate_bias": "i_gate.bias",
          "forget_gate": "f_gate.weight", "forget_gate_bias": "f_gate.bias"}
_WHOLE_SEQUENCE = 1 << 30


class MatrixMemory(Mixer):
    """``out_scale``: a constant factor on the result.  ``names``: tensor names below the part's prefix."""

    def __init__(self, hidden_size: int, num_heads: int, qk_dim: int, v_dim: int, gate_cap: float, eps: float,
                 out_scale: float = 1.0, names: Optional[Mapping[str, str]] = None):
        super().__init__(hidden_size=hidden_size, num_heads=num_heads, qk_dim=qk_dim, v_dim=v_dim, gate_cap=gate_cap,
                         eps=eps, out_scale=out_scale, names=names)
        if min(hidden_size, num_heads, qk_dim, v_dim) <= 0 or not gate_cap > 0:
            raise ValueError("sizes and gate_cap must be positive")
        if qk_dim > K.SSD_MAX_STATE:
            raise ValueError(f"qk_dim must be at most {K.SSD_MAX_STATE}, got {qk_dim}")
        self.hidden_size, self.n_heads = int(hidden_size), int(num_heads)
        self.qk_dim, self.v_dim = int(qk_dim), int(v_dim)
        self.gate_cap, self.eps, self.out_scale = float(gate_cap), float(eps), float(out_scale)
        self.names = dict(_NAMES)
        self.names.update(names or {})
        # the state-space kernels' view of the recurrence: x = v, B = k, C = q, a group per head, no convolution
        self.shape = K.SsdShape(self.n_heads, self.n_heads, self.qk_dim, self.v_dim, 1)
        self.w_in: Optional[Linear] = None        # rows v | k | q | gate | i | f
        self.wo: Optional[Linear] = None
        self.prompt_views: Optional[tuple] = None
        self.b_i = self.b_f = self.norm = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        n, d, H = self.names, self.hidden_size, self.n_heads
        return {
            n["q"]: ParamSpec((H * self.qk_dim, d)), n["k"]: ParamSpec((H * self.qk_dim, d)),
            n["v"]: ParamSpec((H * self.v_dim, d)), n["gate"]: ParamSpec((H * self.v_dim, d)),
            n["out"]: ParamSpec((d, H * self.v_dim)), n["norm"]: ParamSpec((H * self.v_dim,), "one_plus_normal"),
            n["input_gate"]: ParamSpec((H, d)), n["input_gate_bias"]: ParamSpec((H,)),
            n["forget_gate"]: ParamSpec((H, d)), n["forget_gate_bias"]: ParamSpec((H,), "one_plus_normal"),
        }

    def state_need(self) -> StateNeed:
        return StateNeed((K.mlstm_state_floats(self.n_heads, self.qk_dim, self.v_dim),), torch.float32)

    def load(self, get: Callable[[str], torch.Tensor], runtime: Any) -> None:
        n, H = self.names, self.n_heads
        self.w_in = Linear(stack_rows(runtime.compute_copy(get(n[k])) for k in
                                      ("v", "k", "q", "gate", "input_gate", "forget_gate")), runtime)
        self.wo = Linear(get(n["out"]), runtime)
        # what enters the recurrence is 32-bit in every precision
        self.b_i, self.b_f, self.norm = (get(n[k]).to(torch.float32).contiguous() for k in
                                         ("input_gate_bias", "forget_gate_bias", "norm"))
        # prompts on the tensor cores: v | k | q and what stays fp32 as contractions of their own over the same rows
        n_vkq = H * (2 * self.qk_dim + self.v_dim)
        self.prompt_views = None
        if n_vkq % 8 == 0 and K.ssd_chunks_takes(runtime.dtype, self.qk_dim, self.v_dim):
            self.prompt_views = (Linear(self.w_in.weight[:n_vkq], runtime), Linear(self.w_in.weight[n_vkq:], runtime))

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx: Any, cache: Any,
                state: Optional[torch.Tensor], positions: Mapping[str, PositionEncoding]) -> None:
        if state is None:
            raise RuntimeError("a matrix memory needs its state")
        H, dk, dv = self.n_heads, self.qk_dim, self.v_dim
        st = state if state.dim() == 2 else state.view(state.shape[0], -1)
        on_tc = self.prompt_views is not None and not ctx.decode and 0 < TC_MIN_TOKENS <= ctx.n_tokens
        if on_tc:
            vkq, rest = self.prompt_views[0](x, STORE), self.prompt_views[1](x, STORE_F32)
        else:
            vkq = self.w_in(x, STORE_F32)                   # [T, v | k | q | gate | i | f (+ padding)] fp32
            rest = vkq[:, H * (2 * dk + dv):]
        gate, zi, zf = rest[:, :H * dv], rest[:, H * dv:H * dv + H], rest[:, H * dv + H:H * dv + 2 * H]
        if ctx.decode:
            o, nq, m = K.mlstm_step(vkq, zi, zf, self.b_i, self.b_f, self.gate_cap, ctx.seq_slot, st, H, dk, dv)
        else:
            seqs, n_seqs, longest = ctx.tiles(_WHOLE_SEQUENCE)
            steps, m = K.mlstm_gates(zi, zf, self.b_i, self.b_f, self.gate_cap, seqs, n_seqs, longest, ctx.seq_slot, st,
                                     H, dk, dv, log_decay=on_tc)
            tiles, n_tiles, _ = ctx.tiles(tc_segment(ctx.n_tokens, H, dv) if on_tc else SEGMENT)
            direct = n_tiles == ctx.n_seqs
            scratch = None if direct else ctx.scratch("mlstm_segments", n_tiles * H * (dk * dv + 1 + dk))
            k0, q0 = H * dv, H * (dv + dk)
            if on_tc:
                o, nq = K.ssd_chunks(vkq, 0, k0, q0, steps, None, None, tiles, n_tiles, direct, ctx.seq_slot, st, scratch,
                                     H, H, dk, dv, norm_off=H * dk * dv)
            else:
                o = K.ssd_segments(vkq, steps, None, tiles, n_tiles, direct, ctx.seq_slot, st, scratch, self.shape)
                nq = K.mlstm_norm_scan(vkq[:, k0:q0], vkq[:, q0:q0 + H * dk], steps, seqs, n_seqs, ctx.seq_slot, st,
                                       H, dk, dv)
        a = K.mlstm_gate_norm(o, nq, m, dk ** -0.5, gate, self.norm, self.eps, self.out_scale, self.wo.weight.dtype,
                              ctx.seq_slot, st, ctx.decode, H, dk, dv)
        self.wo(a, ADD_F32, residual)


MIXERS.register("matrix_memory", MatrixMemory)
