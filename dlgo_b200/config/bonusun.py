"""Typed configuration of the Bonusun design, read from its config.json keys.

A Bonusun model is a list of layers on several residual streams (hyper-connections) behind layer norms with weight and
bias, a span of which runs several times in a row.  A layer's mixer is grouped-query attention (head norms, rotation, an
optional sliding window, a sink per head), such an attention beside a matrix memory with exponential gates, or a recurrent
block around a real-gated linear recurrent unit.  The feed-forward is a dense one with gelu, a mixture of clamped gated
experts chosen within the best groups plus a gated shared expert, or absent:

    {"architecture": "Bonusun", "vocab": V, "width": d, "streams": s, "residual_mult": m, "norm": {"eps": e},
     "loop": null | {"start": a, "stop": b, "times": n},
     "layers": [{"type": "attention",
                 "mixer": {"heads": H, "kv_heads": G, "dim": n, "vdim": p, "scale": c,
                           "rot": null | {"base": b, "dims": r, "scaling": null | {"factor": f}},
                           "mask": null | {"size": w}},
                 "mlp": null | {"kind": "dense", "ff": f}
                             | {"kind": "moe", "expert": {"ff": f, "limit": l},
                                "router": {"experts": E, "top": k, "scale": s, "groups": null | {"count": c, "keep": m}},
                                "shared": null | {"ff": f, "limit": l}}},
                {"type": "parallel",
                 "mixer": {"left": {...an attention...}, "right": {"heads": H, "dim": n, "vdim": p, "gate_cap": c},
                           "left_scale": a, "right_scale": b}, "mlp": ...},
                {"type": "rglru", "mixer": {"width": w, "blocks": b, "conv": taps}, "mlp": ...}, ...]}

Tensor names: ``embed``, ``head``, ``final.norm``, ``final.norm.b`` and, for layer i, ``l<i>.norm1|norm2`` and their ``.b``,
``l<i>.hc1|hc2.in|out|mix``, ``l<i>.mix.*``, ``l<i>.mlp.*``.  Every pass of the looped span keeps its own cache and state.

Every size and every constant that can differ between two models of the design comes from the file; what the design fixes
(which norm, which activation, the pairing of the rotation, the factor of the recurrence's decay) is in the parts this
description names.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple, Union

from .llama import _need, _opt
from .monolix import _obj
from .ragilorn import _positive
from .registry import ConfigError, register_architecture
from .spec import ArchitectureSpec, LayerSpec, PartSpec, RunEntry

# Angles are formed from the position itself and the recurrences have no horizon: the cache's size bounds a sequence.
NO_CONTEXT_LIMIT = 1 << 20
MAX_STREAMS = 8
GLU_ALPHA, GLU_OFFSET = 1.702, 1.0      # of an expert's clamped gated product
DECAY_RATE = 8.0                        # of the recurrent unit's decay
GROUP_TOP = 2                           # choice scores that make a group's score


def _number(d: Mapping[str, Any], key: str, where: str, positive: bool = False) -> float:
    try:
        v = _need(d, key, float)
    except ConfigError as e:
        raise ConfigError(f"config.json: {where}{key}: {e}") from None
    if positive and not v > 0:
        raise ConfigError(f"config.json: {where}{key} must be positive, got {v}")
    return v


@dataclass(frozen=True)
class BonusunAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: Optional[float]       # None: no rotation
    rot_dims: int
    rot_factor: Optional[float]     # None: frequencies as they are
    window: Optional[int]           # None: every earlier position

    kind = "attention"

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str) -> "BonusunAttention":
        heads, kv, dim, vdim = (_positive(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim"))
        if heads % kv:
            raise ConfigError(f"config.json: {where}kv_heads ({kv}) must divide heads ({heads})")
        base, dims, factor = None, 0, None
        rot = _obj(m, "rot", where, required=False)
        if rot is not None:
            base, dims = _number(rot, "base", where + "rot.", positive=True), _need(rot, "dims", int)
            if dims % 2 or not 0 <= dims <= dim:
                raise ConfigError(f"config.json: {where}rot.dims must be even and at most dim ({dim}), got {dims}")
            scaling = _obj(rot, "scaling", where + "rot.", required=False)
            if scaling is not None:
                factor = _number(scaling, "factor", where + "rot.scaling.", positive=True)
            if dims == 0:
                base, factor = None, None
        mask = _obj(m, "mask", where, required=False)
        window = None if mask is None else _positive(mask, "size", where + "mask.")
        return cls(heads, kv, dim, vdim, _number(m, "scale", where), base, dims, factor, window)

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "scale": self.scale}
        if self.rot_base is not None:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.rot_factor is not None:
                d["rot"]["scaling"] = {"factor": self.rot_factor}
        if self.window is not None:
            d["mask"] = {"size": self.window}
        return d

    def position_encoding(self) -> Optional[str]:
        if self.rot_base is None:
            return None
        return f"rotary_{self.dim}_{self.rot_dims}_{self.rot_base!r}_{self.rot_factor!r}"

    def position_spec(self) -> PartSpec:
        scaling = None if self.rot_factor is None else {"rope_type": "linear", "factor": self.rot_factor}
        return PartSpec("rotary_frequencies", {"head_dim": self.dim, "rotary_dim": self.rot_dims, "theta": self.rot_base,
                                               "scaling": scaling})

    def part(self, width: int, eps: float) -> PartSpec:
        return PartSpec("headnorm_attention", {
            "hidden_size": width, "num_heads": self.heads, "num_kv_heads": self.kv_heads, "qk_dim": self.dim,
            "v_dim": self.vdim, "scale": self.scale, "eps": eps, "window": self.window,
            "position_encoding": self.position_encoding(), "sink": True,
            # (a windowed group gives pages back early, so the window is part of its name)
            "cache_group": "full" if self.window is None else f"window{self.window}",
            "names": {"q": "q", "k": "k", "v": "v", "q_norm": "q.norm", "k_norm": "k.norm", "sink": "sink", "out": "o"}})


@dataclass(frozen=True)
class BonusunMemory:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str) -> "BonusunMemory":
        return cls(*(_positive(m, k, where) for k in ("heads", "dim", "vdim")), _number(m, "gate_cap", where, positive=True))

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "gate_cap": self.gate_cap}

    def part(self, width: int, eps: float) -> PartSpec:
        return PartSpec("matrix_memory", {
            "hidden_size": width, "num_heads": self.heads, "qk_dim": self.dim, "v_dim": self.vdim, "gate_cap": self.gate_cap,
            "eps": eps, "names": {"q": "q", "k": "k", "v": "v", "gate": "g", "out": "o", "norm": "norm", "input_gate": "i",
                                  "input_gate_bias": "i.b", "forget_gate": "f", "forget_gate_bias": "f.b"}})


@dataclass(frozen=True)
class BonusunParallel:
    left: BonusunAttention
    right: BonusunMemory
    left_scale: float
    right_scale: float

    kind = "parallel"

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str) -> "BonusunParallel":
        return cls(BonusunAttention.read(_obj(m, "left", where), where + "left."),
                   BonusunMemory.read(_obj(m, "right", where), where + "right."),
                   _number(m, "left_scale", where), _number(m, "right_scale", where))

    def to_dict(self) -> Dict[str, Any]:
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale,
                "right_scale": self.right_scale}

    def part(self, width: int, eps: float) -> PartSpec:
        return PartSpec("parallel_mixers", {"mixers": (("left.", self.left.part(width, eps), self.left_scale),
                                                       ("right.", self.right.part(width, eps), self.right_scale))})


@dataclass(frozen=True)
class BonusunRecurrent:
    width: int
    blocks: int
    conv: int

    kind = "rglru"

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str) -> "BonusunRecurrent":
        r = cls(*(_positive(m, k, where) for k in ("width", "blocks", "conv")))
        if r.width % r.blocks:
            raise ConfigError(f"config.json: {where}blocks ({r.blocks}) must divide width ({r.width})")
        return r

    def to_dict(self) -> Dict[str, Any]:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}

    def part(self, width: int, eps: float) -> PartSpec:
        return PartSpec("rglru", {
            "hidden_size": width, "width": self.width, "parts": self.blocks, "conv_taps": self.conv, "rate": DECAY_RATE,
            "names": {"y": "y", "y_bias": "y.b", "x": "x", "x_bias": "x.b", "conv": "conv", "conv_bias": "conv.b", "r": "ra",
                      "r_bias": "ra.b", "i": "ri", "i_bias": "ri.b", "decay": "lam", "out": "o"}})


@dataclass(frozen=True)
class BonusunDense:
    ff: int

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": "dense", "ff": self.ff}

    def part(self, width: int) -> PartSpec:
        return PartSpec("two_matrix_mlp", {"hidden_size": width, "intermediate_size": self.ff, "activation": "gelu_tanh",
                                           "names": {"up": "up", "down": "down"}})


@dataclass(frozen=True)
class BonusunMoE:
    ff: int
    limit: float
    experts: int
    top: int
    scale: float
    group_count: int                # 1 and 1: no groups
    group_keep: int
    shared_ff: Optional[int]        # None: no shared expert
    shared_limit: float

    @classmethod
    def read(cls, mlp: Mapping[str, Any], where: str) -> "BonusunMoE":
        e, r = _obj(mlp, "expert", where), _obj(mlp, "router", where)
        experts, top = _positive(r, "experts", where + "router."), _positive(r, "top", where + "router.")
        groups = _obj(r, "groups", where + "router.", required=False)
        count, keep = (1, 1) if groups is None else (_positive(groups, "count", where + "router.groups."),
                                                     _positive(groups, "keep", where + "router.groups."))
        if experts % count or keep > count:
            raise ConfigError(f"config.json: {where}router: {experts} experts do not form {count} equal groups of which "
                              f"{keep} are kept")
        if top > keep * (experts // count):
            raise ConfigError(f"config.json: {where}router.top is {top}; the kept groups hold {keep * (experts // count)}")
        shared = _obj(mlp, "shared", where, required=False)
        ff, limit = _positive(e, "ff", where + "expert."), _number(e, "limit", where + "expert.", positive=True)
        return cls(ff, limit, experts, top, _opt(r, "scale", float, 1.0), count, keep,
                   None if shared is None else _positive(shared, "ff", where + "shared."),
                   0.0 if shared is None else _number(shared, "limit", where + "shared.", positive=True))

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit},
                             "router": {"experts": self.experts, "top": self.top, "scale": self.scale,
                                        "groups": {"count": self.group_count, "keep": self.group_keep}}}
        if self.shared_ff is not None:
            d["shared"] = {"ff": self.shared_ff, "limit": self.shared_limit}
        return d

    def part(self, width: int) -> PartSpec:
        return PartSpec("routed_experts", {
            "hidden_size": width, "intermediate_size": self.ff, "num_experts": self.experts, "top": self.top,
            "group_count": self.group_count, "group_keep": self.group_keep, "group_top": GROUP_TOP, "score": "sigmoid",
            "renormalize": True, "correction": True, "weight_scale": self.scale, "gated": True, "activation": "silu",
            "clamp": (self.limit, GLU_ALPHA, GLU_OFFSET), "shared_size": self.shared_ff, "shared_gate": True,
            "shared_clamp": None if self.shared_ff is None else (self.shared_limit, GLU_ALPHA, GLU_OFFSET),
            "names": {"router": "router", "correction": "correction", "expert": "e{}.", "gate": "gate", "up": "up",
                      "down": "down", "shared_gate_proj": "shared.gate", "shared_up": "shared.up",
                      "shared_down": "shared.down", "shared_gate": "shared.sg"}})


_MIXERS = {c.kind: c for c in (BonusunAttention, BonusunParallel, BonusunRecurrent)}
Mixer = Union[BonusunAttention, BonusunParallel, BonusunRecurrent]
MLP = Union[None, BonusunDense, BonusunMoE]


def _mlp(mlp: Any, where: str) -> MLP:
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"config.json: {where[:-1]} must be null or an object of kind 'dense' or 'moe'")
    return BonusunDense(_positive(mlp, "ff", where)) if mlp["kind"] == "dense" else BonusunMoE.read(mlp, where)


@dataclass(frozen=True)
class BonusunConfig:
    vocab: int
    width: int
    streams: int
    residual_mult: float
    norm_eps: float
    layers: Tuple[Tuple[Mixer, MLP], ...]
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    architecture: str = "Bonusun"

    # ------------------------------------------------------------------ parsing
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "BonusunConfig":
        layers_in = d.get("layers")
        if not isinstance(layers_in, (list, tuple)) or not layers_in:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers: List[Tuple[Mixer, MLP]] = []
        for i, L in enumerate(layers_in):
            where = f"layers[{i}]."
            if not isinstance(L, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = L.get("type")
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where}type is {kind!r}; this design has {', '.join(sorted(_MIXERS))}")
            layers.append((_MIXERS[kind].read(_obj(L, "mixer", where), where + "mixer."), _mlp(L.get("mlp"), where + "mlp.")))
        n = len(layers)
        loop = _obj(d, "loop", "", required=False)
        a, b, times = 0, 0, 1
        if loop is not None:
            a, b, times = _need(loop, "start", int), _need(loop, "stop", int), _need(loop, "times", int)
            if not (0 <= a <= b <= n) or times < 1:
                raise ConfigError(f"config.json: loop {a}..{b} x {times} does not fit {n} layers")
        streams = _opt(d, "streams", int, 1)
        if not 1 <= streams <= MAX_STREAMS:
            raise ConfigError(f"config.json: 'streams' must be 1 to {MAX_STREAMS}, got {streams}")
        return cls(vocab=_positive(d, "vocab", ""), width=_positive(d, "width", ""), streams=streams,
                   residual_mult=_opt(d, "residual_mult", float, 1.0), norm_eps=_number(_obj(d, "norm", ""), "eps", "norm."),
                   layers=tuple(layers), loop_start=a, loop_stop=b, loop_times=times,
                   architecture=str(d.get("architecture") or (d.get("architectures") or ["Bonusun"])[0]))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
                "residual_mult": self.residual_mult, "norm": {"eps": self.norm_eps},
                "layers": [{"type": m.kind, "mixer": m.to_dict(), "mlp": None if f is None else f.to_dict()}
                           for m, f in self.layers],
                "loop": {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}}

    # ------------------------------------------------------- architecture as data
    def run_order(self) -> List[int]:
        """Layer indices in the order they run: the looped span repeats in a row, the rest follow."""
        span = list(range(self.loop_start, self.loop_stop))
        return list(range(self.loop_start)) + span * self.loop_times + list(range(self.loop_stop, len(self.layers)))

    def architecture_spec(self) -> ArchitectureSpec:
        d = self.width
        norm = PartSpec("layernorm", {"size": d, "eps": self.norm_eps, "name": "", "bias_name": ".b"})
        conn = PartSpec("hyper_connection", {"streams": self.streams, "result_scale": self.residual_mult,
                                             "names": {"read": "in", "write": "out", "mix": "mix"}})
        layers: List[LayerSpec] = []
        positions: Dict[str, PartSpec] = {}
        for i, (mixer, mlp) in enumerate(self.layers):
            for a in (mixer, getattr(mixer, "left", None)):
                if isinstance(a, BonusunAttention) and a.position_encoding() is not None:
                    positions[a.position_encoding()] = a.position_spec()
            norms, connections = {"mixer_norm": norm}, {"mixer_conn": conn}
            names = {"mixer": "mix.", "mixer_norm": "norm1", "mixer_conn": "hc1."}
            ffn = None
            if mlp is not None:
                ffn = mlp.part(d)
                norms["ffn_norm"], connections["ffn_conn"] = norm, conn
                names.update({"ffn": "mlp.", "ffn_norm": "norm2", "ffn_conn": "hc2."})
            layers.append(LayerSpec(prefix=f"l{i}.", block="hyper_prenorm", mixer=mixer.part(d, self.norm_eps), ffn=ffn,
                                    norms=norms, names=names, connections=connections))
        spec = ArchitectureSpec(
            name=self.architecture, hidden_size=d, vocab_size=self.vocab, max_positions=NO_CONTEXT_LIMIT,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": d, "name": "embed"}),
            embedding_prefix="",
            layers=layers,
            order=[RunEntry(i) for i in self.run_order()],     # every pass of a repeated layer keeps its own cache
            final_norm=norm, final_norm_prefix="final.norm",
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": d, "tied_to": None, "name": "head"}),
            head_prefix="",
            position_encodings=positions,
            bos_token_id=None, stop_token_ids=(),
            streams=self.streams,
        )
        spec.validate()
        return spec


register_architecture("Bonusun", BonusunConfig)
