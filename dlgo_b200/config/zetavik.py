"""Typed configuration of the Zetavik design, read from its config.json keys.

A Zetavik model is a list of layers whose mixer and feed-forward stand side by side behind one layer norm
(``x <- x + (mixer(n) + ff(n))``, ``n = norm(x)``); the head is the embedding table.  A layer's mixer is a
state-space recurrence with a scalar decay per head and token, latent attention (queries and keys through latents, a
rotated part, an output gate per head), or linear attention with a fixed decay per head.  The feed-forward is a dense
one with the square of relu, a mixture of gated experts chosen within the best groups plus a shared expert, or absent:

    {"architecture": "Zetavik", "vocab": V, "width": d, "norm": {"eps": e},
     "layers": [{"type": "mamba2" | "latent_attention" | "lightning",
                 "mixer": {...sizes and constants of the mixer...},
                 "mlp": null | {"kind": "dense", "ff": f}
                             | {"kind": "moe", "expert": {"ff": f},
                                "router": {"experts": E, "top": k, "scale": s, "groups": {"count": c, "keep": m}},
                                "shared": {"ff": fs}}}, ...]}

Tensor names: ``embed``, ``final.norm`` and, for layer i, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``.

Every size and every constant that can differ between two models of the design comes from the file; constants the
design fixes (which norm, which activation, the pairing of the rotation) are in the parts this description names.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Mapping, Optional, Tuple, Union

from .llama import _as, _need, _opt
from .monolix import _obj
from .ragilorn import _positive
from .registry import ConfigError, register_architecture
from .spec import ArchitectureSpec, LayerSpec, PartSpec, RunEntry

MIXER_KINDS = ("mamba2", "latent_attention", "lightning")
# Angles are formed from the position itself and the recurrences have no horizon: the cache's size bounds a sequence.
NO_CONTEXT_LIMIT = 1 << 20


@dataclass(frozen=True)
class ZetavikStateSpace:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    kind = "mamba2"

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str) -> "ZetavikStateSpace":
        r = cls(*(_positive(m, k, where) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))
        if r.heads % r.groups:
            raise ConfigError(f"config.json: {where}groups ({r.groups}) must divide heads ({r.heads})")
        if (r.heads * r.vdim) % r.norm_groups:
            raise ConfigError(f"config.json: {where}norm_groups ({r.norm_groups}) must divide heads * vdim "
                              f"({r.heads * r.vdim})")
        return r

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.conv,
                "norm_groups": self.norm_groups}


@dataclass(frozen=True)
class ZetavikLatent:
    heads: int
    dim: int                    # unrotated query/key size of a head
    rot_dim: int                # rotated part of a head
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float

    kind = "latent_attention"

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str) -> "ZetavikLatent":
        sizes = [_positive(m, k, where) for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank")]
        if sizes[2] % 2:
            raise ConfigError(f"config.json: {where}rot_dim must be even, got {sizes[2]}")
        rot = _obj(m, "rot", where)
        base = _need(rot, "base", float)
        dims = _opt(rot, "dims", int, sizes[2])
        if base <= 0 or dims != sizes[2]:
            raise ConfigError(f"config.json: {where}rot.base must be positive and rot.dims equal rot_dim ({sizes[2]}): "
                              "the rotated part turns as a whole")
        return cls(*sizes, _need(m, "scale", float), base)

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
                "kv_rank": self.kv_rank, "scale": self.scale, "rot": {"base": self.rot_base, "dims": self.rot_dim}}


@dataclass(frozen=True)
class ZetavikLightning:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    kind = "lightning"

    @classmethod
    def read(cls, m: Mapping[str, Any], where: str) -> "ZetavikLightning":
        heads, dim, vdim = (_positive(m, k, where) for k in ("heads", "dim", "vdim"))
        decay = m.get("decay")
        if not isinstance(decay, (list, tuple)) or len(decay) != heads:
            raise ConfigError(f"config.json: {where}decay must list one number per head ({heads})")
        return cls(heads, dim, vdim, tuple(_as(x, "decay", float) for x in decay))

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


@dataclass(frozen=True)
class ZetavikDense:
    ff: int

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class ZetavikMoE:
    ff: int
    experts: int
    top: int
    scale: float
    group_count: int            # 1 and 1: no groups
    group_keep: int
    shared_ff: Optional[int]    # None: no shared expert

    @classmethod
    def read(cls, mlp: Mapping[str, Any], where: str) -> "ZetavikMoE":
        ff = _positive(_obj(mlp, "expert", where), "ff", where + "expert.")
        r = _obj(mlp, "router", where)
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
        return cls(ff, experts, top, _opt(r, "scale", float, 1.0), count, keep,
                   None if shared is None else _positive(shared, "ff", where + "shared."))

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff},
                             "router": {"experts": self.experts, "top": self.top, "scale": self.scale,
                                        "groups": {"count": self.group_count, "keep": self.group_keep}}}
        if self.shared_ff is not None:
            d["shared"] = {"ff": self.shared_ff}
        return d


_MIXERS = {c.kind: c for c in (ZetavikStateSpace, ZetavikLatent, ZetavikLightning)}
Mixer = Union[ZetavikStateSpace, ZetavikLatent, ZetavikLightning]
MLP = Union[None, ZetavikDense, ZetavikMoE]


def _mlp(mlp: Any, where: str) -> MLP:
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"config.json: {where[:-1]} must be null or an object of kind 'dense' or 'moe'")
    return ZetavikDense(_positive(mlp, "ff", where)) if mlp["kind"] == "dense" else ZetavikMoE.read(mlp, where)


@dataclass(frozen=True)
class ZetavikConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[Tuple[Mixer, MLP], ...]
    architecture: str = "Zetavik"

    # ------------------------------------------------------------------ parsing
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "ZetavikConfig":
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
                raise ConfigError(f"config.json: {where}type is {kind!r}; this design has {', '.join(MIXER_KINDS)}")
            layers.append((_MIXERS[kind].read(_obj(L, "mixer", where), where + "mixer."),
                           _mlp(L.get("mlp"), where + "mlp.")))
        return cls(vocab=_positive(d, "vocab", ""), width=_positive(d, "width", ""),
                   norm_eps=_need(_obj(d, "norm", ""), "eps", float), layers=tuple(layers),
                   architecture=str(d.get("architecture") or (d.get("architectures") or ["Zetavik"])[0]))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps},
                "layers": [{"type": m.kind, "mixer": m.to_dict(), "mlp": None if f is None else f.to_dict()}
                           for m, f in self.layers]}

    # ------------------------------------------------------- architecture as data
    def _mixer_spec(self, m: Mixer, positions: Dict[str, PartSpec]) -> PartSpec:
        d, eps = self.width, self.norm_eps
        if isinstance(m, ZetavikStateSpace):
            return PartSpec("mamba2", {
                "hidden_size": d, "num_heads": m.heads, "v_dim": m.vdim, "state_size": m.state, "num_groups": m.groups,
                "conv_taps": m.conv, "norm_groups": m.norm_groups, "eps": eps,
                "names": {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "decay": "A_log",
                          "skip": "D", "norm": "norm", "out": "o"}})
        if isinstance(m, ZetavikLightning):
            return PartSpec("lightning_attention", {
                "hidden_size": d, "num_heads": m.heads, "qk_dim": m.dim, "v_dim": m.vdim, "decay": m.decay, "eps": eps,
                "names": {"q": "q", "k": "k", "v": "v", "gate": "g", "out": "o", "norm": "norm"}})
        pe = f"rotary_{m.rot_dim}_{m.rot_base!r}"
        positions.setdefault(pe, PartSpec("rotary_frequencies", {"head_dim": m.rot_dim, "rotary_dim": m.rot_dim,
                                                                 "theta": m.rot_base}))
        return PartSpec("latent_attention", {
            "hidden_size": d, "num_heads": m.heads, "qk_dim": m.dim, "v_dim": m.vdim, "kv_rank": m.kv_rank,
            "q_rank": m.q_rank, "scale": m.scale, "eps": eps, "rope_dim": m.rot_dim, "position_encoding": pe,
            "head_gate": True, "cache_group": "latent",
            "names": {"q_down": "dq", "q_norm": "dq.norm", "q_up": "uq", "kv_down": "dkv", "kv_norm": "dkv.norm",
                      "k_up": "uk", "v_up": "uv", "gate": "g", "out": "o"}})

    def _ffn_spec(self, f: Union[ZetavikDense, ZetavikMoE]) -> PartSpec:
        if isinstance(f, ZetavikDense):
            return PartSpec("relu2_mlp", {"hidden_size": self.width, "intermediate_size": f.ff,
                                          "names": {"up": "up", "down": "down"}})
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "intermediate_size": f.ff, "num_experts": f.experts, "top": f.top,
            "group_count": f.group_count, "group_keep": f.group_keep, "score": "softmax", "renormalize": False,
            "weight_scale": f.scale, "gated": True, "activation": "silu", "shared_size": f.shared_ff,
            "names": {"router": "router", "expert": "e{}.", "gate": "gate", "up": "up", "down": "down",
                      "shared_gate_proj": "shared.gate", "shared_up": "shared.up", "shared_down": "shared.down"}})

    def architecture_spec(self) -> ArchitectureSpec:
        d = self.width
        norm = PartSpec("layernorm", {"size": d, "eps": self.norm_eps, "name": ""})
        positions: Dict[str, PartSpec] = {}
        layers: List[LayerSpec] = []
        for i, (m, f) in enumerate(self.layers):
            names = {"mixer": "mix.", "mixer_norm": "norm1"}
            if f is not None:
                names["ffn"] = "mlp."
            layers.append(LayerSpec(prefix=f"l{i}.", block="parallel_prenorm", mixer=self._mixer_spec(m, positions),
                                    ffn=None if f is None else self._ffn_spec(f), norms={"mixer_norm": norm}, names=names))
        spec = ArchitectureSpec(
            name=self.architecture, hidden_size=d, vocab_size=self.vocab, max_positions=NO_CONTEXT_LIMIT,
            embedding=PartSpec("token_embedding", {"vocab_size": self.vocab, "hidden_size": d, "name": "embed"}),
            embedding_prefix="",
            layers=layers, order=[RunEntry(i) for i in range(len(layers))],
            final_norm=norm, final_norm_prefix="final.norm",
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "hidden_size": d, "tied_to": "embed"}),
            head_prefix="",
            position_encodings=positions,
            bos_token_id=None, stop_token_ids=(),
        )
        spec.validate()
        return spec


register_architecture("Zetavik", ZetavikConfig)
