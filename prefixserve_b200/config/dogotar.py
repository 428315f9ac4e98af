"""Typed Dogotar configuration, read from the keys of a model folder's config.json.

Dogotar is a decoder whose layers are listed one by one: each entry of ``layers`` names its mixer (``attention``: windowed, with
rotated positions; ``parallel``: a chunked attention without positions beside a matrix memory), the mixer's sizes, and its
feed-forward (dense, or none).  Keys:

    architecture: "Dogotar"
    vocab, width, norm.eps
    layers[i].type, layers[i].mixer.{...}, layers[i].mlp = {kind: "dense", ff} | null
      attention: heads, kv_heads, dim, vdim, scale, softcap, mask.size, v_mix,
                 rot.{base, dims, scaling.factor}
      parallel:  left.{heads, kv_heads, dim, vdim, scale, softcap, mask.size}, left_scale,
                 right.{heads, dim, vdim, gate_cap}, right_scale

Without ``mask`` an attention sees every earlier key, without ``softcap`` its scores are not capped, without ``rot`` nothing is
rotated, without ``rot.scaling`` the frequencies are as they are, without ``v_mix`` the values are the layer's own.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .llama import UnsupportedModelError
from .nerenex import _need, _positive

ARCHITECTURE = "Dogotar"


@dataclass(frozen=True)
class LinearRotation:
    base: float
    dims: int                # leading elements of a head that turn
    factor: float | None     # every frequency is divided by it; None: no scaling

    @staticmethod
    def from_dict(r: Mapping[str, Any], dim: int, where: str) -> "LinearRotation":
        dims = _positive(_need(r, "dims", where), f"{where}.dims")
        if dims % 2 or dims > dim:
            raise UnsupportedModelError(f"config.json: {where}.dims must be even and at most {dim}, is {dims}")
        scaling = r.get("scaling")
        factor = None if scaling is None else float(_need(scaling, "factor", f"{where}.scaling"))
        if factor is not None and not factor > 0:
            raise UnsupportedModelError(f"config.json: {where}.scaling.factor must be positive, is {factor}")
        return LinearRotation(base=float(_need(r, "base", where)), dims=dims, factor=factor)

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.factor is not None:
            out["scaling"] = {"factor": self.factor}
        return out


@dataclass(frozen=True)
class CappedAttentionConfig:
    """An attention's sizes; what ``reach`` means (a window or a chunk) is up to the layer that holds it."""

    heads: int
    kv_heads: int
    dim: int              # query/key size per head
    vdim: int             # value size per head
    scale: float
    softcap: float | None
    reach: int | None     # mask.size
    rot: LinearRotation | None = None
    v_mix: bool = False

    kind = "attention"

    @staticmethod
    def from_dict(m: Mapping[str, Any], where: str, plain: bool = False) -> "CappedAttentionConfig":
        """``plain``: a branch without positions and value mixing."""
        dim = _positive(_need(m, "dim", where), f"{where}.dim")
        mask, cap, rot = m.get("mask"), m.get("softcap"), None if plain else m.get("rot")
        cfg = CappedAttentionConfig(
            heads=_positive(_need(m, "heads", where), f"{where}.heads"),
            kv_heads=_positive(_need(m, "kv_heads", where), f"{where}.kv_heads"),
            dim=dim,
            vdim=_positive(m.get("vdim", dim), f"{where}.vdim"),
            scale=float(_need(m, "scale", where)),
            softcap=None if cap is None else float(cap),
            reach=None if mask is None or mask.get("size") is None else _positive(mask["size"], f"{where}.mask.size"),
            rot=None if rot is None else LinearRotation.from_dict(rot, dim, f"{where}.rot"),
            v_mix=False if plain else bool(m.get("v_mix", False)),
        )
        if cfg.heads % cfg.kv_heads:
            raise UnsupportedModelError(f"config.json: {where}: {cfg.heads} heads cannot share {cfg.kv_heads} key/value heads")
        if cfg.softcap is not None and not cfg.softcap > 0:
            raise UnsupportedModelError(f"config.json: {where}.softcap must be positive, is {cfg.softcap}")
        return cfg

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.softcap is not None:
            out["softcap"] = self.softcap
        if self.reach is not None:
            out["mask"] = {"size": self.reach}
        if self.rot is not None:
            out["rot"] = self.rot.to_dict()
        if self.v_mix:
            out["v_mix"] = True
        return out


@dataclass(frozen=True)
class MatrixMemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @staticmethod
    def from_dict(m: Mapping[str, Any], where: str) -> "MatrixMemoryConfig":
        dim = _positive(_need(m, "dim", where), f"{where}.dim")
        cfg = MatrixMemoryConfig(heads=_positive(_need(m, "heads", where), f"{where}.heads"), dim=dim,
                                 vdim=_positive(m.get("vdim", dim), f"{where}.vdim"), gate_cap=float(_need(m, "gate_cap", where)))
        if not cfg.gate_cap > 0:
            raise UnsupportedModelError(f"config.json: {where}.gate_cap must be positive, is {cfg.gate_cap}")
        return cfg

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "gate_cap": self.gate_cap}


@dataclass(frozen=True)
class PairConfig:
    left: CappedAttentionConfig
    right: MatrixMemoryConfig
    left_scale: float
    right_scale: float

    kind = "parallel"

    @staticmethod
    def from_dict(m: Mapping[str, Any], where: str) -> "PairConfig":
        return PairConfig(left=CappedAttentionConfig.from_dict(_need(m, "left", where), f"{where}.left", plain=True),
                          right=MatrixMemoryConfig.from_dict(_need(m, "right", where), f"{where}.right"),
                          left_scale=float(_need(m, "left_scale", where)), right_scale=float(_need(m, "right_scale", where)))

    def to_dict(self) -> dict[str, Any]:
        return {"left": self.left.to_dict(), "left_scale": self.left_scale, "right": self.right.to_dict(), "right_scale": self.right_scale}


_MIXERS = {"attention": CappedAttentionConfig, "parallel": PairConfig}


@dataclass(frozen=True)
class DogotarLayer:
    mixer: CappedAttentionConfig | PairConfig
    ff: int | None        # inner size of the dense feed-forward; None: no feed-forward


@dataclass(frozen=True)
class DogotarConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[DogotarLayer, ...]
    stop_token_ids: frozenset[int] = frozenset()

    architecture = ARCHITECTURE

    def value_source(self) -> int | None:
        """The layer whose values later layers mix into theirs: the first with ``v_mix``."""
        return next((i for i, layer in enumerate(self.layers) if getattr(layer.mixer, "v_mix", False)), None)

    @staticmethod
    def from_dicts(raw: Mapping[str, Any], generation: Mapping[str, Any] | None = None) -> "DogotarConfig":
        if raw.get("architecture") != ARCHITECTURE and ARCHITECTURE not in (raw.get("architectures") or []):
            raise UnsupportedModelError(f"config.json does not describe a {ARCHITECTURE} model")
        layers: list[DogotarLayer] = []
        for i, entry in enumerate(_need(raw, "layers", "the top level")):
            where = f"layers[{i}]"
            kind = _need(entry, "type", where)
            if kind not in _MIXERS:
                raise UnsupportedModelError(f"config.json: {where}.type {kind!r} is not one of {sorted(_MIXERS)}")
            mixer = _MIXERS[kind].from_dict(_need(entry, "mixer", where), f"{where}.mixer")
            mlp = entry.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise UnsupportedModelError(f"config.json: {where}.mlp.kind {mlp.get('kind')!r} is not built (dense)")
            layers.append(DogotarLayer(mixer, None if mlp is None else _positive(_need(mlp, "ff", f"{where}.mlp"), f"{where}.mlp.ff")))
        if not layers:
            raise UnsupportedModelError("config.json: a model needs at least one layer")
        stops: set[int] = set()
        eos = (generation or {}).get("eos_token_id")
        if eos is not None:
            stops.update(int(t) for t in (eos if isinstance(eos, (list, tuple)) else [eos]))
        cfg = DogotarConfig(
            vocab=_positive(_need(raw, "vocab", "the top level"), "vocab"),
            width=_positive(_need(raw, "width", "the top level"), "width"),
            norm_eps=float(_need(_need(raw, "norm", "the top level"), "eps", "norm")),
            layers=tuple(layers),
            stop_token_ids=frozenset(stops),
        )
        sizes = {layer.mixer.kv_heads * layer.mixer.vdim for layer in layers if getattr(layer.mixer, "v_mix", False)}
        if len(sizes) > 1:
            raise UnsupportedModelError(f"config.json: layers that mix values must have as many value channels, not {sorted(sizes)}")
        return cfg

    def to_config_json(self) -> dict[str, Any]:
        return {
            "architecture": ARCHITECTURE,
            "vocab": self.vocab,
            "width": self.width,
            "norm": {"eps": self.norm_eps},
            "layers": [{"type": layer.mixer.kind, "mixer": layer.mixer.to_dict(),
                        "mlp": None if layer.ff is None else {"kind": "dense", "ff": layer.ff}} for layer in self.layers],
        }
