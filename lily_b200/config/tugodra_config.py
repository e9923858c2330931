"""Typed configuration of the Tugodra decoder, read from its ``config.json``.

The file lists the layers one by one; every layer names the type of its mixer and carries the sizes and constants of the
mixer and of its feed-forward (or ``null`` for none), so layers of one model may differ.  Keys read here:

    architecture, vocab, width, norm.eps, embedding.scale (optional, 1), max_positions (optional)
    layers[i].type    "attention" | "latent_attention" | "mlstm"
    layers[i].mixer   attention: heads, kv_heads, dim, vdim, scale, mask.size (optional: all keys), rot.{dims, base}
                      (optional), kv_from (optional: the layer whose keys and values this one reads)
                      latent_attention: heads, dim, rot_dim, vdim, kv_rank, scale, rot.{dims, base} (optional)
                      mlstm: heads, dim, vdim, gate_cap
    layers[i].mlp     null, or {kind: "moe", expert.ff, router.{experts, top, groups.{count, keep}}, shared.ff}
                      (groups and shared optional)
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Union

from lily_b200.config.model_config import ConfigError
from lily_b200.config.zirurax_config import _need


def _rotation(d: Dict[str, Any], width: int, where: str):
    """(rotated dimensions, base) of a mixer whose rotated part has ``width`` columns; (0, _) without rotation."""
    rot = d.get("rot") or {}
    dims, base = int(rot.get("dims") or 0), float(rot.get("base") or 10000.0)
    if dims < 0 or dims % 2 or dims > width:
        raise ConfigError(f"{where}.rot.dims {dims} must be even and within {width}")
    if dims and not base > 0.0:
        raise ConfigError(f"{where}.rot.base must be positive")
    return dims, base


@dataclass(frozen=True)
class TugodraAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]             # None: all keys
    rotary_dims: int                  # 0: no rotation
    rotary_base: float
    kv_from: Optional[int]            # None: the layer caches keys and values of its own

    @classmethod
    def from_dict(cls, d: Dict[str, Any], where: str) -> "TugodraAttentionConfig":
        size, source = (d.get("mask") or {}).get("size"), d.get("kv_from")
        dim = _need(d, "dim", where)
        dims, base = _rotation(d, dim, where)
        out = cls(heads=_need(d, "heads", where), kv_heads=_need(d, "kv_heads", where), dim=dim, vdim=_need(d, "vdim", where),
                  scale=_need(d, "scale", where, float), window=None if size is None else int(size), rotary_dims=dims, rotary_base=base,
                  kv_from=None if source is None else int(source))
        if min(out.heads, out.kv_heads, out.dim, out.vdim) < 1 or out.heads % out.kv_heads:
            raise ConfigError(f"{where}: sizes must be positive and heads a multiple of kv_heads")
        if not out.scale > 0 or (out.window is not None and out.window < 1):
            raise ConfigError(f"{where}: scale and mask.size must be positive")
        return out

    @property
    def cached(self):
        """What a layer that reads this one's keys and values must agree with."""
        return self.kv_heads, self.dim, self.vdim, self.rotary_dims, self.rotary_base


@dataclass(frozen=True)
class TugodraLatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rotary_dims: int
    rotary_base: float

    @classmethod
    def from_dict(cls, d: Dict[str, Any], where: str) -> "TugodraLatentConfig":
        if d.get("kv_from") is not None:
            raise ConfigError(f"{where}.kv_from: only attention layers read another layer's keys and values")
        rot_dim = _need(d, "rot_dim", where)
        dims, base = _rotation(d, rot_dim, where)
        out = cls(heads=_need(d, "heads", where), dim=_need(d, "dim", where), rot_dim=rot_dim, vdim=_need(d, "vdim", where),
                  kv_rank=_need(d, "kv_rank", where), scale=_need(d, "scale", where, float), rotary_dims=dims, rotary_base=base)
        if min(out.heads, out.dim, out.vdim, out.kv_rank) < 1 or out.rot_dim < 0 or not out.scale > 0:
            raise ConfigError(f"{where}: sizes and scale must be positive")
        return out


@dataclass(frozen=True)
class TugodraMlstmConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, d: Dict[str, Any], where: str) -> "TugodraMlstmConfig":
        out = cls(heads=_need(d, "heads", where), dim=_need(d, "dim", where), vdim=_need(d, "vdim", where),
                  gate_cap=_need(d, "gate_cap", where, float))
        if min(out.heads, out.dim, out.vdim) < 1 or not out.gate_cap > 0:
            raise ConfigError(f"{where}: sizes and gate_cap must be positive")
        return out


MIXERS = {"attention": TugodraAttentionConfig, "latent_attention": TugodraLatentConfig, "mlstm": TugodraMlstmConfig}


@dataclass(frozen=True)
class TugodraMoeConfig:
    ff: int
    experts: int
    top: int
    groups: int                       # 0: the choice is among all experts
    keep_groups: int
    shared_ff: int                    # 0: no shared expert

    @classmethod
    def from_dict(cls, d: Dict[str, Any], where: str) -> "TugodraMoeConfig":
        if d.get("kind", "moe") != "moe":
            raise ConfigError(f"{where}.kind {d.get('kind')!r} is not a feed-forward of this architecture (have: moe)")
        router, shared = d.get("router") or {}, d.get("shared")
        groups = router.get("groups") or {}
        out = cls(ff=_need(d.get("expert") or {}, "ff", f"{where}.expert"), experts=_need(router, "experts", f"{where}.router"),
                  top=_need(router, "top", f"{where}.router"), groups=_need(groups, "count", f"{where}.router.groups") if groups else 0,
                  keep_groups=_need(groups, "keep", f"{where}.router.groups") if groups else 0,
                  shared_ff=_need(shared, "ff", f"{where}.shared") if shared else 0)
        if out.ff < 1 or not 1 <= out.top <= out.experts or out.shared_ff < 0:
            raise ConfigError(f"{where}: top {out.top} of {out.experts} experts, ff {out.ff}, shared {out.shared_ff}")
        if groups and (out.groups < 1 or out.experts % out.groups or not 1 <= out.keep_groups <= out.groups
                       or out.top > out.keep_groups * (out.experts // out.groups)):
            raise ConfigError(f"{where}.router: top {out.top} of the best {out.keep_groups} of {out.groups} groups of {out.experts} experts")
        return out


@dataclass(frozen=True)
class TugodraLayerConfig:
    type: str
    mixer: Union[TugodraAttentionConfig, TugodraLatentConfig, TugodraMlstmConfig]
    mlp: Optional[TugodraMoeConfig]

    @property
    def kv_from(self) -> Optional[int]:
        return self.mixer.kv_from if isinstance(self.mixer, TugodraAttentionConfig) else None


@dataclass
class TugodraConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: List[TugodraLayerConfig]
    max_positions: int = 1 << 17
    torch_dtype: str = "bfloat16"

    @classmethod
    def from_dict(cls, cfg: Dict[str, Any], generation: Optional[Dict[str, Any]] = None,
                  architecture: Optional[str] = None) -> "TugodraConfig":
        listed = cfg.get("layers")
        if not isinstance(listed, list) or not listed:
            raise ConfigError("config.json lacks the list 'layers'")
        layers = []
        for i, layer in enumerate(listed):
            where = f"layers[{i}]"
            kind = layer.get("type")
            if kind not in MIXERS:
                raise ConfigError(f"{where}.type {kind!r} is not a layer type of this architecture (have: {', '.join(MIXERS)})")
            mlp = layer.get("mlp")
            layers.append(TugodraLayerConfig(kind, MIXERS[kind].from_dict(layer.get("mixer") or {}, f"{where}.mixer"),
                                             None if mlp is None else TugodraMoeConfig.from_dict(mlp, f"{where}.mlp")))
        embedding = cfg.get("embedding") or {}
        out = cls(architecture=architecture or str(cfg.get("architecture", "Tugodra")),
                  vocab=_need(cfg, "vocab", "config"), width=_need(cfg, "width", "config"),
                  eps=_need(cfg.get("norm") or {}, "eps", "norm", float),
                  embed_scale=float(embedding["scale"]) if embedding.get("scale") is not None else 1.0, layers=layers,
                  max_positions=int(cfg.get("max_positions") or (1 << 17)), torch_dtype=str(cfg.get("torch_dtype") or "bfloat16"))
        if out.vocab < 1 or out.width < 1 or not out.eps > 0:
            raise ConfigError("vocab and width must be positive, norm.eps above zero")
        for i, layer in enumerate(layers):
            j = layer.kv_from
            if j is None:
                continue
            if not 0 <= j < i or layers[j].type != "attention" or layers[j].kv_from is not None:
                raise ConfigError(f"layers[{i}].mixer.kv_from = {j} names no earlier attention layer with keys and values of its own")
            if layers[j].mixer.cached != layer.mixer.cached:
                raise ConfigError(f"layers[{i}] cannot read the keys of layers[{j}]: other heads, sizes or rotation")
        return out

    def summary(self) -> str:
        kinds = ", ".join(f"{k} {sum(1 for layer in self.layers if layer.type == k)}" for k in MIXERS)
        return f"{self.architecture} layers={len(self.layers)} ({kinds}) width={self.width} vocab={self.vocab} eps={self.eps}"
