"""Typed configuration of the Nafazen decoder, read from its ``config.json``.

The file lists the layers one by one; every layer names its type and carries the sizes and constants of its mixer
and of its feed-forward (or ``null`` for none), so layers of one model may differ.  Keys read here:

    architecture, vocab, width, norm.eps, embedding.scale (optional, 1), logit_softcap (optional), max_positions (optional)
    layers[i].type    "latent_attention" | "latent_attention_2"
    layers[i].mixer   heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, kv_from (optional: the layer whose cached rows
                      this one reads), rot.{dims, base, scaling.{factor, original, fast, slow}} (rot and scaling optional)
    layers[i].mlp     null, {kind: "dense", ff}, or
                      {kind: "moe", expert.ff, router.{experts, top}, shared.ff (shared optional)}
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Union

from lily_b200.config.model_config import ConfigError, RopeScaling
from lily_b200.config.zirurax_config import _need

MIXERS = ("latent_attention", "latent_attention_2")      # the two kinds differ in what their ``mixer`` holds, not in how it is read


@dataclass(frozen=True)
class NafazenAttentionConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rotary_dims: int                  # 0: no rotation
    rotary_base: float
    rotary_scaling: RopeScaling
    kv_from: Optional[int]            # None: the layer caches rows of its own

    @classmethod
    def from_dict(cls, d: Dict[str, Any], where: str) -> "NafazenAttentionConfig":
        rot = d.get("rot") or {}
        source = d.get("kv_from")
        out = cls(heads=_need(d, "heads", where), dim=_need(d, "dim", where), rot_dim=_need(d, "rot_dim", where),
                  vdim=_need(d, "vdim", where), q_rank=_need(d, "q_rank", where), kv_rank=_need(d, "kv_rank", where),
                  scale=_need(d, "scale", where, float), rotary_dims=int(rot.get("dims") or 0),
                  rotary_base=float(rot.get("base") or 10000.0),
                  rotary_scaling=RopeScaling.yarn(rot.get("scaling"), f"{where}.rot.scaling"),
                  kv_from=None if source is None else int(source))
        if min(out.heads, out.dim, out.vdim, out.q_rank, out.kv_rank) < 1 or out.rot_dim < 0:
            raise ConfigError(f"{where}: sizes must be positive")
        if out.rotary_dims < 0 or out.rotary_dims % 2 or out.rotary_dims > out.rot_dim:
            raise ConfigError(f"{where}.rot.dims {out.rotary_dims} must be even and within rot_dim {out.rot_dim}")
        if out.rotary_dims and not out.rotary_base > 1.0:
            raise ConfigError(f"{where}.rot.base must be above one")
        if not out.scale > 0:
            raise ConfigError(f"{where}.scale must be positive")
        return out

    @property
    def cached(self):
        """What a layer that reads this one's rows must agree with."""
        return self.kv_rank, self.rot_dim, self.rotary_dims, self.rotary_base, self.rotary_scaling


@dataclass(frozen=True)
class NafazenDenseConfig:
    ff: int


@dataclass(frozen=True)
class NafazenMoeConfig:
    ff: int
    experts: int
    top: int
    shared_ff: int                    # 0: no shared expert

    @classmethod
    def from_dict(cls, d: Dict[str, Any], where: str) -> "NafazenMoeConfig":
        router, shared = d.get("router") or {}, d.get("shared")
        out = cls(ff=_need(d.get("expert") or {}, "ff", f"{where}.expert"), experts=_need(router, "experts", f"{where}.router"),
                  top=_need(router, "top", f"{where}.router"), shared_ff=_need(shared, "ff", f"{where}.shared") if shared else 0)
        if out.ff < 1 or not 1 <= out.top <= out.experts or out.shared_ff < 0:
            raise ConfigError(f"{where}: top {out.top} of {out.experts} experts, ff {out.ff}, shared {out.shared_ff}")
        return out


@dataclass(frozen=True)
class NafazenLayerConfig:
    type: str
    mixer: NafazenAttentionConfig
    mlp: Union[None, NafazenDenseConfig, NafazenMoeConfig]


@dataclass
class NafazenConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    embed_scale: float
    logit_softcap: Optional[float]
    layers: List[NafazenLayerConfig]
    max_positions: int = 1 << 17
    torch_dtype: str = "bfloat16"

    @classmethod
    def from_dict(cls, cfg: Dict[str, Any], generation: Optional[Dict[str, Any]] = None,
                  architecture: Optional[str] = None) -> "NafazenConfig":
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
            if mlp is None:
                ff = None
            elif mlp.get("kind") == "dense":
                ff = NafazenDenseConfig(_need(mlp, "ff", f"{where}.mlp"))
                if ff.ff < 1:
                    raise ConfigError(f"{where}.mlp.ff must be positive")
            elif mlp.get("kind") == "moe":
                ff = NafazenMoeConfig.from_dict(mlp, f"{where}.mlp")
            else:
                raise ConfigError(f"{where}.mlp.kind {mlp.get('kind')!r} is not a feed-forward of this architecture (have: dense, moe)")
            layers.append(NafazenLayerConfig(kind, NafazenAttentionConfig.from_dict(layer.get("mixer") or {}, f"{where}.mixer"), ff))
        embedding = cfg.get("embedding") or {}
        cap = cfg.get("logit_softcap")
        out = cls(architecture=architecture or str(cfg.get("architecture", "Nafazen")),
                  vocab=_need(cfg, "vocab", "config"), width=_need(cfg, "width", "config"),
                  eps=_need(cfg.get("norm") or {}, "eps", "norm", float),
                  embed_scale=float(embedding["scale"]) if embedding.get("scale") is not None else 1.0,
                  logit_softcap=float(cap) if cap else None, layers=layers,
                  max_positions=int(cfg.get("max_positions") or (1 << 17)), torch_dtype=str(cfg.get("torch_dtype") or "bfloat16"))
        if out.vocab < 1 or out.width < 1 or not out.eps > 0:
            raise ConfigError("vocab and width must be positive, norm.eps above zero")
        for i, layer in enumerate(layers):
            j = layer.mixer.kv_from
            if j is None:
                continue
            if not 0 <= j < i or layers[j].mixer.kv_from is not None:
                raise ConfigError(f"layers[{i}].mixer.kv_from = {j} names no earlier layer with cached rows of its own")
            if layers[j].mixer.cached != layer.mixer.cached:
                raise ConfigError(f"layers[{i}] cannot read the rows of layers[{j}]: another latent, rotated part or rotation")
        return out

    def summary(self) -> str:
        readers = sum(1 for layer in self.layers if layer.mixer.kv_from is not None)
        return (f"{self.architecture} layers={len(self.layers)} (reading another's cache: {readers}) width={self.width} "
                f"vocab={self.vocab} eps={self.eps}")
