"""The Nafazen decoder as a ``ModelSpec``.

Every layer is a post-norm block: ``x += norm1(mixer(x))`` and, where it has a feed-forward, ``x += norm2(ff(x))``; the norms
have one gain for all columns.  The mixer is a softmax attention over a cached low-rank latent (``latent_attention``, no
output gate, all keys) that rotates interleaved pairs, in some layers with YaRN-scaled frequencies; a layer with ``kv_from``
is a run of the schedule that ``reads`` another run's cache and projects no keys or values of its own.  The feed-forward is
``down(xielu(up x))``, or a routed mixture with sigmoid scores whose weights multiply the experts' inputs, with a gated
shared expert.  The embedding is scaled, the head is a table of its own, the logits are capped.  Tensor names are the
checkpoint's own (``l<i>.norm1``, ``l<i>.mix.dkv``, ``l<i>.mlp.e3.gate``, ...).
"""

from __future__ import annotations

from lily_b200.config.nafazen_config import NafazenConfig, NafazenDenseConfig
from lily_b200.config.registry import register_architecture
from lily_b200.parts.base import ModelSpec, ScheduleEntry
from lily_b200.parts.block import PostNormBlockSpec
from lily_b200.parts.experts import RoutedExpertsSpec
from lily_b200.parts.latent_attention import LatentAttentionSpec
from lily_b200.parts.mlp import DenseMLPSpec
from lily_b200.parts.norm import RMSNormSpec
from lily_b200.parts.rope import RopeSpec

_FF_NAMES = (("up", "up"), ("down", "down"), ("act", "act"))


def build_spec(cfg: NafazenConfig) -> ModelSpec:
    norm = RMSNormSpec(cfg.width, cfg.eps, suffix="", single_gain=True)
    blocks, ignored = [], []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        rope = RopeSpec(m.rot_dim, m.rotary_dims, m.rotary_base, m.rotary_scaling, interleaved=True, exact_frequencies=True) \
            if m.rotary_dims else None
        mixer = LatentAttentionSpec(cfg.width, m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, cfg.eps,
                                    position=rope, out_gate=False, own_kv=m.kv_from is None)
        if layer.mlp is None:
            ff = None
            ignored.append(f"l{i}.norm2")                   # a layer without feed-forward has no use for its norm
        elif isinstance(layer.mlp, NafazenDenseConfig):
            ff = DenseMLPSpec(cfg.width, layer.mlp.ff, activation="xielu", names=_FF_NAMES)
        else:
            e = layer.mlp
            ff = RoutedExpertsSpec(cfg.width, e.ff, e.experts, 0, e.top, scores="sigmoid", correction=False, renormalise=False,
                                   activation="silu", weight_on="input", shared_size=e.shared_ff)
        blocks.append(PostNormBlockSpec(prefix=f"l{i}", mixer=mixer, feed_forward=ff, norm=norm))
    schedule = [ScheduleEntry(i, reads=layer.mixer.kv_from) for i, layer in enumerate(cfg.layers)]
    return ModelSpec(architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=cfg.width, blocks=blocks,
                     schedule=schedule, final_norm=norm, embed_name="embed", final_norm_prefix="final.norm", head_name="head",
                     max_position=cfg.max_positions, ignored_tensors=tuple(ignored), embed_scale=cfg.embed_scale,
                     logit_softcap=cfg.logit_softcap)


register_architecture("Nafazen", NafazenConfig.from_dict, build_spec)
