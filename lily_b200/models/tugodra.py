"""The Tugodra decoder as a ``ModelSpec``.

Every layer is a sandwich block, ``x += norm1b(mixer(norm1(x)))`` and, where it has a feed-forward, ``x += norm2b(ff(norm2(x)))``,
whose norms take no mean and no variance (``dynamic_tanh``).  The mixer is a windowed grouped-query attention with interleaved
rotation, unit q and k heads and one output gate a head (a layer with ``kv_from`` is a run of the schedule that ``reads``
another run's keys and values), a softmax attention over a cached low-rank latent with a sink a head, or a matrix memory with
exponential gates.  The feed-forward is a routed mixture of ungated squared-ReLU experts with sigmoid scores, a correction of
the choice, a choice within the best groups, renormalised weights and a gated shared expert.  The embedding is scaled, the head is a table of its own.
Tensor names are the checkpoint's own (``l<i>.norm1``, ``l<i>.mix.dkv``, ``l<i>.mlp.e3.up``, ...).
"""

from __future__ import annotations

from lily_b200.config.registry import register_architecture
from lily_b200.config.tugodra_config import TugodraConfig
from lily_b200.parts.attention import AttentionSpec
from lily_b200.parts.base import ModelSpec, ScheduleEntry
from lily_b200.parts.block import SandwichBlockSpec
from lily_b200.parts.experts import RoutedExpertsSpec
from lily_b200.parts.latent_attention import LatentAttentionSpec
from lily_b200.parts.mlstm import MlstmSpec
from lily_b200.parts.norm import DynamicTanhSpec
from lily_b200.parts.rope import RopeSpec

_ATTENTION_NAMES = tuple((r, r) for r in ("q", "k", "v", "o", "g"))


def _mixer(cfg: TugodraConfig, layer):
    m = layer.mixer
    if layer.type == "mlstm":
        return MlstmSpec(cfg.width, m.heads, m.dim, m.vdim, m.gate_cap, cfg.eps)
    latent = layer.type == "latent_attention"
    rope = RopeSpec(m.rot_dim if latent else m.dim, m.rotary_dims, m.rotary_base, interleaved=not latent, exact_frequencies=True) \
        if m.rotary_dims else None
    if latent:
        return LatentAttentionSpec(cfg.width, m.heads, m.dim, m.rot_dim, m.vdim, 0, m.kv_rank, m.scale, cfg.eps, position=rope,
                                   out_gate=False, sink=True)
    return AttentionSpec(cfg.width, m.heads, m.kv_heads, m.dim, qk_norm=True, qk_gain=False, norm_eps=cfg.eps, window=m.window,
                         scale=m.scale, position=rope, v_head_dim=m.vdim, head_gate=True, own_kv=m.kv_from is None, names=_ATTENTION_NAMES)


def build_spec(cfg: TugodraConfig) -> ModelSpec:
    norm = DynamicTanhSpec(cfg.width)
    blocks, ignored = [], []
    for i, layer in enumerate(cfg.layers):
        e, ff = layer.mlp, None
        if e is None:
            ignored.append(f"l{i}.norm2")                   # a layer without feed-forward has no use for its norms
        else:
            ff = RoutedExpertsSpec(cfg.width, e.ff, e.experts, 0, e.top, scores="sigmoid", activation="relu2", shared_size=e.shared_ff,
                                   groups=e.groups, keep_groups=e.keep_groups)
        blocks.append(SandwichBlockSpec(prefix=f"l{i}", mixer=_mixer(cfg, layer), feed_forward=ff, norm=norm))
    return ModelSpec(architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=cfg.width, blocks=blocks,
                     schedule=[ScheduleEntry(i, reads=layer.kv_from) for i, layer in enumerate(cfg.layers)], final_norm=norm,
                     embed_name="embed", final_norm_prefix="final.norm", head_name="head", max_position=cfg.max_positions,
                     ignored_tensors=tuple(ignored), embed_scale=cfg.embed_scale)


register_architecture("Tugodra", TugodraConfig.from_dict, build_spec)
