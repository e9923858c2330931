"""Softmax attention over a low-rank latent of keys and values, with the latent alone in the paged cache.

Queries go through a latent of their own: ``c_q = rms(W_dq h) * g_q``, ``q = W_uq c_q``, head by head
``[head_dim unrotated | rot_dim rotated]``; or, with ``q_rank`` 0, ``q = W_q h``.  ``W_dkv h`` gives ``kv_rank + rot_dim`` numbers: the first ``kv_rank``,
RMS-normed with a gain, are the latent ``c``; the rest, rotated by position, are one key part shared by all heads.
Per head the unrotated key is ``W_uk c`` and the value ``W_uv c``; the score is
``(q_unrotated . k_unrotated + q_rotated . k_rotated) * scale`` over the visible positions (all, or the last
``window``); with ``sink`` the softmax's denominator also holds ``exp(sink_h)``, a learned number a head that has no key and no
value and is not scaled; each head's output is multiplied by ``sigmoid(W_g h)`` of that head (``out_gate``), and ``W_o`` closes the part.

Only ``[c | rotated key part]`` is cached: one row of ``kv_rank + rot_dim`` numbers per position for all heads
(``CacheNeed`` with one kv head and ``values_in_keys``).  Since ``q_u . (W_uk c) = (W_uk^T q_u) . c``, the unrotated
query part of each head is carried into the latent's space once per token (a product per head), the attention kernel
then runs over the cached rows as they are, all heads sharing them, with the first ``kv_rank`` columns of a row as its
values, and ``W_uv`` is applied to each head's weighted sum of latents afterwards (``W_uv sum_j p_j c_j``).  A prompt's
portion and a decoded token take the same path, so what a position's logits are does not depend on how it arrived.

With ``own_kv`` False the mixer has no ``W_dkv``: it attends to rows that another run's mixer has cached (a schedule entry
that ``reads`` that run), with its own queries, ``W_uk`` and ``W_uv``.  The two then agree in ``kv_rank``, ``rot_dim`` and
position encoding.  An interleaved position encoding is served by reordering the rotated rows of ``W_uq`` and ``W_dkv`` once,
at load time (a score does not change when the columns of query and key are reordered alike).

The three projections that read the mixer's input (query latent, key/value latent, gate) are one product with a
float32 result (partial sums for a few tokens); the two RMS norms, the rotation angles, the scores and the softmax are
float32 in both precisions.  The two products per head write into the rows the next kernel reads, rounded once.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

import torch

from lily_b200.parts.attention import AttentionPlan, LayerCache
from lily_b200.parts.base import BuildContext, CacheNeed, Mixer, TensorSpec, build_part, register_part
from lily_b200.parts.rope import pairing_order


@dataclass(frozen=True)
class LatentAttentionSpec:
    hidden_size: int
    num_heads: int
    head_dim: int                 # unrotated query/key columns a head
    rot_dim: int                  # rotated query/key columns a head (the key's are shared by all heads)
    v_head_dim: int
    q_rank: int                   # 0: the queries are projected from the mixer's input
    kv_rank: int
    scale: float
    norm_eps: float
    window: Optional[int] = None  # None: all keys; n: the last n keys
    position: Any = None          # a position spec over the rot_dim columns (e.g. RopeSpec) or None
    out_gate: bool = True         # each head's output times sigmoid(W_g h) of the head
    sink: bool = False            # a learned number a head in the softmax's denominator
    own_kv: bool = True           # False: the cached rows are another run's; this mixer projects none
    kind: str = "latent_attention"
    # names of the tensors under the part's prefix
    names: Optional[Tuple[Tuple[str, str], ...]] = None

    _DEFAULTS = (("dq", "dq"), ("dq_norm", "dq.norm"), ("uq", "uq"), ("dkv", "dkv"), ("dkv_norm", "dkv.norm"),
                 ("uk", "uk"), ("uv", "uv"), ("g", "g"), ("o", "o"), ("q", "q"), ("sink", "sink"))

    def name(self, role: str) -> str:
        return dict(self.names or ()).get(role, dict(self._DEFAULTS)[role])

    @property
    def row(self) -> int:
        """Numbers cached for one position."""
        return self.kv_rank + self.rot_dim


@register_part("mixer", "latent_attention")
class LatentAttention(Mixer):
    graph_safe = True

    def __init__(self, spec: LatentAttentionSpec, prefix: str, ctx: BuildContext):
        if min(spec.num_heads, spec.head_dim, spec.v_head_dim, spec.kv_rank) < 1 or min(spec.rot_dim, spec.q_rank) < 0:
            raise ValueError("sizes of the latent attention are positive")
        self.spec, self.prefix, self.ctx = spec, prefix, ctx
        self.position = build_part("position", spec.position, prefix, ctx) if spec.position is not None else None
        if self.position is not None and self.position.rotary_dim > spec.rot_dim:
            raise ValueError(f"{self.position.rotary_dim} rotated columns do not fit the {spec.rot_dim} set aside for them")
        self.sinks = None
        self.w_down = self.w_uq = self.w_uk = self.w_uv = self.w_o = self.q_gain = self.kv_gain = None

    # ---- what it needs ----------------------------------------------------------

    def cache_need(self) -> CacheNeed:
        s = self.spec
        return CacheNeed(1, s.row, s.window, s.kv_rank, values_in_keys=True)

    def tensors(self) -> Dict[str, TensorSpec]:
        s, p = self.spec, self.prefix
        h = s.num_heads
        q = h * (s.head_dim + s.rot_dim)
        if s.q_rank:
            out = {f"{p}.{s.name('dq')}": TensorSpec((s.q_rank, s.hidden_size)),
                   f"{p}.{s.name('dq_norm')}": TensorSpec((s.q_rank,), role="vector", init="gain"),
                   f"{p}.{s.name('uq')}": TensorSpec((q, s.q_rank))}
        else:
            out = {f"{p}.{s.name('q')}": TensorSpec((q, s.hidden_size))}
        out = {**out,
               f"{p}.{s.name('uk')}": TensorSpec((h * s.head_dim, s.kv_rank)),
               f"{p}.{s.name('uv')}": TensorSpec((h * s.v_head_dim, s.kv_rank)),
               f"{p}.{s.name('o')}": TensorSpec((s.hidden_size, h * s.v_head_dim))}
        if s.own_kv:
            out[f"{p}.{s.name('dkv')}"] = TensorSpec((s.row, s.hidden_size))
            out[f"{p}.{s.name('dkv_norm')}"] = TensorSpec((s.kv_rank,), role="vector", init="gain")
        if s.out_gate:
            out[f"{p}.{s.name('g')}"] = TensorSpec((h, s.hidden_size))
        if s.sink:
            out[f"{p}.{s.name('sink')}"] = TensorSpec((h,), role="vector", init="normal")
        return out

    def _rotation_order(self) -> Optional[torch.Tensor]:
        """For an interleaved encoding: the stored row of the rotated part that goes to each place of it."""
        if self.position is None or not self.position.interleaved:
            return None
        return pairing_order(self.spec.rot_dim, self.position.rotary_dim)

    def load(self, get) -> None:
        s, p = self.spec, self.prefix
        g = lambda role: get(f"{p}.{s.name(role)}")
        h, order = s.num_heads, self._rotation_order()
        parts = [g("dq")] if s.q_rank else []
        if s.own_kv:
            dkv = g("dkv")
            if order is not None:
                dkv = torch.cat([dkv[:s.kv_rank], dkv[s.kv_rank:][order.to(dkv.device)]], 0)
            parts.append(dkv)
        if s.out_gate:
            parts.append(g("g"))
        self.w_down = torch.cat(parts, 0).contiguous() if parts else None      # [q_rank (| kv_rank + rot) (| heads)] rows
        self.q_gain = g("dq_norm").float().contiguous() if s.q_rank else None
        # a mixer that caches nothing has no gain of its own there and reads none
        self.kv_gain = g("dkv_norm").float().contiguous() if s.own_kv else torch.ones(s.kv_rank, dtype=torch.float32, device=self.ctx.device)
        self.sinks = g("sink").float().contiguous() if s.sink else None
        uq = g("uq" if s.q_rank else "q")
        if order is not None:
            width = uq.shape[1]
            uq = uq.view(h, s.head_dim + s.rot_dim, width)
            uq = torch.cat([uq[:, :s.head_dim], uq[:, s.head_dim:][:, order.to(uq.device)]], 1).reshape(-1, width)
        self.w_uq = uq.contiguous()
        # per head [out, in]: q' = W_uk^T q_u takes W_uk^T [kv_rank, head_dim]; the value takes W_uv [v, kv_rank] as stored
        self.w_uk = g("uk").view(h, s.head_dim, s.kv_rank).transpose(1, 2).contiguous()
        self.w_uv = g("uv").view(h, s.v_head_dim, s.kv_rank).contiguous()
        self.w_o = g("o").contiguous()

    # ---- one step ----------------------------------------------------------------

    def _plan(self, batch, group: int, dtype, page: int):
        """How this step's attention runs for these sizes in cache group ``group`` (made once a step, shared by the
        layers of one size): the heads are the query heads of one kv head."""
        s, ops = self.spec, self.ctx.ops
        key = ("latent_attention", group, s.num_heads, s.row, s.kv_rank, dtype, page)

        def make(b):
            nd = b.num_decode
            decode = ops.plan_decode_attention(dtype, nd, s.num_heads, 1, s.row, b.max_decode_len, even=b.decode_even,
                                               dv=s.kv_rank, values_in_keys=True, page_size=page)
            rows = tiles = None
            if b.num_requests > nd:
                rows = ops.prefill_tile_rows(dtype, s.row, page, b.num_tokens - nd, dv=s.kv_rank, values_in_keys=True,
                                             heads=s.num_heads)
                tiles = ops.prefill_tiles(b.h_prefix_lens, b.h_new_lens, nd, rows, b.token_ids.device)
            return AttentionPlan(decode, rows, tiles)
        return batch.plan(key, make)

    def forward(self, x, batch, cache: LayerCache, state=None, write_cache: bool = True):
        s, ops = self.spec, self.ctx.ops
        page, h = self.ctx.page_size, s.num_heads
        table = batch.block_tables[cache.group]
        plan = self._plan(batch, cache.group, cache.data.dtype, page)
        cos, sin = self.position.tables() if self.position is not None else (None, None)
        rotary_dim = self.position.rotary_dim if self.position is not None else 0
        down = None
        if self.w_down is not None:
            down = ops.linear_split(x, self.w_down)             # [tokens, q latent (| kv latent | rotated) (| gates)], float32
            if down is None:
                down = ops.linear(x, self.w_down, out_dtype=torch.float32)
        write_cache = write_cache and s.own_kv
        cq = None
        if s.q_rank or write_cache:
            cq = ops.latent_prepare(down, 0, s.q_rank, s.q_rank, s.kv_rank, s.rot_dim, rotary_dim, self.q_gain, self.kv_gain,
                                    s.norm_eps, cos, sin, batch.positions, batch.token_req, table, cache.data, page,
                                    write_kv=write_cache)
        q = ops.linear(cq if s.q_rank else x, self.w_uq)                 # [tokens, heads * (head_dim + rot)]
        sunk = {"sinks": self.sinks} if s.sink else {}
        tokens = q.shape[0]
        queries = torch.empty((tokens, h * s.row), dtype=q.dtype, device=q.device)
        ops.head_linear(q.view(tokens, h, s.head_dim + s.rot_dim)[:, :, :s.head_dim], self.w_uk,
                        out=queries.view(tokens, h, s.row)[:, :, :s.kv_rank])
        ops.latent_query(queries, q, h, s.head_dim, s.kv_rank, s.rot_dim, rotary_dim, cos, sin, batch.positions)
        mixed = torch.empty((tokens, h * s.kv_rank), dtype=q.dtype, device=q.device)
        nd, dec = batch.num_decode, plan.decode
        if nd:
            scratch = batch.workspace.floats("attention_decode", dec.scratch_floats) if dec.scratch_floats else None
            ops.attention_decode(queries[:nd], cache.data, table, batch.seq_lens, mixed[:nd], scratch, dec.splits, h, 1,
                                 s.row, page, s.scale, s.window, dv=s.kv_rank, values_in_keys=True, **sunk)
        if batch.num_requests > nd:
            tile_req, tile_start = plan.tiles
            ops.attention_prefill(queries, cache.data, table, batch.cu_seqlens, batch.prefix_lens, tile_req, tile_start,
                                  mixed, h, 1, s.row, page, s.scale, s.window, tile_rows=plan.tile_rows, dv=s.kv_rank,
                                  values_in_keys=True, **sunk)
        mixed = mixed.view(tokens, h, s.kv_rank)
        if s.out_gate:
            values = ops.head_linear(mixed, self.w_uv, out_dtype=torch.float32)                         # [heads, tokens, v]
            out = ops.head_gate(values, down, s.q_rank + (s.row if s.own_kv else 0), q.dtype)
        else:
            out = torch.empty((tokens, h * s.v_head_dim), dtype=q.dtype, device=q.device)
            ops.head_linear(mixed, self.w_uv, out=out.view(tokens, h, s.v_head_dim))
        return ops.linear_auto(out, self.w_o)
