"""A linear-attention mixer with a matrix memory and exponential gates (the mLSTM of the xLSTM family), with its state in the
request's slot.

One projection of the input gives ``[q | k | v | gate]`` and the two gates' inputs ``[i | f]``, one number a head each: q and k
with ``heads`` heads of ``head_dim`` (q times ``head_dim^-0.5``), v and the gate with heads of ``v_head_dim``.  Per head the log
gates are ``i = cap tanh((W_i h + b_i) / cap)`` and ``f = logsigmoid(cap tanh((W_f h + b_f) / cap))``; with S a ``head_dim x
v_head_dim`` matrix, n a vector and m a number, all zero when the request starts,

    m_t = max(f + m, i);    S <- exp(f + m - m_t) S + exp(i - m_t) k v^T;    n <- exp(f + m - m_t) n + exp(i - m_t) k
    o_t = S^T q / (max(|n . q|, exp(-m_t)) + floor)

then each head's o is divided by its root mean square, the heads are multiplied by a gain and by ``sigmoid(gate)``, and
projected out.

What a request carries from step to step is one float32 row of its slot (``StateNeed``): the heads' matrices with n as one more
column ``[heads, v_head_dim + 1, head_dim]``, then the heads' m.  The kernels reach it through ``batch.slots`` on the device, so a
step in which every request brings one token can be captured in a CUDA graph (``graph_safe``); a portion of a prompt
continues from the same row, whatever its length.  The gates' inputs leave their product in float32; gates, scale, state, the
sums over it and the unit norm by head are float32 in both precisions.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional, Tuple

import torch

from lily_b200.parts.base import BuildContext, Mixer, StateNeed, TensorSpec, register_part


@dataclass(frozen=True)
class MlstmSpec:
    hidden_size: int
    heads: int
    head_dim: int
    v_head_dim: int
    gate_cap: float
    norm_eps: float
    floor: float = 1e-6
    kind: str = "mlstm"
    # names of the tensors under the part's prefix
    names: Optional[Tuple[Tuple[str, str], ...]] = None

    _DEFAULTS = (("q", "q"), ("k", "k"), ("v", "v"), ("gate", "g"), ("i", "i"), ("f", "f"), ("i_bias", "i.b"), ("f_bias", "f.b"),
                 ("norm", "norm"), ("o", "o"))

    def name(self, role: str) -> str:
        return dict(self.names or ()).get(role, dict(self._DEFAULTS)[role])

    @property
    def key_columns(self) -> int:
        return self.heads * self.head_dim

    @property
    def inner(self) -> int:
        return self.heads * self.v_head_dim

    @property
    def projected(self) -> int:
        """Columns ahead of the gates' inputs."""
        return 2 * self.key_columns + 2 * self.inner


@register_part("mixer", "mlstm")
class Mlstm(Mixer):
    graph_safe = True

    def __init__(self, spec: MlstmSpec, prefix: str, ctx: BuildContext):
        if min(spec.heads, spec.head_dim, spec.v_head_dim) < 1 or not spec.gate_cap > 0:
            raise ValueError("heads, head sizes and the gates' cap are positive")
        self.spec, self.prefix, self.ctx = spec, prefix, ctx
        self.w_in = self.w_o = self.i_bias = self.f_bias = self.gain = None

    # ---- what it needs ----------------------------------------------------------

    @property
    def matrix_floats(self) -> int:
        s = self.spec
        return s.heads * (s.v_head_dim + 1) * s.head_dim

    def state_need(self) -> StateNeed:
        floats = self.matrix_floats + self.spec.heads
        return StateNeed((floats + -floats % 4,), torch.float32)              # whole 16-byte pieces a row

    def tensors(self) -> Dict[str, TensorSpec]:
        s, p = self.spec, self.prefix
        n = lambda role: f"{p}.{s.name(role)}"
        return {n("q"): TensorSpec((s.key_columns, s.hidden_size)), n("k"): TensorSpec((s.key_columns, s.hidden_size)),
                n("v"): TensorSpec((s.inner, s.hidden_size)), n("gate"): TensorSpec((s.inner, s.hidden_size)),
                n("i"): TensorSpec((s.heads, s.hidden_size)), n("f"): TensorSpec((s.heads, s.hidden_size)),
                n("i_bias"): TensorSpec((s.heads,), role="vector", init="normal"),
                n("f_bias"): TensorSpec((s.heads,), role="vector", init="normal"),
                n("norm"): TensorSpec((s.inner,), role="vector", init="gain"), n("o"): TensorSpec((s.hidden_size, s.inner))}

    def load(self, get) -> None:
        s, p = self.spec, self.prefix
        g = lambda role: get(f"{p}.{s.name(role)}")
        # one matrix for everything that reads the mixer's input, [q | k | v | gate | i | f | zero rows up to a multiple of 8]
        rows = [g(r) for r in ("q", "k", "v", "gate", "i", "f")]
        total = sum(r.shape[0] for r in rows)
        self.w_in = torch.cat(rows + [rows[0].new_zeros((-total % 8, s.hidden_size))]).contiguous()
        self.w_o = g("o").contiguous()
        self.i_bias, self.f_bias = g("i_bias").float().contiguous(), g("f_bias").float().contiguous()
        self.gain = g("norm").float().contiguous()

    # ---- one step ----------------------------------------------------------------

    def _project(self, x):
        """(rows that hold q, k, v and the output gate; rows that hold the gates' inputs in float32, and their first column)."""
        s, ops = self.spec, self.ctx.ops
        whole = ops.linear_split(x, self.w_in)
        if whole is None and (x.dtype == torch.float32 or x.shape[0] <= 64):
            whole = ops.linear(x, self.w_in, out_dtype=torch.float32)
        if whole is not None:
            return whole, whole, s.projected
        return ops.linear(x, self.w_in[:s.projected]), ops.linear(x, self.w_in[s.projected:], out_dtype=torch.float32), 0

    def forward(self, x, batch, cache, state, write_cache: bool = True):
        s, ops = self.spec, self.ctx.ops
        proj, gates, i_col = self._project(x)
        v_col = 2 * s.key_columns
        # long portions run as chunks side by side; the cut is planned once a step for the layers of one size
        plan = batch.plan(("mlstm_plan", s.heads, s.head_dim, s.v_head_dim), lambda b: ops.mlstm_plan(
            b.h_new_lens, x.dtype, s.heads, s.head_dim, s.v_head_dim, b.token_ids.device))
        need = ops.mlstm_workspace_floats(plan, s.heads, s.head_dim, s.v_head_dim)
        room = batch.workspace.floats("mlstm_chunks", need) if need and batch.workspace is not None else None
        y, nq, m = ops.mlstm_scan(proj, 0, s.key_columns, v_col, gates, i_col, i_col + s.heads, self.i_bias, self.f_bias, s.gate_cap,
                                  s.head_dim ** -0.5, state, batch.cu_seqlens, batch.slots, batch.num_requests, s.heads, s.head_dim,
                                  s.v_head_dim, plan=plan, workspace=room)
        out = ops.mlstm_out(y, nq, m, proj, v_col + s.inner, self.gain, s.floor, s.norm_eps, state, self.matrix_floats, batch.cu_seqlens,
                            batch.token_req, batch.slots, self.ctx.dtype)
        return ops.linear_auto(out, self.w_o)
