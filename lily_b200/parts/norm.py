"""Norms fused with the residual add: RMSNorm, and a norm that squashes instead of dividing (``DynamicTanh``).

``forward(residual, delta)`` adds ``delta`` into the float32 residual stream in place and
returns the normalised activations in the compute dtype: the fused-add convention of
lily/layers/layernorm.py:11-47 with the sum kept in float32.  With ``rows`` only those rows are
normalised (the final norm before the logits).

A norm may also stand behind a sublayer: ``behind(mult)`` gives what turns the sublayer's output into a pending delta
(``NormedDelta``, ``TanhDelta``) that the norm which comes next folds into the stream in its own pass.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict

from lily_b200.parts.base import BuildContext, Norm, TensorSpec, register_part


@dataclass
class NormedDelta:
    """A sublayer's output that enters the residual stream as ``mult * (rms(delta) * gain)``, its own root mean
    square (with ``eps``) taken over the row first (a norm behind the sublayer as well as ahead of it).  A block hands
    it on as its pending delta; the norm that follows folds it into the stream in the pass in which it normalises."""

    delta: Any                 # [tokens, size] in the compute dtype, or float32 partial sums [splits, tokens, size]
    gain: Any                  # float32 [size]
    eps: float
    mult: float = 1.0
    normalise: bool = True     # False: ``mult * (delta * gain)``, a gain per column without the division (a layer scale)


@dataclass
class TanhDelta:
    """A sublayer's output that enters the residual stream as ``mult * (gain * tanh(alpha * delta) + shift)``."""

    delta: Any                 # as in ``NormedDelta``
    alpha: float
    gain: Any                  # float32 [size]
    shift: Any                 # float32 [size]
    mult: float = 1.0

    @property
    def norm(self):
        return self.alpha, self.gain, self.shift


@dataclass(frozen=True)
class RMSNormSpec:
    size: int
    eps: float
    kind: str = "rmsnorm"
    suffix: str = ".weight"        # the gain's name is the part's prefix followed by this ("" where the prefix is the name)
    offset: float = 0.0            # the checkpoint stores the gain minus this (1.0: gains stored around zero); the sum
                                   # is formed once, in float32, when the gain is loaded
    single_gain: bool = False      # the checkpoint stores one number that serves all columns (shape [])


@register_part("norm", "rmsnorm")
class RMSNorm(Norm):
    def __init__(self, spec: RMSNormSpec, prefix: str, ctx: BuildContext):
        self.spec, self.prefix, self.ctx = spec, prefix, ctx
        self.weight = None

    def tensors(self) -> Dict[str, TensorSpec]:
        return {f"{self.prefix}{self.spec.suffix}": TensorSpec(() if self.spec.single_gain else (self.spec.size,), role="vector", init="gain")}

    def load(self, get) -> None:
        self.weight = get(f"{self.prefix}{self.spec.suffix}")
        if self.spec.offset:
            self.weight = (self.weight.float() + self.spec.offset).contiguous()
        if self.spec.single_gain:
            self.weight = self.weight.float().reshape(1).expand(self.spec.size).contiguous()      # the kernels read a gain a column

    def behind(self, mult: float = 1.0, divides: bool = True):
        """What a block wraps a sublayer's output in when this norm stands behind the sublayer (``divides`` False: its gain alone)."""
        gain = self.weight.float().contiguous()                  # it enters a float32 sum
        return lambda delta: NormedDelta(delta, gain, self.spec.eps, float(mult), divides)

    def forward(self, residual, delta=None, delta_bias=None, rows=None, write_residual=True, also=None, out_dtype=None):
        """``delta`` may be a tuple of tensors to be summed; ``delta_bias`` a float32 vector added to every row;
        ``also`` another norm of this kind and size whose output of the same rows is wanted too (returns a pair)."""
        if isinstance(delta, TanhDelta):
            self.ctx.ops.add_tanh_norm(residual, delta.delta, delta.norm, delta.mult, None, None)
            delta = None
        if isinstance(delta, NormedDelta):
            if delta_bias is not None or also is not None:
                raise ValueError("a normalised delta comes alone: no stream vector and no second norm in the same pass")
            return self.ctx.ops.add_normed_rmsnorm(residual, delta.delta, delta.gain, delta.eps, delta.mult, self.weight,
                                                   self.spec.eps, out_dtype or self.ctx.dtype, rows=rows,
                                                   write_residual=write_residual and rows is None,
                                                   **({} if delta.normalise else {"normalise": False}))
        deltas = [d for d in delta if d is not None] if isinstance(delta, (tuple, list)) else ([delta] if delta is not None else [])
        if delta_bias is None and also is None and len(deltas) <= 1:
            return self.ctx.ops.add_rmsnorm(residual, deltas[0] if deltas else None, self.weight, self.spec.eps,
                                            out_dtype or self.ctx.dtype, rows=rows, write_residual=write_residual)
        if rows is not None:
            # gathered rows: the sum goes into the stream first, then the plain form reads the rows
            self.ctx.ops.add_rmsnorm_multi(residual, deltas, [], self.spec.eps, self.ctx.dtype, bias=delta_bias)
            return self.ctx.ops.add_rmsnorm(residual, None, self.weight, self.spec.eps, out_dtype or self.ctx.dtype, rows=rows)
        if also is not None and (also.spec.eps != self.spec.eps or also.spec.size != self.spec.size):
            raise ValueError("two norms share a pass over the rows only with one size and one eps")
        gains = [self.weight.float()] + ([also.weight.float()] if also is not None else [])
        outs = self.ctx.ops.add_rmsnorm_multi(residual, deltas, gains, self.spec.eps, out_dtype or self.ctx.dtype,
                                              bias=delta_bias, write_residual=write_residual)
        return outs if also is not None else outs[0]


@dataclass(frozen=True)
class DynamicTanhSpec:
    """``gain * tanh(alpha * x) + shift``: a scalar ``alpha``, a gain and a shift a column; no mean and no variance."""

    size: int
    kind: str = "dynamic_tanh"
    suffix: str = ""               # the gain's, the scalar's and the shift's names are the part's prefix followed by these
    alpha_suffix: str = ".alpha"
    shift_suffix: str = ".b"


@register_part("norm", "dynamic_tanh")
class DynamicTanh(Norm):
    def __init__(self, spec: DynamicTanhSpec, prefix: str, ctx: BuildContext):
        self.spec, self.prefix, self.ctx = spec, prefix, ctx
        self.alpha = 0.0
        self.weight = self.shift = None

    def tensors(self) -> Dict[str, TensorSpec]:
        s, p = self.spec, self.prefix
        return {f"{p}{s.suffix}": TensorSpec((s.size,), role="vector", init="gain"),
                f"{p}{s.alpha_suffix}": TensorSpec((), role="vector", init="half"),
                f"{p}{s.shift_suffix}": TensorSpec((s.size,), role="vector", init="zeros")}

    def load(self, get) -> None:
        s, p = self.spec, self.prefix
        # every column enters float32 arithmetic; the scalar travels as a kernel argument
        self.alpha = float(get(f"{p}{s.alpha_suffix}").float().item())
        self.weight = get(f"{p}{s.suffix}").float().contiguous()
        self.shift = get(f"{p}{s.shift_suffix}").float().contiguous()

    @property
    def norm(self):
        return self.alpha, self.weight, self.shift

    def behind(self, mult: float = 1.0, divides: bool = True):
        if not divides:
            raise ValueError("a norm that squashes has no form with the gain alone")
        return lambda delta: TanhDelta(delta, self.alpha, self.weight, self.shift, float(mult))

    def forward(self, residual, delta=None, delta_bias=None, rows=None, write_residual=True, also=None, out_dtype=None):
        ops, dtype = self.ctx.ops, out_dtype or self.ctx.dtype
        if also is not None:
            raise ValueError("this norm shares no pass with another norm of the same rows")
        post, mult = None, 1.0
        if isinstance(delta, TanhDelta):
            post, mult, delta = delta.norm, delta.mult, delta.delta
        elif isinstance(delta, NormedDelta):
            ops.add_normed(residual, delta.delta, delta.gain, delta.eps, delta.mult, residual.dtype,
                           **({} if delta.normalise else {"normalise": False}))
            delta = None
        elif isinstance(delta, (tuple, list)):
            deltas = [d for d in delta if d is not None]
            delta = deltas[0] if deltas else None
            if len(deltas) > 1:
                ops.add_rmsnorm_multi(residual, deltas, [], 1.0, dtype)
                delta = None
        if delta_bias is not None:
            ops.add_rmsnorm_multi(residual, [], [], 1.0, dtype, bias=delta_bias)
        return ops.add_tanh_norm(residual, delta, post, mult, self.norm, dtype, rows=rows, write_residual=write_residual and rows is None)


def enter_stream(ops, residual, delta, dtype, bias=None):
    """Adds a pending ``delta`` (a tensor, several of them, a ``NormedDelta`` or None) and ``bias`` (a row vector) into the
    float32 stream in place and returns the new stream itself in ``dtype``: what a sublayer takes that has no norm ahead
    of it.  With ``dtype`` float32 that is ``residual``, which the next call changes."""
    if isinstance(delta, (NormedDelta, TanhDelta)) and bias is not None:
        raise ValueError("a normalised delta comes alone: no stream vector in the same pass")
    if isinstance(delta, TanhDelta):
        out = ops.add_tanh_norm(residual, delta.delta, delta.norm, delta.mult, None, None if dtype == residual.dtype else dtype)
        return residual if out is None else out
    if isinstance(delta, NormedDelta):
        return ops.add_normed(residual, delta.delta, delta.gain, delta.eps, delta.mult, dtype,
                              **({} if delta.normalise else {"normalise": False}))
    deltas = [d for d in delta if d is not None] if isinstance(delta, (tuple, list)) else ([delta] if delta is not None else [])
    if deltas or bias is not None:
        ops.add_rmsnorm_multi(residual, deltas, [], 1.0, dtype, bias=bias)
    return ops.cast(residual, dtype)
