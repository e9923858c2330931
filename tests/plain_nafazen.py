"""Plain, slow implementation of the Nafazen decoder, for tests only.

Whole sequences, no cache, one function per mechanism, float32 on the CPU unless
``precision(torch.float64)`` is in force.  It reads the raw ``config.json`` dictionary and the
checkpoint's own tensor names and shares no code with ``lily_b200``.

The design in this file's notation.  The stream starts as ``x = s E[token]``.  A layer is
``x <- x + n1(mixer(x))`` and then ``x <- x + n2(ff(x))``: nothing is normalised ahead of a sublayer, and what comes out of
one is, with ``n(y) = g y / sqrt(mean(y^2) + eps)`` and one number ``g`` a norm.  The mixer is a softmax attention over a
low-rank latent of keys and values; some layers have no latent of their own and read another layer's.  The feed-forward
is ``down(xielu(up x))`` or a routed mixture of gated experts with a shared expert beside them.  The logits are
``cap tanh(W n(x) / cap)``.
"""

from __future__ import annotations

import math
from typing import Dict, Optional, Tuple

import torch

Tensor = torch.Tensor

_COMPUTE = [torch.float32]


class precision:
    def __init__(self, dtype):
        self.dtype = dtype

    def __enter__(self):
        _COMPUTE.append(self.dtype)

    def __exit__(self, *exc):
        _COMPUTE.pop()


def _c(t: Tensor) -> Tensor:
    return t.to(_COMPUTE[-1])


def unit_rms(x: Tensor, eps: float) -> Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def single_gain_norm(y: Tensor, g: Tensor, eps: float) -> Tensor:
    """The model's norm: one gain for all columns."""
    return unit_rms(y, eps) * _c(g)


def silu(z: Tensor) -> Tensor:
    return z * torch.sigmoid(z)


# --------------------------------------------------------------------------- rotation

def frequencies(rot: dict) -> Tuple[Tensor, float]:
    """The pairs' frequencies (float32) and the factor of both tables."""
    dims, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(f, dtype=torch.float64).float(), 1.0
    turn = lambda t: dims * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(turn(sc["fast"])), 0)
    hi = min(math.ceil(turn(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64).float(), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_pairs(x: Tensor, positions: Tensor, rot: dict) -> Tensor:
    """x [t, ..., n]: columns 2i and 2i + 1 of the first ``dims`` form a pair that is turned by position * f_i; the rest passes."""
    dims = rot["dims"]
    f, stretch = frequencies(rot)
    ang = positions.to(torch.float32)[:, None] * f[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    cos, sin = (_c(ang.cos()) * stretch).view(shape), (_c(ang.sin()) * stretch).view(shape)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * cos - v * sin, v * cos + u * sin], -1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], -1)


# --------------------------------------------------------------------------- latent attention

def latent_rows(h: Tensor, w: Dict[str, Tensor], p: str, c: dict, eps: float, positions: Tensor) -> Tuple[Tensor, Tensor]:
    """What a layer keeps of each position: the normed latent and the rotated key part shared by all heads."""
    rank = c["kv_rank"]
    down = h @ _c(w[f"{p}.dkv"]).t()
    return unit_rms(down[:, :rank], eps) * _c(w[f"{p}.dkv.norm"]), rotate_pairs(down[:, rank:], positions, c["rot"])


def causal_softmax(scores: Tensor) -> Tensor:
    t = scores.shape[0]
    seen = torch.ones(t, t, dtype=torch.bool).tril()
    return torch.softmax(scores.masked_fill(~seen, float("-inf")), -1)


def latent_attention_mixer(h: Tensor, w: Dict[str, Tensor], p: str, c: dict, eps: float, positions: Tensor,
                           rows: Optional[Tuple[Tensor, Tensor]] = None) -> Tuple[Tensor, Tuple[Tensor, Tensor]]:
    """The mixer's output and the rows it attended to (its own, or those it was given)."""
    t = h.shape[0]
    heads, d, dr, dv = c["heads"], c["dim"], c["rot_dim"], c["vdim"]
    cq = unit_rms(h @ _c(w[f"{p}.dq"]).t(), eps) * _c(w[f"{p}.dq.norm"])
    q = (cq @ _c(w[f"{p}.uq"]).t()).view(t, heads, d + dr)
    q_plain, q_rot = q[..., :d], rotate_pairs(q[..., d:], positions, c["rot"])
    latent, k_rot = latent_rows(h, w, p, c, eps, positions) if rows is None else rows
    k_plain = (latent @ _c(w[f"{p}.uk"]).t()).view(t, heads, d)
    v = (latent @ _c(w[f"{p}.uv"]).t()).view(t, heads, dv)
    out = [causal_softmax((q_plain[:, n] @ k_plain[:, n].t() + q_rot[:, n] @ k_rot.t()) * float(c["scale"])) @ v[:, n]
           for n in range(heads)]
    return torch.cat(out, -1) @ _c(w[f"{p}.o"]).t(), (latent, k_rot)


# --------------------------------------------------------------------------- feed-forward

def xielu(z: Tensor, pq: Tensor) -> Tensor:
    a, b = torch.nn.functional.softplus(_c(pq)[0]), torch.nn.functional.softplus(_c(pq)[1])
    neg = torch.clamp(z, max=0.0)
    return torch.where(z > 0, a * z * z + 0.5 * z, (0.5 + b) * (torch.expm1(neg) - neg) + 0.5 * z)


def dense_ff(h: Tensor, w: Dict[str, Tensor], p: str) -> Tensor:
    return xielu(h @ _c(w[f"{p}.up"]).t(), w[f"{p}.act"]) @ _c(w[f"{p}.down"]).t()


def gated_expert(h: Tensor, w: Dict[str, Tensor], p: str) -> Tensor:
    return (silu(h @ _c(w[f"{p}.gate"]).t()) * (h @ _c(w[f"{p}.up"]).t())) @ _c(w[f"{p}.down"]).t()


def route(h: Tensor, w: Dict[str, Tensor], p: str, top: int) -> Tuple[Tensor, Tensor]:
    """(chosen experts [t, top], their weights [t, top]): the largest sigmoid scores, taken as they are."""
    s = torch.sigmoid(h.float() @ w[f"{p}.router"].float().t())
    best = torch.topk(s, top, dim=-1)
    return best.indices, best.values


def moe_ff(h: Tensor, w: Dict[str, Tensor], p: str, c: dict) -> Tensor:
    chosen, weights = route(h, w, p, c["router"]["top"])
    out = torch.zeros_like(h)
    for n in range(h.shape[0]):
        for e, a in zip(chosen[n].tolist(), weights[n].tolist()):
            out[n] += gated_expert(a * h[n:n + 1], w, f"{p}.e{e}")[0]            # the weight goes in, not on what comes out
    if c.get("shared"):
        out = out + gated_expert(h, w, f"{p}.shared") * torch.sigmoid(h @ _c(w[f"{p}.shared.sg"]).t())
    return out


# --------------------------------------------------------------------------- the model

def forward(cfg: dict, w: Dict[str, Tensor], tokens, return_layers: bool = False):
    """Logits [t, vocab] of one sequence (and, on request, the stream after every layer)."""
    eps = float(cfg["norm"]["eps"])
    ids = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(len(ids))
    x = _c(w["embed"])[ids] * float(cfg["embedding"]["scale"])
    kept, seen = {}, []
    for i, ly in enumerate(cfg["layers"]):
        p, c = f"l{i}", ly["mixer"]
        src = c.get("kv_from")
        y, kept[i] = latent_attention_mixer(x, w, f"{p}.mix", c, eps, positions, None if src is None else kept[src])
        x = x + single_gain_norm(y, w[f"{p}.norm1"], eps)
        mlp = ly.get("mlp")
        if mlp is not None:
            y = dense_ff(x, w, f"{p}.mlp") if mlp["kind"] == "dense" else moe_ff(x, w, f"{p}.mlp", mlp)
            x = x + single_gain_norm(y, w[f"{p}.norm2"], eps)
        seen.append(x)
    logits = single_gain_norm(x, w["final.norm"], eps) @ _c(w["head"]).t()
    cap = cfg.get("logit_softcap")
    if cap:
        logits = cap * torch.tanh(logits / cap)
    return (logits, torch.stack(seen)) if return_layers else logits
