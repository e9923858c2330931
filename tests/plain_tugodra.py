"""Plain, slow implementation of the Tugodra decoder, for tests only.

Whole sequences, no cache, one function per mechanism, float32 on the CPU unless
``precision(torch.float64)`` is in force.  It reads the raw ``config.json`` dictionary and the
checkpoint's own tensor names and shares no code with ``lily_b200``.

The design in this file's notation.  The stream starts as ``x = s E[token]``; a layer is

    x <- x + D_1b(mixer(D_1(x)))        x <- x + D_2b(ff(D_2(x)))        D(y) = w tanh(a y) + b

with ``a`` one number a norm and ``w``, ``b`` vectors (the second line only where the layer has a feed-forward).  The
mixer is one of

* ``attention``: grouped-query attention over the last ``size`` positions, interleaved rotation, then unit root mean
  square of each query and key head, each head's output times a sigmoid of its own; some layers attend to the keys and
  values that another layer has made;
* ``latent_attention``: softmax attention over a low-rank latent of keys and values, every key visible, with one learned
  number per head in the softmax's denominator;
* ``mlstm``: a matrix and a vector per head with exponential input gates and a running maximum as their scale.

The feed-forward is a routed mixture of ``down(max(up x, 0)^2)`` experts, chosen within the best groups of experts, and a
shared expert of the same form times a sigmoid of the token.  The logits are ``W D(x)``.
"""

from __future__ import annotations

from typing import Dict, Optional, Tuple

import torch
import torch.nn.functional as F

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


def squash(y: Tensor, w: Dict[str, Tensor], name: str) -> Tensor:
    """The model's norm: no mean, no variance, a tanh."""
    return torch.tanh(y * _c(w[f"{name}.alpha"]).reshape(())) * _c(w[name]) + _c(w[f"{name}.b"])


# --------------------------------------------------------------------------- rotation

def turn(u: Tensor, v: Tensor, positions: Tensor, rot: dict) -> Tuple[Tensor, Tensor]:
    """The pairs (u_i, v_i), i the last axis, turned by position * base^(-2 i / dims)."""
    dims = rot["dims"]
    f = torch.tensor([float(rot["base"]) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64).float()
    ang = positions.to(torch.float32)[:, None] * f[None, :]
    shape = [u.shape[0]] + [1] * (u.dim() - 2) + [dims // 2]
    cos, sin = _c(ang.cos()).view(shape), _c(ang.sin()).view(shape)
    return u * cos - v * sin, v * cos + u * sin


def rotate_neighbours(x: Tensor, positions: Tensor, rot: dict) -> Tensor:
    """Columns 2i and 2i + 1 of the first ``dims`` are a pair."""
    dims = rot["dims"]
    a, b = turn(x[..., 0:dims:2], x[..., 1:dims:2], positions, rot)
    return torch.cat([torch.stack([a, b], -1).flatten(-2), x[..., dims:]], -1)


def rotate_halves(x: Tensor, positions: Tensor, rot: dict) -> Tensor:
    """Columns i and i + dims / 2 of the first ``dims`` are a pair."""
    dims = rot["dims"]
    a, b = turn(x[..., :dims // 2], x[..., dims // 2:dims], positions, rot)
    return torch.cat([a, b, x[..., dims:]], -1)


# --------------------------------------------------------------------------- windowed attention

def window_mask(t: int, size: Optional[int]) -> Tensor:
    """seen[i, j]: key j is visible to query i."""
    back = torch.arange(t)[:, None] - torch.arange(t)[None, :]
    return (back >= 0) & (back < size if size else True)


def attention_keys_values(h: Tensor, w: Dict[str, Tensor], p: str, c: dict, eps: float, positions: Tensor) -> Tuple[Tensor, Tensor]:
    """What a layer keeps of each position: rotated unit keys [t, kv heads, dim] and values [t, kv heads, vdim]."""
    t, g = h.shape[0], c["kv_heads"]
    k = (h @ _c(w[f"{p}.k"]).t()).view(t, g, c["dim"])
    v = (h @ _c(w[f"{p}.v"]).t()).view(t, g, c["vdim"])
    return unit_rms(rotate_neighbours(k, positions, c["rot"]), eps), v


def attention_mixer(h: Tensor, w: Dict[str, Tensor], p: str, c: dict, eps: float, positions: Tensor,
                    kept: Optional[Tuple[Tensor, Tensor]] = None) -> Tuple[Tensor, Tuple[Tensor, Tensor]]:
    """The mixer's output and the keys and values it attended to (its own, or those it was given)."""
    t, heads = h.shape[0], c["heads"]
    q = unit_rms(rotate_neighbours((h @ _c(w[f"{p}.q"]).t()).view(t, heads, c["dim"]), positions, c["rot"]), eps)
    k, v = attention_keys_values(h, w, p, c, eps, positions) if kept is None else kept
    gate = torch.sigmoid(h @ _c(w[f"{p}.g"]).t())
    seen = window_mask(t, (c.get("mask") or {}).get("size"))
    share = heads // c["kv_heads"]
    out = []
    for n in range(heads):
        s = (q[:, n] @ k[:, n // share].t()) * float(c["scale"])
        out.append((torch.softmax(s.masked_fill(~seen, float("-inf")), -1) @ v[:, n // share]) * gate[:, n:n + 1])
    return torch.cat(out, -1) @ _c(w[f"{p}.o"]).t(), (k, v)


# --------------------------------------------------------------------------- latent attention with a sink

def softmax_with_sink(scores: Tensor, sink: Tensor) -> Tensor:
    """exp(s_j) / (exp(sink) + sum_j exp(s_j)): one more column that has no value."""
    full = torch.cat([scores, sink.reshape(1, 1).expand(scores.shape[0], 1).to(scores.dtype)], -1)
    return torch.softmax(full, -1)[:, :-1]


def latent_attention_mixer(h: Tensor, w: Dict[str, Tensor], p: str, c: dict, eps: float, positions: Tensor) -> Tensor:
    t, heads, d, dr, dv, rank = h.shape[0], c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    q = (h @ _c(w[f"{p}.q"]).t()).view(t, heads, d + dr)
    q_plain, q_rot = q[..., :d], rotate_halves(q[..., d:], positions, c["rot"])
    down = h @ _c(w[f"{p}.dkv"]).t()
    latent = unit_rms(down[:, :rank], eps) * _c(w[f"{p}.dkv.norm"])
    k_rot = rotate_halves(down[:, rank:], positions, c["rot"])
    k_plain = (latent @ _c(w[f"{p}.uk"]).t()).view(t, heads, d)
    v = (latent @ _c(w[f"{p}.uv"]).t()).view(t, heads, dv)
    seen = window_mask(t, None)
    out = []
    for n in range(heads):
        s = (q_plain[:, n] @ k_plain[:, n].t() + q_rot[:, n] @ k_rot.t()) * float(c["scale"])
        out.append(softmax_with_sink(s.masked_fill(~seen, float("-inf")), _c(w[f"{p}.sink"])[n]) @ v[:, n])
    return torch.cat(out, -1) @ _c(w[f"{p}.o"]).t()


# --------------------------------------------------------------------------- matrix memory

def mlstm_head(q: Tensor, k: Tensor, v: Tensor, i: Tensor, f: Tensor) -> Tensor:
    """One head, token by token.  q, k [t, d]; v [t, dv]; log gates i, f [t].  The scale m starts at zero."""
    S = torch.zeros((k.shape[1], v.shape[1]), dtype=q.dtype)
    n = torch.zeros((k.shape[1],), dtype=q.dtype)
    m = torch.zeros((), dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep * S + write * torch.outer(k[t], v[t])
        n = keep * n + write * k[t]
        m = new
        out.append((S.t() @ q[t]) / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6))
    return torch.stack(out)


def mlstm_gates(h: Tensor, w: Dict[str, Tensor], p: str, cap: float) -> Tuple[Tensor, Tensor]:
    """Log input and log forget gates [t, heads]."""
    soft = lambda z: cap * torch.tanh(z / cap)
    i = soft(h @ _c(w[f"{p}.i"]).t() + _c(w[f"{p}.i.b"]))
    return i, F.logsigmoid(soft(h @ _c(w[f"{p}.f"]).t() + _c(w[f"{p}.f.b"])))


def mlstm_mixer(h: Tensor, w: Dict[str, Tensor], p: str, c: dict, eps: float) -> Tensor:
    t, heads, d, dv = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q = (h @ _c(w[f"{p}.q"]).t()).view(t, heads, d) * d ** -0.5
    k = (h @ _c(w[f"{p}.k"]).t()).view(t, heads, d)
    v = (h @ _c(w[f"{p}.v"]).t()).view(t, heads, dv)
    i, f = mlstm_gates(h, w, p, float(c["gate_cap"]))
    o = torch.cat([unit_rms(mlstm_head(q[:, n], k[:, n], v[:, n], i[:, n], f[:, n]), eps) for n in range(heads)], -1)
    return (o * _c(w[f"{p}.norm"]) * torch.sigmoid(h @ _c(w[f"{p}.g"]).t())) @ _c(w[f"{p}.o"]).t()


# --------------------------------------------------------------------------- feed-forward

def expert(h: Tensor, w: Dict[str, Tensor], p: str) -> Tensor:
    return torch.clamp(h @ _c(w[f"{p}.up"]).t(), min=0.0) ** 2 @ _c(w[f"{p}.down"]).t()


def route(h: Tensor, w: Dict[str, Tensor], p: str, r: dict) -> Tuple[Tensor, Tensor]:
    """(chosen experts [t, top], their weights [t, top])."""
    s = torch.sigmoid(h.to(_COMPUTE[-1]) @ _c(w[f"{p}.router"]).t())
    choice = s + _c(w[f"{p}.correction"])
    groups = r.get("groups")
    if groups:
        size = r["experts"] // groups["count"]
        g = choice.view(-1, groups["count"], size)
        best = torch.topk(g, min(2, size), dim=-1).values.sum(-1)
        keep = torch.zeros_like(best, dtype=torch.bool).scatter_(1, torch.topk(best, groups["keep"], dim=-1).indices, True)
        choice = g.masked_fill(~keep[..., None], float("-inf")).flatten(1)
    chosen = torch.topk(choice, r["top"], dim=-1).indices
    picked = s.gather(1, chosen)
    return chosen, picked / (picked.sum(-1, keepdim=True) + 1e-20)


def moe_ff(h: Tensor, w: Dict[str, Tensor], p: str, c: dict) -> Tensor:
    chosen, weights = route(h, w, p, c["router"])
    out = torch.zeros_like(h)
    for e in range(c["router"]["experts"]):
        rows, place = torch.where(chosen == e)
        if len(rows):
            out[rows] += weights[rows, place][:, None] * expert(h[rows], w, f"{p}.e{e}")
    if c.get("shared"):
        out = out + expert(h, w, f"{p}.shared") * torch.sigmoid(h @ _c(w[f"{p}.shared.sg"]).t())
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
        h = squash(x, w, f"{p}.norm1")
        if ly["type"] == "attention":
            src = c.get("kv_from")
            y, kept[i] = attention_mixer(h, w, f"{p}.mix", c, eps, positions, None if src is None else kept[src])
        elif ly["type"] == "latent_attention":
            y = latent_attention_mixer(h, w, f"{p}.mix", c, eps, positions)
        elif ly["type"] == "mlstm":
            y = mlstm_mixer(h, w, f"{p}.mix", c, eps)
        else:
            raise ValueError(ly["type"])
        x = x + squash(y, w, f"{p}.norm1b")
        if ly.get("mlp") is not None:
            x = x + squash(moe_ff(squash(x, w, f"{p}.norm2"), w, f"{p}.mlp", ly["mlp"]), w, f"{p}.norm2b")
        seen.append(x)
    logits = squash(x, w, "final.norm") @ _c(w["head"]).t()
    return (logits, torch.stack(seen)) if return_layers else logits
