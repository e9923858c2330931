"""Small Tugodra configurations and random weights for the tests, made here from the design alone (no code of
``lily_b200`` decides a name or a shape)."""

from __future__ import annotations

import json
import math
import os
import random
from typing import Dict, Optional

import torch


def attention(heads=4, kv_heads=2, dim=12, vdim=12, window: Optional[int] = 9, scale=0.4, dims=None, base=10000.0,
              kv_from: Optional[int] = None, mlp: Optional[dict] = None) -> dict:
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"dims": dim if dims is None else dims, "base": base}}
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def latent(heads=3, dim=8, rot_dim=4, vdim=12, kv_rank=24, scale=0.35, base=10000.0, mlp: Optional[dict] = None) -> dict:
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"dims": rot_dim, "base": base}}}


def mlstm(heads=2, dim=8, vdim=12, cap=10.0, mlp: Optional[dict] = None) -> dict:
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def moe(ff=24, experts=6, top=2, groups: Optional[int] = 3, keep=2, shared: Optional[int] = 40) -> dict:
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups:
        out["router"]["groups"] = {"count": groups, "keep": keep}
    if shared:
        out["shared"] = {"ff": shared}
    return out


# Sizes that differ from layer to layer; windows of 1 and more; a layer's keys read by a layer that looks less far and by one
# that looks further back than the layer itself; values of another size than keys; a part of a head rotated; layers without
# feed-forward; groups of one expert, one group, no groups; with and without a shared expert; all experts chosen.
VARIED = {"architecture": "Tugodra", "vocab": 131, "width": 48, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.7},
          "layers": [attention(mlp=moe()),
                     latent(heads=2, dim=6, rot_dim=8, vdim=6, kv_rank=18, scale=0.5, base=100.0, mlp=moe(ff=16, experts=5, top=2, groups=5, keep=3)),
                     mlstm(mlp=moe(ff=8, experts=4, top=4, groups=1, keep=1, shared=None)),
                     attention(window=23, kv_from=0),
                     attention(heads=6, kv_heads=1, dim=20, vdim=7, dims=8, window=1, scale=0.3, base=50.0, mlp=moe(groups=None, top=3, shared=16)),
                     mlstm(heads=3, dim=20, vdim=5, cap=4.0),
                     attention(window=4, kv_from=0, scale=0.7, mlp=moe(ff=40, experts=8, top=1, groups=2, keep=1, shared=24)),
                     latent(heads=5, dim=4, rot_dim=2, vdim=9, kv_rank=40)]}

# Sharp attention: a large scale puts nearly all weight on the best visible key, so a key that is lost, kept too long, or
# turned by another angle changes the output outright.
SHARP = {"architecture": "Tugodra", "vocab": 97, "width": 32, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
         "layers": [attention(heads=2, kv_heads=1, dim=8, vdim=8, window=17, scale=2.0, mlp=moe(groups=None, top=6)),
                    attention(heads=2, kv_heads=1, dim=8, vdim=8, window=40, scale=2.0, kv_from=0),
                    latent(heads=2, dim=8, rot_dim=8, vdim=8, kv_rank=16, scale=3.0, mlp=moe(groups=None, top=6)),
                    mlstm(heads=1, dim=16, vdim=16, cap=20.0)]}

# Wider layers on the tensor-core kernels' sizes.
WIDE = {"architecture": "Tugodra", "vocab": 257, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.2},
        "layers": [attention(heads=8, kv_heads=2, dim=64, vdim=64, window=70, scale=0.1, mlp=moe(ff=64, experts=8, top=3, groups=4, keep=2, shared=96)),
                   latent(heads=6, dim=32, rot_dim=16, vdim=32, kv_rank=112, scale=0.14, mlp=moe(ff=32, experts=8, top=2, groups=2, keep=1, shared=64)),
                   mlstm(heads=2, dim=64, vdim=96, cap=15.0, mlp=moe(ff=32, experts=4, top=2, groups=None, shared=64)),
                   attention(heads=8, kv_heads=2, dim=64, vdim=64, window=130, scale=0.08, kv_from=0),
                   mlstm(heads=4, dim=48, vdim=32, cap=8.0),
                   attention(heads=2, kv_heads=2, dim=128, vdim=128, dims=64, window=33, scale=0.06, mlp=moe(ff=64, experts=4, top=1, groups=2, keep=2))]}


def random_config(seed: int) -> dict:
    """A configuration drawn at random: 2 to 7 layers of any mixer, with and without feed-forward, readers of an earlier layer's
    keys with windows of their own, widths that are and are not multiples of 8."""
    rng = random.Random(seed)
    width = rng.choice([24, 40, 64, 72, 96, 136, 44, 50])
    layers = []
    for i in range(rng.randint(2, 7)):
        mlp = None
        if rng.random() < 0.6:
            groups, size = rng.choice([(None, 1), (1, 4), (2, 3), (4, 2), (3, 1)])
            experts = rng.randint(1, 9) if groups is None else groups * size
            keep = rng.randint(1, groups) if groups else 1
            top = rng.randint(1, min(4, experts if groups is None else keep * size))
            mlp = moe(rng.choice([8, 24, 40]), experts, top, groups, keep, rng.choice([None, 8, 48]))
        kind = rng.choice(["attention", "attention", "latent", "mlstm"])
        if kind == "attention":
            own = [j for j, ly in enumerate(layers) if ly["type"] == "attention" and "kv_from" not in ly["mixer"]]
            window = rng.choice([1, 5, 16, 17, 64, 65, 100])
            if own and rng.random() < 0.5:
                j = rng.choice(own)
                ly = attention(window=window, kv_from=j, mlp=mlp)
                ly["mixer"] = dict(layers[j]["mixer"], mask={"size": window}, kv_from=j, scale=rng.choice([0.1, 0.5]))
            else:
                kv = rng.choice([1, 2, 3])
                dim = rng.choice([4, 12, 16, 32, 64, 64, 128])
                ly = attention(kv * rng.choice([1, 2, 4]), kv, dim, dim if rng.random() < 0.6 else rng.choice([5, 8, 48]), window,
                               rng.choice([0.1, 0.3]), rng.choice([dim, dim // 2]), rng.choice([100.0, 10000.0]), mlp=mlp)
        elif kind == "latent":
            rank = rng.choice([8, 24, 40, 64, 120]) if rng.random() < 0.7 else rng.choice([10, 18, 34])
            ly = latent(rng.randint(1, 6), rng.choice([4, 8, 16, 32]), rng.choice([2, 4, 8, 16]), rng.choice([4, 8, 20, 32]), rank,
                        rng.choice([0.2, 0.5]), rng.choice([100.0, 10000.0]), mlp=mlp)
        else:
            ly = mlstm(rng.randint(1, 4), rng.choice([4, 6, 16, 32, 48, 64, 128]), rng.choice([4, 7, 16, 32, 64, 96]), rng.choice([2.0, 8.0, 15.0]), mlp=mlp)
        layers.append(ly)
    return {"architecture": "Tugodra", "vocab": rng.choice([61, 128, 300]), "width": width, "norm": {"eps": rng.choice([1e-5, 1e-6])},
            "embedding": {"scale": rng.choice([0.25, 1.0, 3.0])}, "layers": layers}


def shapes(cfg: dict) -> Dict[str, tuple]:
    w = cfg["width"]
    out = {"embed": (cfg["vocab"], w), "head": (cfg["vocab"], w)}

    def norm(name):
        out.update({name: (w,), f"{name}.b": (w,), f"{name}.alpha": ()})
    norm("final.norm")
    for i, ly in enumerate(cfg["layers"]):
        m, p = ly["mixer"], f"l{i}"
        h = m["heads"]
        norm(f"{p}.norm1")
        norm(f"{p}.norm1b")
        mix = lambda name, *shape: out.update({f"{p}.mix.{name}": shape})
        if ly["type"] == "attention":
            mix("q", h * m["dim"], w)
            if m.get("kv_from") is None:
                mix("k", m["kv_heads"] * m["dim"], w)
                mix("v", m["kv_heads"] * m["vdim"], w)
            mix("g", h, w)
        elif ly["type"] == "latent_attention":
            mix("q", h * (m["dim"] + m["rot_dim"]), w)
            mix("dkv", m["kv_rank"] + m["rot_dim"], w)
            mix("dkv.norm", m["kv_rank"])
            mix("uk", h * m["dim"], m["kv_rank"])
            mix("uv", h * m["vdim"], m["kv_rank"])
            mix("sink", h)
        else:
            for name, cols in (("q", m["dim"]), ("k", m["dim"]), ("v", m["vdim"]), ("g", m["vdim"]), ("i", 1), ("f", 1)):
                mix(name, h * cols, w)
            mix("i.b", h)
            mix("f.b", h)
            mix("norm", h * m["vdim"])
        mix("o", w, h * m["vdim"])
        mlp = ly["mlp"]
        if mlp is None:
            continue
        norm(f"{p}.norm2")
        norm(f"{p}.norm2b")
        out.update({f"{p}.mlp.router": (mlp["router"]["experts"], w), f"{p}.mlp.correction": (mlp["router"]["experts"],)})
        parts = [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        if mlp.get("shared"):
            parts.append(("shared", mlp["shared"]["ff"]))
            out[f"{p}.mlp.shared.sg"] = (1, w)
        for name, ff in parts:
            out.update({f"{p}.mlp.{name}.up": (ff, w), f"{p}.mlp.{name}.down": (w, ff)})
    return out


def make_weights(cfg: dict, seed: int, dtype=torch.float32) -> Dict[str, torch.Tensor]:
    """Random weights at scales that keep every mechanism alive: projections of unit gain, norms whose tanh is neither linear
    nor saturated, sinks that take a good part of the softmax, forget gates from fast to slow, input gates on both sides of
    the running maximum, router scores that spread, corrections that change choices and go below zero."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        n = lambda: torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = n()
        elif last == "alpha":
            t = 0.7 + 0.2 * torch.rand((), generator=g)
        elif last in ("norm1", "norm1b", "norm2", "norm2b") or name == "final.norm":
            t = 1.0 + 0.2 * n()
        elif name.endswith((".i.b",)):
            t = -0.5 + n()
        elif name.endswith(".f.b"):
            t = 2.5 + 2.0 * n()
        elif last == "b":
            t = 0.2 * n()
        elif name.endswith((".dkv.norm", ".mix.norm")):
            t = 1.0 + 0.2 * n()
        elif last == "sink":
            t = 1.0 + n()
        elif last == "correction":
            t = 0.4 * n() - 0.3
        elif last == "router" or name.endswith((".mix.i", ".mix.f")):
            t = 2.0 * n() / math.sqrt(shape[-1])
        else:
            t = n() / math.sqrt(shape[-1])
        out[name] = t.to(dtype)
    return out


def write_model_dir(path: str, cfg: dict, weights: Dict[str, torch.Tensor]) -> str:
    from lily_b200.weights.safetensors_io import write_safetensors

    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"),
                      [(n, t.dtype, tuple(t.shape)) for n, t in weights.items()], {"format": "pt"},
                      produce=lambda n: weights[n])
    return path


def tokens(n: int, vocab: int, seed: int):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()
