"""Small Nafazen configurations and random weights for the tests, made here from the design alone (no code of
``lily_b200`` decides a name or a shape)."""

from __future__ import annotations

import json
import math
import os
import random
from typing import Dict, Optional

import torch


def layer(kind="latent_attention", heads=3, dim=8, rot_dim=4, vdim=12, q_rank=20, kv_rank=24, scale=0.35, base=10000.0,
          yarn: Optional[dict] = None, kv_from: Optional[int] = None, mlp: Optional[dict] = None) -> dict:
    rot = {"dims": rot_dim, "base": base}
    if yarn:
        rot["scaling"] = yarn
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale, "rot": rot}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": kind, "mixer": m, "mlp": mlp}


def dense(ff=40) -> dict:
    return {"kind": "dense", "ff": ff}


def moe(ff=24, experts=5, top=2, shared: Optional[int] = 40) -> dict:
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}

# Sizes that differ from layer to layer; a layer's rows read by two later layers of other head counts and head sizes, with
# other layers between; one layer without feed-forward; top of 1 and of all experts; with and without a shared expert.
VARIED = {"architecture": "Nafazen", "vocab": 131, "width": 48, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.7},
          "logit_softcap": 9.0,
          "layers": [layer(yarn=YARN, rot_dim=12, mlp=dense(56)),
                     layer("latent_attention_2", heads=2, dim=6, rot_dim=8, vdim=6, q_rank=10, kv_rank=18, scale=0.5, base=100.0, mlp=moe()),
                     layer(heads=5, dim=4, rot_dim=6, vdim=4, kv_rank=16, yarn=dict(YARN, factor=1.0), mlp=moe(ff=16, experts=3, top=3, shared=None)),
                     layer("latent_attention_2", heads=4, dim=10, rot_dim=8, vdim=14, q_rank=24, kv_rank=18, scale=0.4, base=100.0, kv_from=1),
                     layer("latent_attention_2", heads=1, dim=16, rot_dim=8, vdim=9, q_rank=7, kv_rank=18, scale=0.7, base=100.0, kv_from=1,
                           mlp=moe(ff=8, experts=7, top=1, shared=16))]}

# Sharp attention: a large scale puts nearly all weight on the best visible key, so a key that is lost, rotated by another
# angle or read from another layer's rows changes the output outright.
SHARP = {"architecture": "Nafazen", "vocab": 97, "width": 32, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
         "logit_softcap": 20.0,
         "layers": [layer("latent_attention_2", heads=2, dim=8, rot_dim=8, vdim=8, q_rank=16, kv_rank=16, scale=3.0, mlp=dense(32)),
                    layer("latent_attention_2", heads=3, dim=4, rot_dim=8, vdim=4, q_rank=12, kv_rank=16, scale=3.0, kv_from=0, mlp=dense(24)),
                    layer(heads=1, dim=16, rot_dim=2, vdim=16, q_rank=8, kv_rank=32, scale=3.0, yarn=YARN, mlp=dense(32))]}

# Wider layers whose rows and ranks are whole 16-byte pieces (the tensor-core kernels' sizes), no cap on the logits.
WIDE = {"architecture": "Nafazen", "vocab": 257, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 0.6},
        "layers": [layer(heads=6, dim=32, rot_dim=16, vdim=32, q_rank=48, kv_rank=112, scale=0.14, yarn=dict(YARN, original=512),
                         mlp=moe(ff=64, experts=8, top=4, shared=128)),
                   layer("latent_attention_2", heads=4, dim=24, rot_dim=32, vdim=40, q_rank=64, kv_rank=64, scale=0.13, base=500.0, mlp=dense(256)),
                   layer("latent_attention_2", heads=8, dim=16, rot_dim=32, vdim=16, q_rank=32, kv_rank=64, scale=0.14, base=500.0, kv_from=1,
                         mlp=moe(ff=32, experts=4, top=2, shared=96))]}


def random_config(seed: int) -> dict:
    """A configuration drawn at random: 2 to 6 layers of either kind, any feed-forward or none, some of them reading the
    rows of an earlier one, widths that are and are not multiples of 8, with and without YaRN, cap and shared expert."""
    rng = random.Random(seed)
    width = rng.choice([24, 40, 64, 72, 96, 136, 44, 50])
    layers = []
    for i in range(rng.randint(2, 6)):
        mlp = rng.choice([dense(rng.choice([16, 40, 72])), None])
        if rng.random() < 0.5:
            experts = rng.randint(1, 9)
            mlp = moe(rng.choice([8, 24, 40]), experts, rng.randint(1, min(4, experts)), rng.choice([None, 8, 48]))
        own = [j for j, ly in enumerate(layers) if "kv_from" not in ly["mixer"]]
        common = dict(heads=rng.randint(1, 6), dim=rng.choice([4, 8, 16, 32]), vdim=rng.choice([4, 8, 20, 32]),
                      q_rank=rng.choice([8, 12, 32]), scale=rng.choice([0.2, 0.5]), mlp=mlp)
        if own and rng.random() < 0.4:
            j = rng.choice(own)
            src = layers[j]["mixer"]
            ly = layer(layers[j]["type"], rot_dim=src["rot_dim"], kv_rank=src["kv_rank"], kv_from=j, **common)
            ly["mixer"]["rot"] = src["rot"]
        else:
            rank = rng.choice([8, 24, 40, 64, 120]) if rng.random() < 0.7 else rng.choice([10, 18, 34])
            yarn = {"factor": rng.choice([0.5, 1.0, 2.0, 8.0]), "original": rng.choice([16, 100, 2048]), "fast": rng.choice([4.0, 32.0]),
                    "slow": rng.choice([0.25, 1.0])} if rng.random() < 0.5 else None
            ly = layer(rng.choice(["latent_attention", "latent_attention_2"]), rot_dim=rng.choice([2, 4, 8, 16]), kv_rank=rank,
                       base=rng.choice([100.0, 10000.0]), yarn=yarn, **common)
        layers.append(ly)
    cfg = {"architecture": "Nafazen", "vocab": rng.choice([61, 128, 300]), "width": width, "norm": {"eps": rng.choice([1e-5, 1e-6])},
           "embedding": {"scale": rng.choice([0.25, 1.0, 3.0])}, "layers": layers}
    if rng.random() < 0.7:
        cfg["logit_softcap"] = rng.choice([5.0, 25.0])
    return cfg


def shapes(cfg: dict) -> Dict[str, tuple]:
    w = cfg["width"]
    out = {"embed": (cfg["vocab"], w), "head": (cfg["vocab"], w), "final.norm": ()}
    for i, ly in enumerate(cfg["layers"]):
        m, p = ly["mixer"], f"l{i}"
        h = m["heads"]
        out[f"{p}.norm1"] = ()
        out.update({f"{p}.mix.dq": (m["q_rank"], w), f"{p}.mix.dq.norm": (m["q_rank"],),
                    f"{p}.mix.uq": (h * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                    f"{p}.mix.uk": (h * m["dim"], m["kv_rank"]), f"{p}.mix.uv": (h * m["vdim"], m["kv_rank"]),
                    f"{p}.mix.o": (w, h * m["vdim"])})
        if m.get("kv_from") is None:
            out.update({f"{p}.mix.dkv": (m["kv_rank"] + m["rot_dim"], w), f"{p}.mix.dkv.norm": (m["kv_rank"],)})
        mlp = ly["mlp"]
        if mlp is None:
            continue
        out[f"{p}.norm2"] = ()
        if mlp["kind"] == "dense":
            out.update({f"{p}.mlp.up": (mlp["ff"], w), f"{p}.mlp.down": (w, mlp["ff"]), f"{p}.mlp.act": (2,)})
            continue
        out[f"{p}.mlp.router"] = (mlp["router"]["experts"], w)
        groups = [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        if mlp.get("shared"):
            groups.append(("shared", mlp["shared"]["ff"]))
            out[f"{p}.mlp.shared.sg"] = (1, w)
        for name, ff in groups:
            out.update({f"{p}.mlp.{name}.gate": (ff, w), f"{p}.mlp.{name}.up": (ff, w), f"{p}.mlp.{name}.down": (w, ff)})
    return out


def make_weights(cfg: dict, seed: int, dtype=torch.float32) -> Dict[str, torch.Tensor]:
    """Random weights at scales that keep every mechanism alive: projections of unit gain, gains around a half (the stream
    grows by every sublayer and is never normalised), router logits that spread over the sigmoid, activation factors on
    both sides of zero."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        n = lambda: torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = n()
        elif last in ("norm1", "norm2"):
            t = 0.5 + 0.2 * n()
        elif name == "final.norm":
            t = 1.3 + 0.1 * n()
        elif name.endswith(("dq.norm", "dkv.norm")):
            t = 1.0 + 0.2 * n()
        elif last == "act":
            t = 0.8 * n()
        elif last == "router":
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
