"""The Nafazen decoder beside the closest decoder of the framework (Godotar: the same kind of attention over a cached
latent, and routed experts) and the dense decoder at equal sizes: prefill and decode throughput through the same step
function, and each kernel of the new design alone against its roofline, beside the like kernel of those two.

    python -m lily_b200.bench.nafazen_bench [--sizes small mid] [--layers 4] [--no-kernels] [--no-models] [--table]
    python bench.py --design nafazen ...          (the same, as one JSON line)

Random weights in bfloat16.  The layers alternate as [attention + dense, attention + experts, attention + dense, attention
over the second layer's cache + experts]; the attention has the size's heads with 128 unrotated and 64 rotated
query/key columns, values of 128, a key/value latent of 512 and a query latent of 3 width / 8 and sees all keys; the dense
feed-forward has 3/2 of the dense decoder's width (two matrices instead of three), the experts are 16 of a quarter of it
each, of which a token takes 3, beside a shared expert of a quarter.  The Godotar decoder has attention layers alone here, without
window, with 16 experts (no identity outputs) of a quarter each and 4 a token, in every other layer, a SwiGLU of the dense
decoder's width else.  Timing as in ``design_bench``.
"""

from __future__ import annotations

import argparse
import json
import sys
from typing import List

import torch

from lily_b200.bench.design_bench import SIZES, dense_config, model_throughput
from lily_b200.bench.kbench import peaks, time_ms


def _attention(z: dict) -> dict:
    return {"heads": z["heads"], "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": 3 * z["width"] // 8, "kv_rank": 512,
            "scale": 192 ** -0.5, "rot": {"dims": 64, "base": 1000000.0}}


def nafazen_config(z: dict, layers: int) -> dict:
    dense = {"kind": "dense", "ff": 3 * z["ff"] // 2}
    moe = {"kind": "moe", "expert": {"ff": z["ff"] // 4}, "router": {"experts": 16, "top": 3}, "shared": {"ff": z["ff"] // 4}}
    scaled = dict(_attention(z), rot={"dims": 64, "base": 1000000.0, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}})
    own, reader = _attention(z), dict(_attention(z), kv_from=1)
    kinds = [{"type": "latent_attention", "mixer": scaled, "mlp": dense}, {"type": "latent_attention_2", "mixer": own, "mlp": moe},
             {"type": "latent_attention", "mixer": scaled, "mlp": dense}, {"type": "latent_attention_2", "mixer": reader, "mlp": moe}]
    return {"architecture": "Nafazen", "vocab": z["vocab"], "width": z["width"], "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6},
            "logit_softcap": 25.0, "layers": [kinds[i % 4] for i in range(layers)]}


def closest_config(z: dict, layers: int) -> dict:
    moe = {"kind": "moe", "expert": {"ff": z["ff"] // 4, "limit": 7.0}, "router": {"experts": 16, "identity": 0, "top": 4}}
    kinds = [{"type": "latent_attention", "mixer": _attention(z), "mlp": {"kind": "dense", "ff": z["ff"]}},
             {"type": "latent_attention", "mixer": _attention(z), "mlp": moe}]
    return {"architecture": "Godotar", "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "logit_scale": 1.0,
            "layers": [kinds[i % 2] for i in range(layers)]}


def kernel_table(z: dict, tokens: int, batch: int, context: int, reps: int = 30, copies: int = 3) -> List[dict]:
    """Each kernel alone, prefill shape (``tokens`` of one request) and decode shape (``batch`` requests of one token)."""
    from lily_b200.csrc import ops

    dev, dt = "cuda", torch.bfloat16
    pk = peaks()
    props = torch.cuda.get_device_properties(0)
    fp32_tflops = props.multi_processor_count * 128 * 2 * (props.clock_rate if hasattr(props, "clock_rate") else 1965000) / 1e9
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *shape: torch.randn(*shape, device=dev, generator=g)
    width, att = z["width"], _attention(z)
    heads, d, rot, rank, q_rank, dv = att["heads"], att["dim"], att["rot_dim"], att["kv_rank"], att["q_rank"], att["vdim"]
    row, page = rank + rot, 64
    rows: List[dict] = []

    def add(name, like, fns, bytes_moved, flops=0.0, flop_peak=None, shape=""):
        ms = time_ms(fns, reps, graph=True)
        r = {"kernel": name, "like": like, "shape": shape, "us": round(ms * 1e3, 2), "hbm_frac": round(bytes_moved / ms / 1e6 / pk["hbm_gbs"], 3)}
        if flops:
            r["flop_frac"] = round(flops / ms / 1e9 / (flop_peak or pk["bf16_tflops"]), 3)
            r["flop_peak"] = "fp32 fma" if flop_peak else "bf16 tensor"
        r["roofline_frac"] = max(r["hbm_frac"], r.get("flop_frac", 0.0))
        r["bound"] = r.get("flop_peak", "hbm") if r.get("flop_frac", 0.0) > r["hbm_frac"] else "hbm"
        rows.append(r)

    cos, sin = torch.rand(context + 1, rot // 2, device=dev), torch.rand(context + 1, rot // 2, device=dev)
    for label, n, reqs in (("prefill", tokens, 1), ("decode", batch, batch)):
        per = n // reqs
        pages = -(-per // page)
        table = torch.arange(1, reqs * pages + 1, device=dev, dtype=torch.int32).view(reqs, pages)
        pos = torch.arange(per, device=dev, dtype=torch.int32).repeat(reqs)
        token_req = torch.arange(reqs, device=dev, dtype=torch.int32).repeat_interleave(per)
        xs = [rnd(n, width).to(dt) for _ in range(copies)]
        # ---- around the sublayers
        resid = [rnd(n, width) for _ in range(copies)]
        gain, unit = torch.full((width,), 0.3, device=dev), torch.ones(width, device=dev)
        add("add_normed", "add_normed_rmsnorm", [lambda r=r, x=x: ops.add_normed(r, x, gain, 1e-6, 1.0, dt) for r, x in zip(resid, xs)],
            n * width * (8 + 2 + 2), shape=label)
        add("add_normed_rmsnorm (sandwich block)", "-", [lambda r=r, x=x: ops.add_normed_rmsnorm(r, x, gain, 1e-6, 1.0, unit, 1e-6, dt)
                                                         for r, x in zip(resid, xs)], n * width * (8 + 2 + 2), shape=label)
        # ---- around the attention
        gq, gk = torch.ones(q_rank, device=dev), torch.ones(rank, device=dev)
        downs = [rnd(n, q_rank + row) for _ in range(copies)]
        caches = [torch.zeros(reqs * pages + 1, page * row, device=dev, dtype=dt) for _ in range(copies)]
        add("latent_prepare", "add_rmsnorm", [lambda x=x, c=c: ops.latent_prepare(x, 0, q_rank, q_rank, rank, rot, rot, gq, gk, 1e-6, cos, sin, pos,
                                                                                  token_req, table, c, page) for x, c in zip(downs, caches)],
            n * (q_rank + row) * 6, shape=label)
        qs = [rnd(n, heads * (d + rot)).to(dt) for _ in range(copies)]
        carried = [torch.empty(n, heads * row, device=dev, dtype=dt) for _ in range(copies)]
        add("latent_query", "-", [lambda q=q, o=o: ops.latent_query(o, q, heads, d, rank, rot, rot, cos, sin, pos) for q, o in zip(qs, carried)],
            n * heads * rot * 4, shape=label)
        uk, uv = (rnd(heads, rank, d) / 16).to(dt), (rnd(heads, dv, rank) / 16).to(dt)
        add("head_linear (W_uk, into the queries)", "gate/up + down products", [
            lambda q=q, o=o: ops.head_linear(q.view(n, heads, d + rot)[:, :, :d], uk, out=o.view(n, heads, row)[:, :, :rank]) for q, o in zip(qs, carried)],
            n * heads * (d + rank) * 2 + uk.numel() * 2, 2.0 * n * heads * d * rank, shape=label)
        mixes = [rnd(n, heads, rank).to(dt) for _ in range(copies)]
        vals = torch.empty(n, heads * dv, device=dev, dtype=dt)
        add("head_linear (W_uv)", "gate/up + down products", [lambda m=m: ops.head_linear(m, uv, out=vals.view(n, heads, dv)) for m in mixes],
            n * heads * (dv + rank) * 2 + uv.numel() * 2, 2.0 * n * heads * dv * rank, shape=label)
        del mixes, carried, qs, downs
        # ---- the plain feed-forward beside the gated one of equal weight
        ff = 3 * z["ff"] // 2
        up, down = (rnd(ff, width) / width ** 0.5).to(dt), (rnd(width, ff) / ff ** 0.5).to(dt)
        add("xielu feed-forward", "gate/up + down products", [lambda x=x: ops.linear_auto(ops.linear_activation(x, up, "xielu", (0.7, 1.2)), down) for x in xs],
            2 * ff * width * 2 + n * (width * 4 + ff * 4), 4.0 * n * ff * width, shape=label)
        add("relu2 feed-forward (Gotivik)", "-", [lambda x=x: ops.linear_auto(ops.linear_activation(x, up, "relu2"), down) for x in xs],
            2 * ff * width * 2 + n * (width * 4 + ff * 4), 4.0 * n * ff * width, shape=label)
        zs = [rnd(n, ff).to(dt) for _ in range(copies)]
        add("activation xielu (a pass of its own)", "silu_mul", [lambda v=v: ops.activation(v, dt, "xielu", (0.7, 1.2)) for v in zs], n * ff * 4, shape=label)
        dense_gu, dense_dn = (rnd(2 * z["ff"], width) / width ** 0.5).to(dt), (rnd(width, z["ff"]) / z["ff"] ** 0.5).to(dt)
        add("gate/up + down products (dense)", "-", [lambda x=x: ops.linear(ops.silu_mul(ops.linear(x, dense_gu)), dense_dn) for x in xs],
            3 * z["ff"] * width * 2 + n * (width * 4 + z["ff"] * 4), 6.0 * n * z["ff"] * width, shape=label)
        del zs, up, down, dense_gu, dense_dn
        # ---- the experts beside the closest model's
        experts, e_ff = 16, z["ff"] // 4
        router = (rnd(experts + 8, width) / width ** 0.5).to(dt)
        corr = rnd(experts) / (2 * experts)
        add("moe_route + align (sigmoid, shared gate)", "moe_route + align", [
            lambda x=x: ops.moe_route(x, router, None, 3, experts, scores="sigmoid", renormalise=False, shared_gate=True, outputs=experts) for x in xs],
            n * width * 2 + (experts + 1) * width * 4, 2.0 * n * (experts + 1) * width, fp32_tflops, shape=label)
        router_g = router[:experts].contiguous()
        add("moe_route + align (Godotar)", "-", [lambda x=x: ops.moe_route(x, router_g, corr, 4, experts) for x in xs],
            n * width * 2 + experts * width * 4, 2.0 * n * experts * width, fp32_tflops, shape=label)
        gu, dn = (rnd(experts, 2 * e_ff, width) / width ** 0.5).to(dt), (rnd(experts, width, e_ff) / e_ff ** 0.5).to(dt)
        for name, like, top in (("moe_experts (weights on inputs, shared)", "moe_experts", 3), ("moe_experts (Godotar)", "-", 4)):
            ours = top == 3
            routed = [ops.moe_route(x, router, None, top, experts, scores="sigmoid", renormalise=False, shared_gate=True, outputs=experts) if ours
                      else ops.moe_route(x, router_g, corr, top, experts) for x in xs]
            how = dict(activation="silu", weight_on_input=True, shared=xs[0]) if ours else dict(limit=7.0, alpha=1.702)
            pairs = n * top
            touched = min(experts, pairs)
            add(name, like, [lambda x=x, r=r: ops.moe_experts(x, r, gu, dn, **how) for x, r in zip(xs, routed)],
                touched * 3 * e_ff * width * 2 + pairs * (width * 2 + e_ff * 4 + width * 4), 6.0 * pairs * e_ff * width, shape=label)
        del gu, dn

    # ---- attention over the cached latent (all keys) beside the dense decoder's attention
    nq, nkv, dd = z["heads"], z["kv_heads"], z["head"]
    pre, cu1 = torch.zeros(1, device=dev, dtype=torch.int32), torch.tensor([0, tokens], device=dev, dtype=torch.int32)
    pairs = tokens * (tokens + 1) / 2
    pages = -(-tokens // page)
    fns, dense_fns = [], []
    for _ in range(copies):
        table = (torch.randperm(pages, device=dev, generator=g) + 1).view(1, pages).to(torch.int32)
        cache, q = rnd(pages + 1, page * row).to(dt), (rnd(tokens, heads * row) / 8).to(dt)
        out = torch.empty((tokens, heads * rank), device=dev, dtype=dt)
        tile = ops.prefill_tile_rows(dt, row, page, tokens, dv=rank, values_in_keys=True, heads=heads)
        tr, ts = ops.prefill_tiles([0], [tokens], 0, tile, dev)
        fns.append(lambda q=q, cache=cache, table=table, out=out, tr=tr, ts=ts, tile=tile: ops.attention_prefill(
            q, cache, table, cu1, pre, tr, ts, out, heads, 1, row, page, att["scale"], None, tile_rows=tile, dv=rank, values_in_keys=True))
        kv, dq = rnd(pages + 1, 2, nkv, page, dd).to(dt), rnd(tokens, nq * dd).to(dt)
        dout = torch.empty_like(dq)
        tile = ops.prefill_tile_rows(dt, dd, page, tokens)
        tr, ts = ops.prefill_tiles([0], [tokens], 0, tile, dev)
        dense_fns.append(lambda q=dq, cache=kv, table=table, out=dout, tr=tr, ts=ts, tile=tile: ops.attention_prefill(
            q, cache, table, cu1, pre, tr, ts, out, nq, nkv, dd, page, dd ** -0.5, None, tile_rows=tile))
    add("latent attention, prefill", "attention_prefill", fns, tokens * (row + heads * (row + rank)) * 2, 2.0 * heads * (row + rank) * pairs,
        shape=f"{tokens} tokens")
    add("attention_prefill (dense heads)", "-", dense_fns, tokens * (2 * nkv + 2 * nq) * dd * 2, 4.0 * nq * dd * pairs, shape=f"{tokens} tokens")
    del fns, dense_fns
    pages = -(-context // page)
    fns, dense_fns = [], []
    for _ in range(copies):
        table = (torch.randperm(batch * pages, device=dev, generator=g) + 1).view(batch, pages).to(torch.int32)
        seq = torch.full((batch,), context, device=dev, dtype=torch.int32)
        cache, q = rnd(batch * pages + 1, page * row).to(dt), (rnd(batch, heads * row) / 8).to(dt)
        out = torch.empty((batch, heads * rank), device=dev, dtype=dt)
        plan = ops.plan_decode_attention(dt, batch, heads, 1, row, context, dv=rank, values_in_keys=True, page_size=page)
        scratch = torch.empty(max(1, plan.scratch_floats), device=dev)
        fns.append(lambda q=q, cache=cache, table=table, out=out, seq=seq, scratch=scratch, plan=plan: ops.attention_decode(
            q, cache, table, seq, out, scratch, plan.splits, heads, 1, row, page, att["scale"], None, dv=rank, values_in_keys=True))
        kv, dq = rnd(batch * pages + 1, 2, nkv, page, dd).to(dt), rnd(batch, nq * dd).to(dt)
        dout = torch.empty_like(dq)
        plan = ops.plan_decode_attention(dt, batch, nq, nkv, dd, context)
        scratch = torch.empty(max(1, plan.scratch_floats), device=dev)
        dense_fns.append(lambda q=dq, cache=kv, table=table, out=dout, seq=seq, scratch=scratch, plan=plan: ops.attention_decode(
            q, cache, table, seq, out, scratch, plan.splits, nq, nkv, dd, page, dd ** -0.5, None, stages=plan.stages))
    add("latent attention, decode", "attention_decode", fns, batch * context * row * 2 + batch * heads * (row + rank) * 2,
        2.0 * batch * heads * (row + rank) * context, shape=f"{batch} x {context}")
    add("attention_decode (dense heads)", "-", dense_fns, batch * context * 2 * nkv * dd * 2 + 2 * batch * nq * dd * 2,
        4.0 * batch * nq * dd * context, shape=f"{batch} x {context}")
    return rows


def run(sizes, layers, tokens, batch, context, steps, kernels=True, models=True) -> dict:
    out = {"design": "Nafazen", "beside": "the Godotar (attention layers alone) and the dense (Qwen3 layer) decoders at equal width and layers",
           "dtype": "bf16", "data": "synthetic: seeded random weights", "peaks": peaks(), "layers": layers,
           "prefill_tokens": tokens, "decode_batch": batch, "context": context, "sizes": {}}
    for name in sizes:
        z = SIZES[name]
        entry = {"shape": z}
        if models:
            entry["nafazen"] = model_throughput(nafazen_config(z, layers), tokens, batch, context, steps)
            entry["godotar"] = model_throughput(closest_config(z, layers), tokens, batch, context, steps)
            entry["dense"] = model_throughput(dense_config(z, layers, context), tokens, batch, context, steps)
        if kernels:
            entry["kernels"] = kernel_table(z, tokens, batch, context)
        out["sizes"][name] = entry
    return out


def main(argv=None) -> int:
    ap = argparse.ArgumentParser()
    ap.add_argument("--sizes", nargs="+", default=["small", "mid"], choices=sorted(SIZES))
    ap.add_argument("--layers", type=int, default=4)
    ap.add_argument("--tokens", type=int, default=2048)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--context", type=int, default=4096)
    ap.add_argument("--steps", type=int, default=20)
    ap.add_argument("--no-kernels", action="store_true")
    ap.add_argument("--no-models", action="store_true")
    ap.add_argument("--table", action="store_true", help="print the kernels as a table on stderr as well")
    a = ap.parse_args(argv)
    out = run(a.sizes, a.layers, a.tokens, a.batch, a.context, a.steps, kernels=not a.no_kernels, models=not a.no_models)
    if a.table:
        for name, entry in out["sizes"].items():
            for k in ("nafazen", "godotar", "dense"):
                if k in entry:
                    print(name, k, entry[k], file=sys.stderr)
            for r in entry.get("kernels", []):
                print(f"{name:6s} {r['kernel']:46s} {r['shape']:14s} {r['us']:10.2f} us  hbm {r['hbm_frac']:.3f}"
                      + (f"  {r['flop_peak']} {r['flop_frac']:.3f}" if "flop_frac" in r else "") + f"  ({r['bound']})", file=sys.stderr)
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
