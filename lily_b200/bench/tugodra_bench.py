"""The Tugodra decoder beside the closest decoder of the framework (Nafazen: attention over a cached latent and sigmoid-routed
experts with a shared one) and the dense decoder at equal sizes: prefill and decode throughput through the same step
function, and each kernel of the new design alone against its roofline, beside the like kernel of the others.

    python -m lily_b200.bench.tugodra_bench [--sizes small mid] [--layers 4] [--no-kernels] [--no-models] [--table]
    python bench.py --design tugodra ...          (the same, as one JSON line)

Random weights in bfloat16.  The layers alternate as [windowed attention, latent attention, mLSTM, windowed attention over the
first layer's keys and values], each with experts: 16 of a quarter of the dense feed-forward width, in 4 groups of which 2 are
kept, 3 a token, beside a shared expert of a quarter.  The windowed attention has the dense decoder's heads, all of a head
rotated; the latent attention its heads with 128 unrotated and 64 rotated columns, values of 128 and a latent of 512; the
mLSTM heads of 256 keys and 512 values, as many as fill the width.  The Nafazen decoder has its latent attention (query latent of
3 width / 8) and 16 experts of a quarter, 3 a token, in every layer.  Timing as in ``design_bench``.
"""

from __future__ import annotations

import argparse
import json
import sys
from typing import List

import torch

from lily_b200.bench.design_bench import SIZES, dense_config, model_throughput
from lily_b200.bench.kbench import peaks, time_ms

EXPERTS, TOP, GROUPS, KEEP = 16, 3, 4, 2


def _latent(z: dict) -> dict:
    return {"heads": z["heads"], "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5,
            "rot": {"dims": 64, "base": 1000000.0}}


def _mlstm(z: dict) -> dict:
    return {"heads": z["width"] // 512, "dim": 256, "vdim": 512, "gate_cap": 15.0}


def tugodra_config(z: dict, layers: int) -> dict:
    moe = {"kind": "moe", "expert": {"ff": z["ff"] // 4}, "router": {"experts": EXPERTS, "top": TOP, "groups": {"count": GROUPS, "keep": KEEP}},
           "shared": {"ff": z["ff"] // 4}}
    att = {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["head"], "vdim": z["head"], "scale": z["head"] ** 0.5,
           "mask": {"size": z["window"]}, "rot": {"dims": z["head"], "base": 1000000.0}}
    kinds = [("attention", att), ("latent_attention", _latent(z)), ("mlstm", _mlstm(z)), ("attention", dict(att, kv_from=0))]
    return {"architecture": "Tugodra", "vocab": z["vocab"], "width": z["width"], "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6},
            "layers": [{"type": kinds[i % 4][0], "mixer": kinds[i % 4][1], "mlp": moe} for i in range(layers)]}


def closest_config(z: dict, layers: int) -> dict:
    moe = {"kind": "moe", "expert": {"ff": z["ff"] // 4}, "router": {"experts": EXPERTS, "top": TOP}, "shared": {"ff": z["ff"] // 4}}
    layer = {"type": "latent_attention", "mixer": dict(_latent(z), q_rank=3 * z["width"] // 8), "mlp": moe}
    return {"architecture": "Nafazen", "vocab": z["vocab"], "width": z["width"], "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6},
            "layers": [layer] * layers}


def kernel_table(z: dict, tokens: int, batch: int, context: int, reps: int = 30, copies: int = 3) -> List[dict]:
    """Each kernel alone, prefill shape (``tokens`` of one request) and decode shape (``batch`` requests of one token)."""
    from lily_b200.csrc import ops

    dev, dt = "cuda", torch.bfloat16
    pk = peaks()
    props = torch.cuda.get_device_properties(0)
    fp32_tflops = props.multi_processor_count * 128 * 2 * (props.clock_rate if hasattr(props, "clock_rate") else 1965000) / 1e9
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *shape: torch.randn(*shape, device=dev, generator=g)
    width, page = z["width"], 64
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

    ml = _mlstm(z)
    nq, nkv, dd = z["heads"], z["kv_heads"], z["head"]
    for label, n, reqs in (("prefill", tokens, 1), ("decode", batch, batch)):
        per = n // reqs
        pages = -(-per // page)
        table = torch.arange(1, reqs * pages + 1, device=dev, dtype=torch.int32).view(reqs, pages)
        pos = torch.arange(per, device=dev, dtype=torch.int32).repeat(reqs)
        token_req = torch.arange(reqs, device=dev, dtype=torch.int32).repeat_interleave(per)
        cu = torch.arange(0, n + 1, per, device=dev, dtype=torch.int32)
        slots = torch.arange(1, reqs + 1, device=dev, dtype=torch.int32)
        xs = [rnd(n, width).to(dt) for _ in range(copies)]
        # ---- around the sublayers
        resid = [rnd(n, width) for _ in range(copies)]
        one, nil = torch.ones(width, device=dev), torch.zeros(width, device=dev)
        add("add_tanh_norm", "add_normed_rmsnorm", [lambda r=r, x=x: ops.add_tanh_norm(r, x, (0.4, one, nil), 1.0, (0.6, one, nil), dt)
                                                    for r, x in zip(resid, xs)], n * width * (8 + 2 + 2), shape=label)
        planes = [rnd(1, n, width) for _ in range(copies)]
        add("add_tanh_norm (float32 sums)", "add_normed_rmsnorm", [lambda r=r, x=x: ops.add_tanh_norm(r, x, (0.4, one, nil), 1.0, (0.6, one, nil), dt)
                                                                   for r, x in zip(resid, planes)], n * width * (8 + 4 + 2), shape=label)
        add("add_normed_rmsnorm (sandwich block)", "-", [lambda r=r, x=x: ops.add_normed_rmsnorm(r, x, one, 1e-6, 1.0, one, 1e-6, dt)
                                                         for r, x in zip(resid, xs)], n * width * (8 + 2 + 2), shape=label)
        # ---- around the windowed attention
        cos, sin = torch.rand(context + 1, dd // 2, device=dev), torch.rand(context + 1, dd // 2, device=dev)
        own = (nq + 2 * nkv) * dd
        ld = own + nq + -(own + nq) % 8
        unit = torch.ones(dd, device=dev)
        for name, cols in (("qk_norm_rope_write (rows with gates)", ld), ("qk_norm_rope_write", own)):
            qkvs = [rnd(n, cols).to(dt) for _ in range(copies)]
            caches = [torch.zeros(reqs * pages + 1, 2, nkv, page, dd, device=dev, dtype=dt) for _ in range(copies)]
            add(name, "qk_norm_rope_write" if cols == ld else "-", [
                lambda x=x, c=c: ops.qk_norm_rope_write(x, unit, unit, 1e-6, cos, sin, pos, token_req, table, c, nq, nkv, dd, dd, page, row=x.shape[1])
                for x, c in zip(qkvs, caches)], n * own * 4, shape=label)
        outs, gates = [rnd(n, nq * dd).to(dt) for _ in range(copies)], [rnd(n, ld).to(dt) for _ in range(copies)]
        add("sigmoid_head_gate", "sigmoid_gate", [lambda o=o, x=x: ops.sigmoid_head_gate(o, x, own, nq) for o, x in zip(outs, gates)],
            n * nq * (dd * 4 + 2), shape=label)
        wide = [rnd(n, nq * dd).to(dt) for _ in range(copies)]
        add("sigmoid_gate", "-", [lambda o=o, x=x: ops.sigmoid_gate(o, x) for o, x in zip(outs, wide)], n * nq * dd * 6, shape=label)
        del outs, gates, wide, qkvs, caches
        # ---- the matrix memory
        h, d, dv = ml["heads"], ml["dim"], ml["vdim"]
        key, inner = h * d, h * dv
        state_floats = h * (dv + 1) * d + h
        state_floats += -state_floats % 4
        projs = [(rnd(n, 2 * key + 2 * inner) / 2).to(dt) for _ in range(copies)]
        zs = [rnd(n, 2 * h) for _ in range(copies)]
        states = [torch.zeros(reqs + 1, state_floats, device=dev) for _ in range(copies)]
        ib, fb = torch.zeros(h, device=dev), torch.full((h,), 3.0, device=dev)
        plan = ops.mlstm_plan([per] * reqs, dt, h, d, dv, dev)
        room = torch.empty(max(1, ops.mlstm_workspace_floats(plan, h, d, dv)), device=dev)
        scan = lambda p, zz, s: ops.mlstm_scan(p, 0, key, 2 * key, zz, 0, h, ib, fb, 15.0, d ** -0.5, s, cu, slots, reqs, h, d, dv, plan=plan,
                                               workspace=room)
        # counted as the token-by-token recurrence: decay, write and read-out of every entry
        add("mlstm_scan", "wkv_scan", [lambda p=p, zz=zz, s=s: scan(p, zz, s) for p, zz, s in zip(projs, zs, states)],
            n * (2 * key + inner) * 2 + n * inner * 4 + 2 * reqs * state_floats * 4, 6.0 * n * h * d * (dv + 1), fp32_tflops, shape=label)
        ys = [scan(p, zz, s) for p, zz, s in zip(projs, zs, states)]
        gain = torch.ones(inner, device=dev)
        add("mlstm_out", "group_rmsnorm_gate", [
            lambda y=y, p=p, s=s: ops.mlstm_out(*y, p, 2 * key + inner, gain, 1e-6, 1e-6, s, h * (dv + 1) * d, cu, token_req, slots, dt)
            for y, p, s in zip(ys, projs, states)], n * inner * 8, shape=label)
        del ys
        wh, wd = width // 64, 64                                              # the wkv mixer of the Godotar decoder
        rkv = [(rnd(n, width).to(dt), (rnd(n, width) / 8).to(dt), rnd(n, width).to(dt), -torch.rand(n, width, device=dev, generator=g)) for _ in range(copies)]
        wstates = [torch.zeros(reqs + 1, wh * wd * wd, device=dev) for _ in range(copies)]
        u = rnd(wh, wd)
        wplan = ops.wkv_plan([per] * reqs, dev)
        wroom = torch.empty(max(1, ops.wkv_workspace_floats(wplan, wh, wd)), device=dev)
        add("wkv_scan (Godotar)", "-", [lambda x=x, s=s: ops.wkv_scan(x[0], x[1], x[2], x[3], u, s, cu, slots, reqs, wh, wd, plan=wplan, workspace=wroom)
                                        for x, s in zip(rkv, wstates)],
            n * width * (6 + 8) + 2 * reqs * wh * wd * wd * 4, 6.0 * n * wh * wd * wd, fp32_tflops, shape=label)
        yy = [rnd(n, width) for _ in range(copies)]
        add("group_rmsnorm_gate (Godotar)", "-", [lambda y=y, x=x: ops.group_rmsnorm_gate(y, x[0], one, wh, 1e-6) for y, x in zip(yy, rkv)],
            n * width * 8, shape=label)
        del rkv, wstates, yy, projs, states
        # ---- the experts beside the closest model's
        e_ff = z["ff"] // 4
        router, corr = (rnd(EXPERTS + 8, width) / width ** 0.5).to(dt), rnd(EXPERTS) / 4
        grouped = dict(scores="sigmoid", shared_gate=True, outputs=EXPERTS, groups=GROUPS, keep_groups=KEEP)
        plain = dict(scores="sigmoid", renormalise=False, shared_gate=True, outputs=EXPERTS)
        add("moe_route + align (groups, correction)", "moe_route + align", [lambda x=x: ops.moe_route(x, router, corr, TOP, EXPERTS, **grouped) for x in xs],
            n * width * 2 + (EXPERTS + 1) * width * 2, 2.0 * n * (EXPERTS + 1) * width, fp32_tflops, shape=label)
        add("moe_route + align (Nafazen)", "-", [lambda x=x: ops.moe_route(x, router, None, TOP, EXPERTS, **plain) for x in xs],
            n * width * 2 + (EXPERTS + 1) * width * 2, 2.0 * n * (EXPERTS + 1) * width, fp32_tflops, shape=label)
        up, dn = (rnd(EXPERTS, e_ff, width) / width ** 0.5).to(dt), (rnd(EXPERTS, width, e_ff) / e_ff ** 0.5).to(dt)
        gu = (rnd(EXPERTS, 2 * e_ff, width) / width ** 0.5).to(dt)
        pairs = n * TOP
        touched = min(EXPERTS, pairs)
        for name, like, w_in, mats, how, route in (
                ("moe_experts (ungated)", "moe_experts", up, 2, dict(activation="relu2"), (corr, grouped)),
                ("moe_experts (Nafazen)", "-", gu, 3, dict(activation="silu", weight_on_input=True), (None, plain))):
            routed = [ops.moe_route(x, router, route[0], TOP, EXPERTS, **route[1]) for x in xs]
            add(name, like, [lambda x=x, r=r: ops.moe_experts(x, r, w_in, dn, shared=x, **how) for x, r in zip(xs, routed)],
                touched * mats * e_ff * width * 2 + pairs * (width * 2 + e_ff * 4 + width * 4), 2.0 * mats * pairs * e_ff * width, shape=label)
        del up, dn, gu

    # ---- attention: the latent form with and without a sink, the windowed form beside the dense decoder's (the same kernels)
    lat = _latent(z)
    heads, rank = lat["heads"], lat["kv_rank"]
    row = rank + lat["rot_dim"]
    sinks = rnd(heads)
    pre, cu1 = torch.zeros(1, device=dev, dtype=torch.int32), torch.tensor([0, tokens], device=dev, dtype=torch.int32)
    pages = -(-tokens // page)
    window = z["window"]
    seen = lambda w: sum(min(i + 1, w or tokens) for i in range(tokens))
    forms = [("latent attention with sinks", "latent attention", True, None), ("latent attention (Nafazen)", "-", False, None)]
    for name, like, sunk, _ in forms:
        fns = []
        for _c in range(copies):
            table = (torch.randperm(pages, device=dev, generator=g) + 1).view(1, pages).to(torch.int32)
            cache, q = rnd(pages + 1, page * row).to(dt), (rnd(tokens, heads * row) / 8).to(dt)
            out = torch.empty((tokens, heads * rank), device=dev, dtype=dt)
            tile = ops.prefill_tile_rows(dt, row, page, tokens, dv=rank, values_in_keys=True, heads=heads)
            tr, ts = ops.prefill_tiles([0], [tokens], 0, tile, dev)
            fns.append(lambda q=q, cache=cache, table=table, out=out, tr=tr, ts=ts, tile=tile: ops.attention_prefill(
                q, cache, table, cu1, pre, tr, ts, out, heads, 1, row, page, lat["scale"], None, tile_rows=tile, dv=rank, values_in_keys=True,
                sinks=sinks if sunk else None))
        add(name + ", prefill", like, fns, tokens * (row + heads * (row + rank)) * 2, 2.0 * heads * (row + rank) * seen(None), shape=f"{tokens} tokens")
    for name, like, w in (("windowed attention", "attention", window), ("attention (dense)", "-", None)):
        fns = []
        for _c in range(copies):
            table = (torch.randperm(pages, device=dev, generator=g) + 1).view(1, pages).to(torch.int32)
            kv, q = rnd(pages + 1, 2, nkv, page, dd).to(dt), rnd(tokens, nq * dd).to(dt)
            out = torch.empty_like(q)
            tile = ops.prefill_tile_rows(dt, dd, page, tokens)
            tr, ts = ops.prefill_tiles([0], [tokens], 0, tile, dev)
            fns.append(lambda q=q, cache=kv, table=table, out=out, tr=tr, ts=ts, tile=tile: ops.attention_prefill(
                q, cache, table, cu1, pre, tr, ts, out, nq, nkv, dd, page, dd ** -0.5, w, tile_rows=tile))
        add(name + ", prefill", like, fns, tokens * (2 * nkv + 2 * nq) * dd * 2, 4.0 * nq * dd * seen(w), shape=f"{tokens} tokens")
    pages = -(-context // page)
    for name, like, sunk, _ in forms:
        fns = []
        for _c in range(copies):
            table = (torch.randperm(batch * pages, device=dev, generator=g) + 1).view(batch, pages).to(torch.int32)
            seq = torch.full((batch,), context, device=dev, dtype=torch.int32)
            cache, q = rnd(batch * pages + 1, page * row).to(dt), (rnd(batch, heads * row) / 8).to(dt)
            out = torch.empty((batch, heads * rank), device=dev, dtype=dt)
            plan = ops.plan_decode_attention(dt, batch, heads, 1, row, context, dv=rank, values_in_keys=True, page_size=page)
            scratch = torch.empty(max(1, plan.scratch_floats), device=dev)
            fns.append(lambda q=q, cache=cache, table=table, out=out, seq=seq, scratch=scratch, plan=plan: ops.attention_decode(
                q, cache, table, seq, out, scratch, plan.splits, heads, 1, row, page, lat["scale"], None, dv=rank, values_in_keys=True,
                sinks=sinks if sunk else None))
        add(name + ", decode", like, fns, batch * context * row * 2 + batch * heads * (row + rank) * 2, 2.0 * batch * heads * (row + rank) * context,
            shape=f"{batch} x {context}")
    for name, like, w in (("windowed attention", "attention", window), ("attention (dense)", "-", None)):
        fns = []
        keys = min(context, w or context)
        for _c in range(copies):
            table = (torch.randperm(batch * pages, device=dev, generator=g) + 1).view(batch, pages).to(torch.int32)
            seq = torch.full((batch,), context, device=dev, dtype=torch.int32)
            kv, q = rnd(batch * pages + 1, 2, nkv, page, dd).to(dt), rnd(batch, nq * dd).to(dt)
            out = torch.empty_like(q)
            plan = ops.plan_decode_attention(dt, batch, nq, nkv, dd, keys)
            scratch = torch.empty(max(1, plan.scratch_floats), device=dev)
            fns.append(lambda q=q, cache=kv, table=table, out=out, seq=seq, scratch=scratch, plan=plan: ops.attention_decode(
                q, cache, table, seq, out, scratch, plan.splits, nq, nkv, dd, page, dd ** -0.5, w, stages=plan.stages))
        add(name + ", decode", like, fns, batch * keys * 2 * nkv * dd * 2 + 2 * batch * nq * dd * 2, 4.0 * batch * nq * dd * keys,
            shape=f"{batch} x {context}")
    return rows


def run(sizes, layers, tokens, batch, context, steps, kernels=True, models=True) -> dict:
    out = {"design": "Tugodra", "beside": "the Nafazen and the dense (Qwen3 layer) decoders at equal width and layers",
           "dtype": "bf16", "data": "synthetic: seeded random weights", "peaks": peaks(), "layers": layers,
           "prefill_tokens": tokens, "decode_batch": batch, "context": context, "sizes": {}}
    for name in sizes:
        z = SIZES[name]
        entry = {"shape": z}
        if models:
            entry["tugodra"] = model_throughput(tugodra_config(z, layers), tokens, batch, context, steps)
            entry["nafazen"] = model_throughput(closest_config(z, layers), tokens, batch, context, steps)
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
            for k in ("tugodra", "nafazen", "dense"):
                if k in entry:
                    print(name, k, entry[k], file=sys.stderr)
            for r in entry.get("kernels", []):
                print(f"{name:6s} {r['kernel']:46s} {r['shape']:14s} {r['us']:10.2f} us  hbm {r['hbm_frac']:.3f}"
                      + (f"  {r['flop_peak']} {r['flop_frac']:.3f}" if "flop_frac" in r else "") + f"  ({r['bound']})", file=sys.stderr)
    print(json.dumps(out))
    return 0


if __name__ == "__main__":
    sys.exit(main())
