"""Each mechanism of the Tugodra decoder alone: parts and kernel faces (CUDA on the GPU, their plain statements on the CPU)
against the functions of ``plain_tugodra``, with inputs made so that a fault shows: keys that stand out at page borders, far
back and on either side of a window's edge, sinks that take most of the softmax, choice scores below zero, groups whose best
expert must not be chosen, values written hundreds of tokens ago, sizes that are not powers of two."""

import math

import pytest
import torch

import kernel_refs
import plain_tugodra as pt
from lily_b200.engine.batch import StepEntry, Workspace, build_step_batch
from lily_b200.parts.attention import AttentionSpec, LayerCache
from lily_b200.parts.base import BuildContext, build_part
from lily_b200.parts.experts import RoutedExpertsSpec
from lily_b200.parts.latent_attention import LatentAttentionSpec
from lily_b200.parts.mlstm import MlstmSpec
from lily_b200.parts.norm import DynamicTanhSpec, NormedDelta, RMSNormSpec, TanhDelta, enter_stream
from lily_b200.parts.rope import RopeSpec

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]


def ops_for(device):
    if device == "cpu":
        return kernel_refs
    from lily_b200.csrc import ops
    return ops


def context(device, dtype, page=16, positions=1024):
    return BuildContext(device=torch.device(device), dtype=dtype, ops=ops_for(device), page_size=page, max_position=positions)


def loader(w, device, dtype):
    return lambda name: w[name].to(device=device, dtype=dtype)


def i32(values, device):
    return torch.tensor(values, dtype=torch.int32, device=device)


def dtypes_of(device):
    return [torch.float32] if device == "cpu" else [torch.float32, torch.bfloat16]


def rounded(x, dtype):
    return x.to(dtype).float()


def cache_layer(spec_row, pages, page, kv_heads, dim, vdim, dtype, device):
    shape = (pages + 1, page * spec_row) if kv_heads is None else \
        ((pages + 1, 2, kv_heads, page, dim) if dim == vdim else (pages + 1, kv_heads * page * (dim + vdim)))
    return torch.full(shape, 3.0, dtype=dtype, device=device)                   # what was never written would show


def run_mixers(parts, xs, cuts, device, dtype, page, cache):
    """The parts one after another over one layer of the cache (the first writes it), each on inputs of its own, the sequence
    cut into ``cuts``; pages in a scrambled order.  Returns one output a part."""
    t = xs[0].shape[0]
    pages = -(-t // page)
    order = (torch.randperm(pages, generator=torch.Generator().manual_seed(1)) + 1).tolist()
    outs, done = [[] for _ in parts], 0
    space = Workspace(torch.device(device))
    for n in cuts:
        batch = build_step_batch([StepEntry(1, [0] * n, [])], [done], [[order[:-(-(done + n) // page)]]], device, workspace=space)
        for k, part in enumerate(parts):
            x = xs[k][done:done + n].to(device=device, dtype=dtype).contiguous()
            y = part.forward(x, batch, LayerCache(0, cache), None, write_cache=k == 0)
            outs[k].append((y.sum(0) if y.dim() == 3 else y).float().cpu())
        done += n
    assert done == t
    return [torch.cat(o) for o in outs]


CUTS = ([230], [120] + [1] * 40 + [70], [7, 2, 41, 2, 1, 1, 64, 3, 109], [130, 100])


# ------------------------------------------------------------------ windowed attention, its own keys and another layer's

def attention_weights(g, width, c, own=True):
    n = lambda *shape: torch.randn(*shape, generator=g)
    h, kv, d, dv = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    w = {"p.q": n(h * d, width) / math.sqrt(width), "p.g": 2 * n(h, width) / math.sqrt(width), "p.o": n(width, h * dv) / math.sqrt(h * dv)}
    if own:
        w.update({"p.k": n(kv * d, width) / math.sqrt(width), "p.v": n(kv * dv, width) / math.sqrt(width)})
    return w


def attention_part(c, width, eps, w, device, dtype, page, own=True):
    rope = RopeSpec(c["dim"], c["rot"]["dims"], c["rot"]["base"], interleaved=True, exact_frequencies=True)
    part = build_part("mixer", AttentionSpec(width, c["heads"], c["kv_heads"], c["dim"], qk_norm=True, qk_gain=False, norm_eps=eps,
                                             window=c["mask"]["size"], scale=c["scale"], position=rope, v_head_dim=c["vdim"], head_gate=True,
                                             own_kv=own, names=tuple((r, r) for r in "qkvog")), "p", context(device, dtype, page))
    assert {k: tuple(s.shape) for k, s in part.tensors().items()} == {k: tuple(v.shape) for k, v in w.items()}
    part.load(loader(w, device, dtype))
    return part


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("heads,kv_heads,d,dv,dims", [(3, 1, 12, 12, 12), (4, 2, 64, 64, 64), (8, 2, 64, 64, 32), (2, 2, 128, 128, 128),
                                                      (5, 5, 20, 7, 8), (20, 1, 64, 64, 64), (2, 1, 6, 40, 6)])
@pytest.mark.parametrize("window,other,page", [(40, 17, 16), (16, 90, 64), (1, 64, 16)])
def test_windowed_attention_with_keys_that_stand_out(device, heads, kv_heads, d, dv, dims, window, other, page):
    """Positions at page borders and elsewhere get inputs that later queries answer to as long as they see them, so a window
    that is one token off changes rows outright; a second mixer with a window of its own (narrower or wider) reads the
    same keys.  Whole, decoded and in portions, on the CUDA-core and both tensor-core kernels."""
    g = torch.Generator().manual_seed(d + heads)
    t, width, eps = 230, 40, 1e-5
    c = {"heads": heads, "kv_heads": kv_heads, "dim": d, "vdim": dv, "scale": 6.0 / d, "mask": {"size": window}, "rot": {"dims": dims, "base": 500.0}}
    c2 = dict(c, mask={"size": other}, scale=4.0 / d)
    w, w2 = attention_weights(g, width, c), attention_weights(g, width, c2, own=False)
    h, h2 = torch.randn(t, width, generator=g), torch.randn(t, width, generator=g)
    probe = torch.randn(width, generator=g)
    for m in (15, 16, 63, 64, 101, 150):
        h[m] = 3.0 * probe
    for dtype in dtypes_of(device):
        wr, wr2 = ({k: rounded(v, dtype) for k, v in x.items()} for x in (w, w2))
        with pt.precision(torch.float64):
            pos = torch.arange(t)
            want, kept = pt.attention_mixer(rounded(h, dtype).double(), wr, "p", c, eps, pos)
            want2, _ = pt.attention_mixer(rounded(h2, dtype).double(), wr2, "p", c2, eps, pos, kept)
        parts = [attention_part(c, width, eps, w, device, dtype, page), attention_part(c2, width, eps, w2, device, dtype, page, own=False)]
        for cuts in CUTS:
            cache = cache_layer(0, -(-t // page), page, kv_heads, d, dv, dtype, device)
            got, got2 = run_mixers(parts, [h, h2], cuts, device, dtype, page, cache)
            tol = 5e-5 if dtype == torch.float32 else 4e-2
            assert float((got - want.float()).abs().max()) < tol * max(1.0, float(want.abs().max())), (dtype, cuts[:3])
            assert float((got2 - want2.float()).abs().max()) < tol * max(1.0, float(want2.abs().max())), (dtype, cuts[:3], "reader")


def test_what_a_window_and_a_gate_do():
    """The plain functions say what the construction above is for: a window one token off, a gate left out, a rotation of
    halves and a norm left out each move the outputs by far more than the comparison allows."""
    g = torch.Generator().manual_seed(5)
    c = {"heads": 2, "kv_heads": 1, "dim": 12, "vdim": 12, "scale": 0.5, "mask": {"size": 16}, "rot": {"dims": 12, "base": 500.0}}
    w = attention_weights(g, 40, c)
    h = torch.randn(120, 40, generator=g)
    h[31] = 3.0 * torch.randn(40, generator=g)
    pos = torch.arange(120)
    want, (k, v) = pt.attention_mixer(h, w, "p", c, 1e-5, pos)
    for size in (15, 17):
        assert float((pt.attention_mixer(h, w, "p", dict(c, mask={"size": size}), 1e-5, pos)[0] - want).abs().max()) > 0.05 * float(want.abs().max())
    ungated, _ = pt.attention_mixer(h, dict(w, **{"p.g": torch.full((2, 40), 0.0)}), "p", c, 1e-5, pos)
    assert float((ungated - want).abs().max()) > 0.1 * float(want.abs().max())
    raw = (h @ w["p.k"].t()).view(120, 1, 12)
    for keys in (pt.unit_rms(pt.rotate_halves(raw, pos, c["rot"]), 1e-5), pt.rotate_neighbours(raw, pos, c["rot"])):
        assert float((pt.attention_mixer(h, w, "p", c, 1e-5, pos, (keys, v))[0] - want).abs().max()) > 0.05 * float(want.abs().max())
    # the norm takes all of a head, so it may stand on either side of the rotation
    assert torch.allclose(pt.rotate_neighbours(pt.unit_rms(raw, 1e-5), pos, c["rot"]), k, atol=1e-5)


# ------------------------------------------------------------------ latent attention with a sink a head

def latent_weights(g, width, c):
    n = lambda *shape: torch.randn(*shape, generator=g)
    heads, d, rot, dv, rank = (c[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    return {"p.q": n(heads * (d + rot), width) / math.sqrt(width), "p.dkv": n(rank + rot, width) / math.sqrt(width), "p.dkv.norm": 1 + 0.2 * n(rank),
            "p.uk": n(heads * d, rank) / math.sqrt(rank), "p.uv": n(heads * dv, rank) / math.sqrt(rank), "p.sink": 1.0 + 2.0 * n(heads),
            "p.o": n(width, heads * dv) / math.sqrt(heads * dv)}


def latent_part(c, width, eps, w, device, dtype, page):
    rope = RopeSpec(c["rot_dim"], c["rot"]["dims"], c["rot"]["base"], exact_frequencies=True)
    part = build_part("mixer", LatentAttentionSpec(width, c["heads"], c["dim"], c["rot_dim"], c["vdim"], 0, c["kv_rank"], c["scale"], eps, position=rope,
                                                   out_gate=False, sink=True), "p", context(device, dtype, page))
    assert {k: tuple(s.shape) for k, s in part.tensors().items()} == {k: tuple(v.shape) for k, v in w.items()}
    part.load(loader(w, device, dtype))
    return part


LATENT_SIZES = [(3, 8, 4, 12, 24), (2, 32, 16, 32, 128), (1, 16, 2, 5, 33), (40, 16, 64, 16, 512), (16, 8, 8, 8, 264), (130, 8, 16, 8, 48), (6, 20, 8, 24, 40)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("heads,d,rot,dv,rank", LATENT_SIZES)
@pytest.mark.parametrize("page,scale", [(16, 4.0), (64, 0.5)])
def test_latent_attention_with_sinks(device, heads, d, rot, dv, rank, page, scale):
    """Sharp scores with positions that stand out, and flat ones of which the sinks take a good part: whole, decoded and in
    portions on the CUDA-core, mma.sync and tcgen05 kernels."""
    g = torch.Generator().manual_seed(rank + d)
    t, width, eps = 230, 40, 1e-5
    c = {"heads": heads, "dim": d, "rot_dim": rot, "vdim": dv, "kv_rank": rank, "scale": scale / math.sqrt(d + rot), "rot": {"dims": rot, "base": 50.0}}
    w = latent_weights(g, width, c)
    h = torch.randn(t, width, generator=g)
    probe = torch.randn(width, generator=g)
    for m in (0, 15, 16, 63, 64, 101):
        h[m] = 3.0 * probe
    for dtype in dtypes_of(device):
        wr = {k: rounded(v, dtype) for k, v in w.items()}
        with pt.precision(torch.float64):
            want = pt.latent_attention_mixer(rounded(h, dtype).double(), wr, "p", c, eps, torch.arange(t)).float()
        part = latent_part(c, width, eps, w, device, dtype, page)
        for cuts in CUTS:
            got, = run_mixers([part], [h], cuts, device, dtype, page, cache_layer(rank + rot, -(-t // page), page, None, 0, 0, dtype, device))
            tol = 5e-5 if dtype == torch.float32 else 6e-2
            assert float((got - want).abs().max()) < tol * max(1.0, float(want.abs().max())), (dtype, cuts[:3])
    if device == "cuda":
        assert ops_for(device).latent_attention_status() == 0


def test_a_sink_left_out_or_counted_twice_shows():
    g = torch.Generator().manual_seed(6)
    s, sink = torch.randn(5, 9, generator=g), torch.tensor(1.3)
    p = pt.softmax_with_sink(s, sink)
    assert torch.allclose(p.sum(-1), 1.0 - torch.exp(sink) / (torch.exp(sink) + torch.exp(s).sum(-1)), atol=1e-6)
    for other in (torch.softmax(s, -1), pt.softmax_with_sink(s, sink + math.log(2.0)), pt.softmax_with_sink(s, 0.1 * sink)):
        assert float((other - p).abs().max()) > 0.01


def rows_attention(q, keys, first, rank, scale, sinks):
    s = torch.einsum("thd,jd->thj", q, keys) * scale
    seen = torch.arange(keys.shape[0])[None, None, :] <= torch.arange(first, first + q.shape[0])[:, None, None]
    s = torch.cat([s.masked_fill(~seen, float("-inf")), sinks[None, :, None].expand(q.shape[0], -1, 1)], -1)
    return torch.softmax(s, -1)[..., :-1] @ keys[:, :rank]


@pytest.mark.gpu
@pytest.mark.parametrize("heads,row,rank", [(5, 64, 64), (32, 576, 512), (6, 272, 264), (130, 64, 48), (7, 30, 17)])
@pytest.mark.parametrize("strength", [-60.0, 0.0, 3.0, 60.0])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sinks_over_cached_rows(heads, row, rank, strength, dtype):
    """Sinks far below every score (nothing changes), among them, and far above (the outputs vanish, without a NaN): decode in
    one and several key ranges, some without a key, and portions, on every kernel the sizes get."""
    from lily_b200.csrc import ops
    page = 64
    g = torch.Generator().manual_seed(row + 1)
    lens = [1, 128, 129, 700]
    pages = [-(-n // page) for n in lens]
    order = (torch.randperm(sum(pages), generator=g) + 1).tolist()
    table = torch.zeros(len(lens), max(pages), dtype=torch.int32)
    at = 0
    for r, n in enumerate(pages):
        table[r, :n] = i32(order[at:at + n], "cpu")
        at += n
    cache = (torch.randn(sum(pages) + 1, page * row, generator=g) * 0.7).to(device="cuda", dtype=dtype)
    held = cache.float().cpu().view(-1, page, row)
    keys = [torch.stack([held[int(table[r, j // page]), j % page] for j in range(n)]) for r, n in enumerate(lens)]
    sinks = strength + torch.randn(heads, generator=g)
    scale = 3.0 / math.sqrt(row)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    q = torch.randn(len(lens), heads * row, generator=g).to(device="cuda", dtype=dtype)
    want = torch.cat([rows_attention(q[r:r + 1].float().cpu().view(1, heads, row), keys[r], n - 1, rank, scale, sinks) for r, n in enumerate(lens)])
    plan = ops.plan_decode_attention(dtype, len(lens), heads, 1, row, max(lens), dv=rank, values_in_keys=True, page_size=page)
    for splits in sorted({1, 2, 5, 12, plan.splits}):
        out = torch.full((len(lens), heads * rank), 7.0, device="cuda", dtype=dtype)
        scratch = torch.empty(max(1, ops.decode_scratch_floats(len(lens), heads, rank, splits)), device="cuda")
        ops.attention_decode(q, cache, table.cuda(), i32(lens, "cuda"), out, scratch, splits, heads, 1, row, page, scale, None, dv=rank,
                             values_in_keys=True, sinks=sinks.cuda())
        assert float((out.float().cpu().view(len(lens), heads, rank) - want).abs().max()) < tol * max(1.0, float(want.abs().max())), splits
    new, prefix = [1, 28, 65, 200], [0, 100, 64, 500]
    q = torch.randn(sum(new), heads * row, generator=g).to(device="cuda", dtype=dtype)
    out = torch.full((sum(new), heads * rank), 7.0, device="cuda", dtype=dtype)
    tile = ops.prefill_tile_rows(dtype, row, page, sum(new), dv=rank, values_in_keys=True, heads=heads)
    cu = [0, 1, 29, 94, 294]
    tr, ts = ops.prefill_tiles(prefix, new, 0, tile, "cuda")
    ops.attention_prefill(q, cache, table.cuda(), i32(cu, "cuda"), i32(prefix, "cuda"), tr, ts, out, heads, 1, row, page, scale, None, tile_rows=tile,
                          dv=rank, values_in_keys=True, sinks=sinks.cuda())
    for r in range(4):
        want = rows_attention(q[cu[r]:cu[r + 1]].float().cpu().view(-1, heads, row), keys[r], prefix[r], rank, scale, sinks)
        assert float((out[cu[r]:cu[r + 1]].float().cpu().view(-1, heads, rank) - want).abs().max()) < tol * max(1.0, float(want.abs().max())), r
    assert ops.latent_attention_status() == 0


# ------------------------------------------------------------------ the matrix memory

def mlstm_weights(g, width, c, forget=2.0, spread=2.0):
    n = lambda *shape: torch.randn(*shape, generator=g)
    h, d, dv = c["heads"], c["dim"], c["vdim"]
    w = {f"p.{r}": n(h * k, width) / math.sqrt(width) for r, k in (("q", d), ("k", d), ("v", dv), ("g", dv))}
    w.update({"p.i": spread * n(h, width) / math.sqrt(width), "p.f": spread * n(h, width) / math.sqrt(width), "p.i.b": n(h),
              "p.f.b": forget + n(h), "p.norm": 1 + 0.2 * n(h * dv), "p.o": n(width, h * dv) / math.sqrt(h * dv)})
    return w


def mlstm_part(c, width, eps, w, device, dtype):
    part = build_part("mixer", MlstmSpec(width, c["heads"], c["dim"], c["vdim"], c["gate_cap"], eps), "p", context(device, dtype))
    assert {k: tuple(s.shape) for k, s in part.tensors().items()} == {k: tuple(v.shape) for k, v in w.items()}
    part.load(loader(w, device, dtype))
    return part


def run_mlstm(part, seqs, plan, device, dtype, slots=None):
    """Sequences side by side: ``plan`` lists steps of (sequence, tokens); single tokens come first in a step."""
    slots = slots or {k: i + 1 for i, k in enumerate(seqs)}
    state = torch.zeros(max(slots.values()) + 1, *part.state_need().shape, device=device)
    done, outs, space = {k: 0 for k in seqs}, {k: [] for k in seqs}, Workspace(torch.device(device))
    for step in plan:
        entries = [StepEntry(slots[k], [0] * n, []) for k, n in step]
        batch = build_step_batch(entries, [done[k] for k, _ in step], [], device, workspace=space)
        x = torch.cat([seqs[k][done[k]:done[k] + n] for k, n in step]).to(device=device, dtype=dtype).contiguous()
        y = part.forward(x, batch, None, state)
        y = (y.sum(0) if y.dim() == 3 else y).float().cpu()
        for (k, n), rows in zip(step, torch.split(y, [n for _, n in step])):
            outs[k].append(rows)
            done[k] += n
    return {k: torch.cat(o) for k, o in outs.items()}, state


MLSTM_SIZES = [(2, 8, 12, 10.0), (3, 20, 5, 2.0), (1, 64, 64, 15.0), (5, 32, 40, 11.0), (2, 48, 96, 8.0), (1, 256, 128, 15.0), (2, 144, 136, 6.0),
               (1, 7, 33, 20.0), (1, 512, 24, 15.0), (1, 16, 640, 15.0)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("heads,d,dv,cap", MLSTM_SIZES)
@pytest.mark.parametrize("forget,spread", [(4.0, 1.0), (0.0, 6.0)])
def test_matrix_memory(device, heads, d, dv, cap, forget, spread):
    """Long memories and short ones, input gates that pass the running maximum again and again and gates that run into their
    cap: a sequence whole (in chunks side by side in bfloat16), decoded, in portions; two sequences side by side, of which
    one's long portion meets the other's single tokens."""
    g = torch.Generator().manual_seed(d + dv)
    width, eps = 40, 1e-5
    c = {"heads": heads, "dim": d, "vdim": dv, "gate_cap": cap}
    w = mlstm_weights(g, width, c, forget, spread)
    seqs = {"a": torch.randn(330, width, generator=g), "b": torch.randn(150, width, generator=g)}
    for dtype in dtypes_of(device):
        wr = {k: rounded(v, dtype) for k, v in w.items()}
        with pt.precision(torch.float64):
            want = {k: pt.mlstm_mixer(rounded(x, dtype).double(), wr, "p", c, eps).float() for k, x in seqs.items()}
        part = mlstm_part(c, width, eps, w, device, dtype)
        plans = [[[("a", 330)], [("b", 150)]], [[("a", 200)], [("b", 130), ("a", 70)]] + [[("a", 1), ("b", 1)]] * 20 + [[("a", 40)]],
                 [[("a", n)] for n in (7, 2, 41, 65, 1, 128, 2, 64, 20)] + [[("b", 1)]] * 3 + [[("b", 129)], [("b", 18)]],
                 [[("b", 100)], [("b", 1), ("a", 129)], [("b", 1), ("a", 1)], [("b", 48), ("a", 200)]]]
        # a token whose read-out nearly cancels is divided by its small root mean square, which magnifies every rounding: 24 rows
        # in 25 keep the bound, and the others stay near it
        tol = 5e-5 if dtype == torch.float32 else 4e-2
        for i, plan in enumerate(plans):
            got, _ = run_mlstm(part, seqs, plan, device, dtype)
            for k in seqs:
                rows = (got[k] - want[k]).abs().max(-1).values.sort().values / max(1.0, float(want[k].abs().max()))
                assert float(rows[int(0.96 * (len(rows) - 1))]) < tol and float(rows[-1]) < 25 * tol, (dtype, i, k, rows[-8:])


@pytest.mark.parametrize("device", DEVICES)
def test_a_value_written_long_ago(device):
    """The first token's value comes back 400 decoded tokens later: forget gates next to one, one strong input gate."""
    c = {"heads": 1, "dim": 16, "vdim": 16, "gate_cap": 30.0}
    width, t = 24, 420
    g = torch.Generator().manual_seed(9)
    w = mlstm_weights(g, width, c)
    w["p.f.b"], w["p.f"] = torch.tensor([25.0]), torch.zeros(1, width)
    w["p.i"], w["p.i.b"] = torch.zeros(1, width), torch.tensor([-12.0])
    w["p.i"][0, 0] = 5.0
    h = 0.3 * torch.randn(t, width, generator=g)
    h[:, 0] = 0.0
    h[0, 0] = 4.0                                                               # the one token whose input gate opens
    for dtype in dtypes_of(device):
        wr = {k: rounded(v, dtype) for k, v in w.items()}
        with pt.precision(torch.float64):
            want = pt.mlstm_mixer(rounded(h, dtype).double(), wr, "p", c, 1e-6).float()
            lost = rounded(h, dtype).double()
            lost[0, 0] = 0.0
            assert float((pt.mlstm_mixer(lost, wr, "p", c, 1e-6).float() - want)[-1].abs().max()) > 0.1 * float(want[-1].abs().max())
        part = mlstm_part(c, width, 1e-6, w, device, dtype)
        for plan in ([[("a", 20)]] + [[("a", 1)]] * 400, [[("a", t)]], [[("a", 5)], [("a", 300)], [("a", 115)]]):
            got, _ = run_mlstm(part, {"a": h}, plan, device, dtype)
            # every answer is the first value times a sign, but where the query is next to orthogonal to its key
            rows = (got["a"] - want).abs().max(-1).values.sort().values
            assert float(rows[int(0.95 * t)]) < (1e-4 if dtype == torch.float32 else 4e-2) * float(want.abs().max())


@pytest.mark.parametrize("device", DEVICES)
def test_the_scale_starts_at_zero_and_is_carried(device):
    """With input gates far below zero the running maximum stays at what the forget gates leave of its start, zero, and the
    denominator is exp(-m), not |n . q|; the slot carries it from step to step."""
    c = {"heads": 2, "dim": 16, "vdim": 8, "gate_cap": 9.0}
    width = 20
    g = torch.Generator().manual_seed(3)
    w = mlstm_weights(g, width, c)
    w["p.i.b"] = torch.tensor([-8.0, -5.0])
    h = torch.randn(90, width, generator=g)
    part = mlstm_part(c, width, 1e-6, w, device, torch.float32)
    want = pt.mlstm_mixer(h, w, "p", c, 1e-6)
    i, f = pt.mlstm_gates(h, w, "p", 9.0)
    m, low = torch.zeros(2), []
    for t in range(90):
        m = torch.maximum(f[t] + m, i[t])
        low.append(m)
    for plan in ([[("a", 90)]], [[("a", 1)]] * 10 + [[("a", 80)]]):
        got, state = run_mlstm(part, {"a": h}, plan, device, torch.float32)
        assert float((got["a"] - want).abs().max()) < 1e-4 * max(1.0, float(want.abs().max()))
        assert torch.allclose(state[1, part.matrix_floats:part.matrix_floats + 2].cpu(), low[-1], atol=1e-5)
        assert float(state[0].abs().max()) == 0.0


@pytest.mark.gpu
def test_chunks_against_one_piece():
    """The chunk kernels against the token-by-token one on the same bfloat16 rows: outputs, normaliser, scale and the state
    left behind, with two long portions, a short one and single tokens in one step, and a state to start from."""
    from lily_b200.csrc import ops
    g = torch.Generator().manual_seed(1)
    for heads, d, dv in ((2, 64, 64), (3, 32, 200), (1, 256, 512), (2, 16, 8), (1, 208, 40)):
        new = [1, 700, 30, 129, 1]
        n, key, inner = sum(new), heads * d, heads * dv
        width = 2 * key + inner + (-(2 * key + inner)) % 8
        proj = torch.randn(n, width, generator=g).cuda().bfloat16()
        gates = (3.0 * torch.randn(n, 2 * heads, generator=g)).cuda()
        floats = heads * (dv + 1) * d + heads
        start = torch.randn(7, floats + -floats % 4, generator=g).cuda()
        ib, fb = torch.zeros(heads).cuda(), torch.full((heads,), 3.0).cuda()
        cu, slots = i32([0, 1, 701, 731, 860, 861], "cuda"), i32([3, 1, 6, 2, 5], "cuda")
        plan = ops.mlstm_plan(new, torch.bfloat16, heads, d, dv, "cuda")
        assert plan.longs == 2 and plan.num_direct == 3 and plan.items == 8 and plan.tiles == 11 + 3
        room = torch.full((ops.mlstm_workspace_floats(plan, heads, d, dv),), float("nan"), device="cuda")
        got_state, want_state = start.clone(), start.clone()
        args = (0, key, 2 * key, gates, 0, heads, ib, fb, 10.0, d ** -0.5)
        got = ops.mlstm_scan(proj, *args, got_state, cu, slots, 5, heads, d, dv, plan=plan, workspace=room)
        want = ops.mlstm_scan(proj, *args, want_state, cu, slots, 5, heads, d, dv)
        for a, b, tol in zip(got, want, (2e-4, 2e-4, 1e-4)):
            assert float((a - b).abs().max()) < tol * max(1.0, float(b.abs().max())), (heads, d, dv)
        assert float((got_state - want_state).abs().max()) < 2e-4 * float(want_state.abs().max())
        assert torch.equal(got_state[[0, 4]], start[[0, 4]])


def test_plan_of_chunks():
    from lily_b200.csrc import ops
    assert ops.mlstm_plan([64, 1, 3], torch.bfloat16, 4, 64, 64, "cpu") is None
    assert ops.mlstm_plan([500], torch.float32, 4, 64, 64, "cpu") is None and ops.mlstm_plan([500], torch.bfloat16, 4, 24, 64, "cpu") is None
    plan = ops.mlstm_plan([65, 1, 300], torch.bfloat16, 4, 64, 64, "cpu")
    assert plan.item_req.tolist() == [0, 2, 2, 2] and plan.item_start.tolist() == [0, 0, 128, 256] and plan.item_len.tolist() == [65, 128, 128, 44]
    assert plan.long_req.tolist() == [0, 2] and plan.long_first.tolist() == [0, 1] and plan.long_count.tolist() == [1, 3] and plan.direct.tolist() == [1]
    assert plan.tile_item.tolist() == [0, 0, 1, 1, 2, 2, 3] and plan.tile_start.tolist() == [0, 64, 0, 64, 0, 64, 0] and plan.tokens == 366
    long = ops.mlstm_plan([30000], torch.bfloat16, 8, 256, 512, "cpu")              # longer chunks, so that the workspace stays bounded
    assert int(long.item_len[0]) > 128 and 4 * ops.mlstm_workspace_floats(long, 8, 256, 512) < 1.1 * ops.SCAN_WORKSPACE + (1 << 24)


# ------------------------------------------------------------------ experts

class _Batch:
    def __init__(self, device):
        self.workspace = Workspace(torch.device(device))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("experts,top,groups,keep,ff,width,shared", [(6, 2, 3, 2, 24, 40, 56), (15, 4, 5, 2, 56, 72, None), (4, 1, 2, 1, 10, 33, 7),
                                                                     (5, 2, 5, 3, 16, 48, 24), (8, 8, 1, 1, 7, 20, 9), (256, 8, 8, 4, 8, 64, 64),
                                                                     (96, 6, 48, 5, 16, 256, 256), (9, 4, None, 1, 32, 64, 40)])
def test_experts_chosen_within_groups(device, experts, top, groups, keep, ff, width, shared):
    """Ungated experts; a group whose best expert is the best of all but whose second is poor is left out; choice scores below
    zero in a kept group come before better ones outside; weights without the correction; one token, a few and many."""
    g = torch.Generator().manual_seed(experts * 10 + top)
    n = lambda *shape: torch.randn(*shape, generator=g)
    w = {"p.router": 2 * n(experts, width) / math.sqrt(width), "p.correction": 0.5 * n(experts) - 0.8}
    for name, f in [(f"e{e}", ff) for e in range(experts)] + ([("shared", shared)] if shared else []):
        w.update({f"p.{name}.up": 2 * n(f, width) / math.sqrt(width), f"p.{name}.down": n(width, f) / math.sqrt(f)})
    c = {"router": {"experts": experts, "top": top}}
    if groups:
        c["router"]["groups"] = {"count": groups, "keep": keep}
    if shared:
        w["p.shared.sg"] = n(1, width) / math.sqrt(width)
        c["shared"] = {"ff": shared}
    h = n(77, width)
    spec = RoutedExpertsSpec(width, ff, experts, 0, top, scores="sigmoid", activation="relu2", shared_size=shared or 0, groups=groups or 0,
                             keep_groups=keep if groups else 0)
    for dtype in dtypes_of(device):
        part = build_part("feed_forward", spec, "p", context(device, dtype))
        assert {k: tuple(s.shape) for k, s in part.tensors().items()} == {k: tuple(v.shape) for k, v in w.items()}
        part.load(loader(w, device, dtype))
        wr = {k: rounded(v, dtype) for k, v in w.items()}
        want = pt.moe_ff(rounded(h, dtype), wr, "p", c)
        for rows in (slice(0, 77), slice(5, 6), slice(40, 49)):
            y = part.forward(h[rows].to(device=device, dtype=dtype).contiguous(), _Batch(device))
            assert y.dtype == torch.float32 and y.shape[0] == 1
            tol = 2e-5 if dtype == torch.float32 else 2e-2
            assert float((y[0].cpu() - want[rows]).abs().max()) < tol * max(1.0, float(want.abs().max())), (dtype, rows)
        ops = ops_for(device)
        big = n(1100, width)                                                  # several tokens share a block on the GPU
        how = {"groups": groups, "keep_groups": keep} if groups else {}
        routing = ops.moe_route(big.to(device=device, dtype=dtype), part.router, part.correction, top, experts, scores="sigmoid",
                                shared_gate=bool(shared), outputs=experts, **how)
        with pt.precision(torch.float64):
            chosen, weights = pt.route(rounded(big, dtype), wr, "p", c["router"])
        mine = routing.chosen.cpu().long()
        same = (mine.sort(-1).values == chosen.sort(-1).values).all(-1)       # two scores may be next to equal
        assert int((~same).sum()) <= 2
        order = mine.argsort(-1)
        diff = (routing.weights.cpu().gather(1, order) - weights.float().gather(1, chosen.argsort(-1)))[same]
        assert float(diff.abs().max()) < 1e-5


@pytest.mark.parametrize("device", DEVICES)
def test_a_group_is_scored_by_two(device):
    """Scores set by hand (router logits through one input column): group 0 has the best expert and a poor second, group 1 two
    good ones, group 2 the second best and a fair one; all choice scores are negative after the correction."""
    ops = ops_for(device)
    s = torch.tensor([0.95, 0.05, 0.70, 0.69, 0.90, 0.30])
    z = torch.log(s / (1 - s))
    h = torch.ones(1, 8)
    router = torch.zeros(8, 8)
    router[:6] = z[:, None] / 8
    corr = torch.full((6,), -2.0)
    for keep, top, want in ((1, 1, {2}), (1, 2, {2, 3}), (2, 1, {4}), (2, 3, {4, 2, 3}), (3, 2, {0, 4})):
        r = ops.moe_route(h.to(device), router.to(device), corr.to(device), top, 6, scores="sigmoid", outputs=6, groups=3, keep_groups=keep)
        assert set(r.chosen[0].tolist()) == want, (keep, top)
        picked = torch.tensor([float(s[e]) for e in r.chosen[0].tolist()])
        assert torch.allclose(r.weights[0].cpu(), picked / picked.sum(), atol=1e-6)
    plain, _ = pt.route(h, {"p.router": router[:6], "p.correction": corr}, "p", {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}})
    assert set(plain[0].tolist()) == {2, 3}


# ------------------------------------------------------------------ norms that squash, the gate a head

@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("tokens", [1, 9, 1030])
@pytest.mark.parametrize("hidden", [48, 321, 1024])
def test_squashing_norms_on_both_sides(device, tokens, hidden):
    """``x + D_b(y)`` into the float32 stream and ``D_a`` of the new rows in one pass: deltas whole, as partial sums and as one
    float32 plane, inputs from next to zero to saturation, gathered rows, and beside norms of the other kind."""
    ops = ops_for(device)
    g = torch.Generator().manual_seed(hidden)
    spread = torch.exp(3.0 * torch.randn(tokens, 1, generator=g) - 2.0)
    resid = torch.randn(tokens, hidden, generator=g) * 3 * spread
    y, parts = torch.randn(tokens, hidden, generator=g) * spread, torch.randn(3, tokens, hidden, generator=g)
    w = {"a": 1 + 0.3 * torch.randn(hidden, generator=g), "a.alpha": torch.tensor(0.7), "a.b": 0.3 * torch.randn(hidden, generator=g),
         "b": 1 + 0.3 * torch.randn(hidden, generator=g), "b.alpha": torch.tensor(1.6), "b.b": 0.3 * torch.randn(hidden, generator=g)}
    for dtype in dtypes_of(device):
        ctx = context(device, dtype)
        ahead, after = (build_part("norm", DynamicTanhSpec(hidden), p, ctx) for p in "ab")
        assert {k: tuple(t.shape) for n in (ahead, after) for k, t in n.tensors().items()} == {k: tuple(v.shape) for k, v in w.items()}
        for n in (ahead, after):
            n.load(loader(w, device, dtype))
        wr = {k: rounded(v, dtype) for k, v in w.items()}
        close = lambda got, want, tol: float(((got.float().cpu() - want).abs() / (want.abs() + 1.0)).max()) < tol
        near = 1e-5 if dtype == torch.float32 else 1e-2
        stream = resid.clone().to(device)
        assert close(ahead.forward(stream), pt.squash(resid, wr, "a"), near) and torch.equal(stream.cpu(), resid)
        for delta, value in ((y.to(device=device, dtype=dtype), rounded(y, dtype)), (parts.to(device), parts.sum(0)), (parts[:1].to(device), parts[0])):
            stream = resid.clone().to(device)
            want = resid + pt.squash(value, wr, "b")
            assert close(ahead.forward(stream, after.behind()(delta)), pt.squash(want, wr, "a"), near)
            assert close(stream, want, 2e-6)
            rows = i32([tokens - 1, 0], device)
            got = ahead.forward(stream, after.behind(0.5)(delta), rows=rows)
            assert close(got, pt.squash(want + 0.5 * pt.squash(value, wr, "b"), wr, "a")[rows.cpu().long()], near) and close(stream, want, 2e-6)
            assert close(enter_stream(ops, stream, after.behind()(delta), dtype), want + pt.squash(value, wr, "b"), near)
        # beside the other kinds: a plain delta, several, a normalised one; and a squashed one ahead of an RMS norm
        stream = resid.clone().to(device)
        assert close(ahead.forward(stream, y.to(device)), pt.squash(resid + y, wr, "a"), near)
        stream = resid.clone().to(device)
        assert close(ahead.forward(stream, (y.to(device), None, parts.to(device)), delta_bias=torch.ones(hidden, device=device)),
                     pt.squash(resid + y + parts.sum(0) + 1.0, wr, "a"), near)
        gain = torch.full((hidden,), 0.4, device=device)
        stream = resid.clone().to(device)
        assert close(ahead.forward(stream, NormedDelta(y.to(device), gain, 1e-5)), pt.squash(resid + 0.4 * pt.unit_rms(y, 1e-5), wr, "a"), near)
        rms = build_part("norm", RMSNormSpec(hidden, 1e-5), "r", ctx)
        rms.load(lambda name: torch.ones(hidden, device=device))
        stream = resid.clone().to(device)
        delta = TanhDelta(y.to(device), *after.norm)
        assert close(rms.forward(stream, delta), pt.unit_rms(resid + pt.squash(y, wr, "b"), 1e-5), near)


@pytest.mark.gpu
def test_the_squash_over_its_whole_range():
    """Against tanh in float64, from 1e-6 to saturation: a few units of float32 in either form."""
    from lily_b200.csrc import ops
    z = torch.cat([torch.logspace(-6, 2, 6000), torch.linspace(0.2, 0.3, 2192)])
    z = torch.cat([z, -z]).view(1, -1)
    one, nil = torch.ones(z.shape[1], device="cuda"), torch.zeros(z.shape[1], device="cuda")
    want = torch.tanh(z.double())
    for dtype in (torch.float32, torch.bfloat16):
        stream = torch.zeros_like(z).cuda()
        ops.add_tanh_norm(stream, z.cuda(), (1.0, one, nil), 1.0, (1.0, one, nil), dtype)
        assert float(((stream.cpu().double() - want).abs() / want.abs()).max()) < (1e-6 if dtype == torch.float32 else 4e-6)


@pytest.mark.parametrize("device", DEVICES)
def test_a_gate_a_head(device):
    ops = ops_for(device)
    g = torch.Generator().manual_seed(2)
    for t, heads, dv, g0, ld in ((70, 3, 20, 5, 8), (1, 8, 128, 64, 72), (9, 1, 64, 0, 1), (33, 6, 7, 11, 24)):
        out = torch.randn(t, heads * dv, generator=g)
        for gate in (2 * torch.randn(t, ld, generator=g), torch.randn(3, t, ld, generator=g)):
            for dtype in dtypes_of(device):
                x, z = out.to(device=device, dtype=dtype), gate.to(device=device, dtype=dtype if gate.dim() == 2 else torch.float32)
                total = z.float().cpu() if gate.dim() == 2 else gate.sum(0)
                want = (rounded(out, dtype).view(t, heads, dv) * torch.sigmoid(total[:, g0:g0 + heads])[:, :, None]).view(t, -1)
                got = ops.sigmoid_head_gate(x, z, g0, heads)
                assert got.data_ptr() == x.data_ptr()
                assert float((got.float().cpu() - want).abs().max()) < (1e-5 if dtype == torch.float32 else 2e-2) * float(want.abs().max())
