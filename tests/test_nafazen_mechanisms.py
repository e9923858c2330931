"""Each mechanism of the Nafazen decoder alone: parts and kernel faces (CUDA on the GPU, their plain statements on the CPU)
against the functions of ``plain_nafazen``, with inputs made so that a fault shows: a cached position that stands out far
back and at page borders, rows read from another layer's cache, scores that the weight on an expert's input must not be
confused with, activation values on both sides of zero and near it, sizes that are not powers of two."""

import math

import pytest
import torch

import kernel_refs
import plain_nafazen as pn
from lily_b200.config.model_config import RopeScaling
from lily_b200.engine.batch import StepEntry, Workspace, build_step_batch
from lily_b200.parts.attention import LayerCache
from lily_b200.parts.base import BuildContext, build_part
from lily_b200.parts.experts import RoutedExpertsSpec
from lily_b200.parts.latent_attention import LatentAttentionSpec
from lily_b200.parts.mlp import DenseMLPSpec
from lily_b200.parts.norm import NormedDelta, RMSNormSpec, enter_stream
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


# ------------------------------------------------------------------ rotation

@pytest.mark.parametrize("scaling", [None, {"factor": 2.0, "original": 300, "fast": 16.0, "slow": 1.0},
                                     {"factor": 8.0, "original": 40, "fast": 4.0, "slow": 0.25}, {"factor": 1.0, "original": 64, "fast": 8.0, "slow": 2.0},
                                     {"factor": 0.5, "original": 4096, "fast": 32.0, "slow": 32.0}])
@pytest.mark.parametrize("dims,base", [(12, 1000.0), (2, 10.0), (64, 300000.0)])
def test_frequencies_and_stretch(scaling, dims, base):
    """Bands that keep their frequency, are slowed, and lie on the ramp; a ramp of no width; the stretch on both tables."""
    spec = RopeSpec(dims, dims, base, RopeScaling.yarn(scaling, "rot.scaling"), interleaved=True, exact_frequencies=True)
    table = build_part("position", spec, "p", context("cpu", torch.float32, positions=700))
    rot = {"dims": dims, "base": base}
    if scaling:
        rot["scaling"] = scaling
    f, stretch = pn.frequencies(rot)
    ang = torch.arange(700, dtype=torch.float32)[:, None] * f[None, :]
    cos, sin = table.tables()
    assert float((cos - ang.cos() * stretch).abs().max()) < 2e-6 * stretch and float((sin - ang.sin() * stretch).abs().max()) < 2e-6 * stretch


def test_the_scaling_changes_what_it_should():
    """The plain function says what the construction is for: fast pairs keep their frequency, slow ones are divided, some
    lie between, and the stretch is not one."""
    plain, _ = pn.frequencies({"dims": 64, "base": 10000.0})
    f, stretch = pn.frequencies({"dims": 64, "base": 10000.0, "scaling": {"factor": 4.0, "original": 512, "fast": 16.0, "slow": 1.0}})
    ratio = f / plain
    assert float(ratio[0]) == 1.0 and abs(float(ratio[-1]) - 0.25) < 1e-6 and bool(((ratio > 0.26) & (ratio < 0.99)).any())
    assert abs(stretch - (0.1 * math.log(4.0) + 1.0)) < 1e-12


# ------------------------------------------------------------------ the attention, its own rows and another layer's

def attention_weights(g, width, c, own=True):
    n = lambda *shape: torch.randn(*shape, generator=g)
    heads, d, rot, dv, q_rank, rank = (c[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
    w = {"p.dq": n(q_rank, width) / math.sqrt(width), "p.dq.norm": 1 + 0.2 * n(q_rank),
         "p.uq": n(heads * (d + rot), q_rank) / math.sqrt(q_rank), "p.uk": n(heads * d, rank) / math.sqrt(rank),
         "p.uv": n(heads * dv, rank) / math.sqrt(rank), "p.o": n(width, heads * dv) / math.sqrt(heads * dv)}
    if own:
        w.update({"p.dkv": n(rank + rot, width) / math.sqrt(width), "p.dkv.norm": 1 + 0.2 * n(rank)})
    return w


def mixer_part(c, width, eps, w, device, dtype, page, own=True):
    rot = c["rot"]
    rope = RopeSpec(c["rot_dim"], rot["dims"], rot["base"], RopeScaling.yarn(rot.get("scaling"), "rot.scaling"), interleaved=True,
                    exact_frequencies=True)
    part = build_part("mixer", LatentAttentionSpec(width, c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["q_rank"], c["kv_rank"],
                                                   c["scale"], eps, position=rope, out_gate=False, own_kv=own), "p", context(device, dtype, page))
    assert set(part.tensors()) == set(w)
    part.load(loader(w, device, dtype))
    return part


def run_mixers(parts, xs, cuts, device, dtype, page, row):
    """The parts one after another over one cached row a position (the first writes it), each on inputs of its own, with
    the sequence cut into ``cuts``; pages in a scrambled order.  Returns one output a part."""
    t = xs[0].shape[0]
    pages = -(-t // page)
    order = (torch.randperm(pages, generator=torch.Generator().manual_seed(1)) + 1).tolist()
    cache = torch.full((pages + 1, page * row), 3.0, dtype=dtype, device=device)      # what was never written would show
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


SIZES = [(3, 8, 4, 12, 20, 24), (2, 32, 16, 32, 48, 128), (1, 16, 2, 5, 9, 33), (5, 12, 32, 8, 16, 72), (40, 16, 64, 16, 32, 512),
         (16, 8, 8, 8, 24, 264), (4, 32, 16, 24, 32, 64), (130, 8, 16, 8, 16, 48), (7, 8, 64, 8, 40, 448)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("heads,d,rot,dv,q_rank,rank", SIZES)
@pytest.mark.parametrize("yarn,page", [(None, 16), ({"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}, 64)])
def test_one_position_that_stands_out(device, heads, d, rot, dv, q_rank, rank, yarn, page):
    """Positions at page borders and far back get inputs that every later query answers to, so a row that is lost, written
    to another place or turned by another angle changes the outputs outright.  A second mixer of other head counts and
    head sizes reads the same rows.  Whole, decoded, and in portions."""
    g = torch.Generator().manual_seed(rank + d)
    t, width, eps = 230, 40, 1e-5
    c = {"heads": heads, "dim": d, "rot_dim": rot, "vdim": dv, "q_rank": q_rank, "kv_rank": rank, "scale": 4.0 / math.sqrt(d + rot),
         "rot": {"dims": rot, "base": 50.0}}
    if yarn:
        c["rot"]["scaling"] = yarn
    c2 = dict(c, heads=3, dim=d + 2, vdim=dv + 1, q_rank=q_rank + 3, scale=3.0 / math.sqrt(d + rot))
    w, w2 = attention_weights(g, width, c), attention_weights(g, width, c2, own=False)
    h, h2 = torch.randn(t, width, generator=g), torch.randn(t, width, generator=g)
    probe = torch.randn(width, generator=g)
    for m in (15, 16, 63, 64, 101):
        h[m] = 3.0 * probe
    for dtype in dtypes_of(device):
        wr, wr2 = ({k: rounded(v, dtype) for k, v in x.items()} for x in (w, w2))
        with pn.precision(torch.float64):
            pos = torch.arange(t)
            want, rows = pn.latent_attention_mixer(rounded(h, dtype).double(), wr, "p", c, eps, pos)
            want2, _ = pn.latent_attention_mixer(rounded(h2, dtype).double(), wr2, "p", c2, eps, pos, rows)
        parts = [mixer_part(c, width, eps, w, device, dtype, page), mixer_part(c2, width, eps, w2, device, dtype, page, own=False)]
        for cuts in ([t], [120] + [1] * 40 + [70], [7, 2, 41, 2, 1, 1, 64, 3, 109], [130, 100]):
            got, got2 = run_mixers(parts, [h, h2], cuts, device, dtype, page, rank + rot)
            tol = 5e-5 if dtype == torch.float32 else 6e-2
            assert float((got - want.float()).abs().max()) < tol * max(1.0, float(want.abs().max())), (dtype, cuts[:3])
            assert float((got2 - want2.float()).abs().max()) < tol * max(1.0, float(want2.abs().max())), (dtype, cuts[:3], "reader")
    if device == "cuda":
        assert ops_for(device).latent_attention_status() == 0


def test_rows_that_stand_out_are_seen():
    """The plain functions say what the construction above is for: dropping one such row, or turning it by the angle of
    the position beside it, moves the outputs by far more than the comparison allows."""
    g = torch.Generator().manual_seed(5)
    c = {"heads": 2, "dim": 8, "rot_dim": 8, "vdim": 8, "q_rank": 16, "kv_rank": 24, "scale": 1.0, "rot": {"dims": 8, "base": 50.0}}
    w = attention_weights(g, 40, c)
    h = torch.randn(120, 40, generator=g)
    h[16] = 3.0 * torch.randn(40, generator=g)
    pos = torch.arange(120)
    want, (latent, turned) = pn.latent_attention_mixer(h, w, "p", c, 1e-5, pos)
    lost = (latent.clone(), turned.clone())
    lost[0][16] = 0.0
    beside = (latent, turned.clone())
    beside[1][16] = pn.rotate_pairs((h[16:17] @ w["p.dkv"].t())[:, 24:], torch.tensor([17]), c["rot"])[0]
    for rows in (lost, beside):
        other, _ = pn.latent_attention_mixer(h, w, "p", c, 1e-5, pos, rows)
        assert float((other - want)[20:].abs().max()) > 0.1 * float(want.abs().max())


def cached_rows(g, lens, page, row, dtype, scale=0.7):
    """A cache of random rows for sequences of these lengths, pages handed out in a scrambled order; the rows of each."""
    pages = [-(-n // page) for n in lens]
    order = (torch.randperm(sum(pages), generator=g) + 1).tolist()
    table = torch.zeros(len(lens), max(pages), dtype=torch.int32)
    at = 0
    for r, n in enumerate(pages):
        table[r, :n] = torch.tensor(order[at:at + n], dtype=torch.int32)
        at += n
    cache = (torch.randn(sum(pages) + 1, page * row, generator=g) * scale).to(device="cuda", dtype=dtype)
    rows = cache.float().cpu().view(-1, page, row)
    return cache, table, [torch.stack([rows[int(table[r, j // page]), j % page] for j in range(n)]) for r, n in enumerate(lens)]


def plain_rows_attention(q, keys, first, rank, scale, window):
    """q [t, heads, row] at positions ``first`` on over keys [n, row]: the values are the first ``rank`` columns."""
    s = torch.einsum("thd,jd->thj", q, keys) * scale
    i = torch.arange(first, first + q.shape[0])[:, None, None]
    j = torch.arange(keys.shape[0])[None, None, :]
    seen = (j <= i) if window is None else ((j <= i) & (i - j < window))
    return torch.softmax(s.masked_fill(~seen, float("-inf")), -1) @ keys[:, :rank]


TC_SIZES = [(5, 64, 64), (7, 88, 72), (3, 120, 88), (32, 576, 512), (24, 264, 256), (6, 272, 264), (130, 64, 48), (3, 640, 8), (1, 16, 8),
            (128, 192, 128), (100, 144, 136)]


@pytest.mark.gpu
@pytest.mark.parametrize("heads,row,rank", TC_SIZES)
@pytest.mark.parametrize("page,window", [(64, None), (128, 50), (64, 130)])
def test_portions_over_cached_rows_on_tcgen05(heads, row, rank, page, window):
    """The tcgen05 kernel against a plain softmax over the rows as they lie in the cache: requests of unequal lengths side
    by side with and without a cached prefix, tiles that end inside a token group, rows that are no multiple of a piece,
    ranks in one and two column blocks, more heads than a block has rows; the scores are sharp (a scale of
    several units), so a wrong key shows."""
    from lily_b200.csrc import ops
    dt = torch.bfloat16
    assert ops.latent_tcgen05(dt, row, rank, page)
    g = torch.Generator().manual_seed(row)
    new, prefix = [37, 5, 130 if heads <= 32 else 20], [200, 0, 64]
    cache, table, keys = cached_rows(g, [a + b for a, b in zip(new, prefix)], page, row, dt)
    q = torch.randn(sum(new), heads * row, generator=g).to(device="cuda", dtype=dt)
    out = torch.zeros(sum(new), heads * rank, device="cuda", dtype=dt)
    scale = 3.0 / math.sqrt(row)
    tile = int(ops.library().lily_latent_attention_tc_tile_tokens(heads))
    cu = [0, new[0], new[0] + new[1], sum(new)]
    tr, ts = ops.prefill_tiles(prefix, new, 0, tile, "cuda")
    ops.attention_prefill(q, cache, table.cuda(), i32(cu, "cuda"), i32(prefix, "cuda"), tr, ts, out, heads, 1, row, page, scale, window,
                          tile_rows=tile, dv=rank, values_in_keys=True)
    for r in range(3):
        want = plain_rows_attention(q[cu[r]:cu[r + 1]].float().cpu().view(-1, heads, row), keys[r], prefix[r], rank, scale, window)
        got = out[cu[r]:cu[r + 1]].float().cpu().view(-1, heads, rank)
        assert float((got - want).abs().max()) < 1e-2 * float(want.abs().max()), r
    assert ops.latent_attention_status() == 0


@pytest.mark.gpu
@pytest.mark.parametrize("heads,row,rank", TC_SIZES)
@pytest.mark.parametrize("window", [None, 140])
def test_decoding_over_cached_rows_on_tcgen05(heads, row, rank, window):
    """One new token a request over rows of very different lengths, the keys in one range and in several (some of them
    without a key for the short requests), and as the plan cuts them."""
    from lily_b200.csrc import ops
    dt, page = torch.bfloat16, 64
    g = torch.Generator().manual_seed(row + 1)
    lens = [1, 128, 129, 700, 64, 1500]
    cache, table, keys = cached_rows(g, lens, page, row, dt)
    q = torch.randn(len(lens), heads * row, generator=g).to(device="cuda", dtype=dt)
    scale = 3.0 / math.sqrt(row)
    want = torch.cat([plain_rows_attention(q[r:r + 1].float().cpu().view(1, heads, row), keys[r], n - 1, rank, scale, window)
                      for r, n in enumerate(lens)])
    plan = ops.plan_decode_attention(dt, len(lens), heads, 1, row, max(lens), dv=rank, values_in_keys=True, page_size=page)
    for splits in (1, 2, 5, 12, plan.splits):
        out = torch.zeros(len(lens), heads * rank, device="cuda", dtype=dt)
        scratch = torch.empty(max(1, ops.decode_scratch_floats(len(lens), heads, rank, splits)), device="cuda")
        ops.attention_decode(q, cache, table.cuda(), i32(lens, "cuda"), out, scratch, splits, heads, 1, row, page, scale, window, dv=rank,
                             values_in_keys=True)
        got = out.float().cpu().view(len(lens), heads, rank)
        assert float((got - want).abs().max()) < 1e-2 * float(want.abs().max()), splits
    assert ops.latent_attention_status() == 0


def test_ranges_of_a_decode_step_over_latents():
    from lily_b200.csrc.ops import choose_latent_splits

    assert choose_latent_splits(8, 32, 512, 4096) == 8 and choose_latent_splits(200, 32, 512, 100) == 1
    for requests in (1, 3, 40, 500):
        for length in (1, 128, 1000, 100000):
            assert 1 <= choose_latent_splits(requests, 16, 256, length) <= max(1, -(-length // 128))


@pytest.mark.parametrize("device", DEVICES)
def test_product_per_head_into_a_view(device):
    ops = ops_for(device)
    g = torch.Generator().manual_seed(2)
    for t, heads, k, n, extra, room in ((70, 3, 20, 37, 6, 5), (1, 8, 128, 512, 64, 64), (9, 32, 64, 128, 0, 0), (300, 5, 40, 64, 8, 16)):
        rows, w = torch.randn(t, heads * (k + extra), generator=g), torch.randn(heads, n, k, generator=g)
        for dtype in dtypes_of(device):
            x = rows.to(device=device, dtype=dtype).view(t, heads, k + extra)[:, :, :k]
            out = torch.full((t, heads * (n + room)), 7.0, dtype=dtype, device=device)
            ops.head_linear(x, w.to(device=device, dtype=dtype), out=out.view(t, heads, n + room)[:, :, :n])
            want = torch.einsum("thk,hnk->thn", rounded(rows, dtype).view(t, heads, k + extra)[:, :, :k], rounded(w, dtype))
            got = out.float().cpu().view(t, heads, n + room)
            assert float((got[:, :, :n] - want).abs().max()) < (1e-4 if dtype == torch.float32 else 1e-2) * float(want.abs().max())
            assert bool((got[:, :, n:] == 7.0).all())


@pytest.mark.parametrize("device", DEVICES)
def test_latents_from_partial_sums(device):
    """The down-projection may arrive as partial sums; a mixer that caches nothing leaves the cache alone."""
    ops = ops_for(device)
    g = torch.Generator().manual_seed(4)
    t, q_rank, rank, rot, page = 21, 30, 40, 12, 8
    parts = torch.randn(3, t, q_rank + rank + rot, generator=g)
    gq, gk = 1 + 0.2 * torch.randn(q_rank, generator=g), 1 + 0.2 * torch.randn(rank, generator=g)
    rotation = {"dims": rot, "base": 100.0}
    f, _ = pn.frequencies(rotation)
    ang = torch.arange(64, dtype=torch.float32)[:, None] * f[None, :]
    pos = torch.arange(5, 5 + t)
    whole = parts.sum(0)
    halves = torch.cat([torch.arange(0, rot, 2), torch.arange(1, rot, 2)])
    for dtype in dtypes_of(device):
        for write in (True, False):
            cache = torch.zeros(6, page * (rank + rot), dtype=dtype, device=device)
            x = parts.clone()
            x[:, :, q_rank + rank:] = x[:, :, q_rank + rank:][:, :, halves]          # the order the reordered weights give
            cq = ops.latent_prepare(x.to(device), 0, q_rank, q_rank, rank, rot, rot, gq.to(device), gk.to(device), 1e-5, ang.cos().to(device),
                                    ang.sin().to(device), i32(pos.tolist(), device), i32([0] * t, device), i32([[2, 5, 1, 4]], device), cache,
                                    page, write_kv=write)
            tol = 1e-5 if dtype == torch.float32 else 2e-2
            assert float((cq.float().cpu() - pn.unit_rms(whole[:, :q_rank], 1e-5) * gq).abs().max()) < tol * 4
            rows = cache.float().cpu().view(6, page, rank + rot)
            if not write:
                assert float(rows.abs().max()) == 0.0
                continue
            got = torch.stack([rows[[2, 5, 1, 4][p // page], p % page] for p in pos.tolist()])
            assert float((got[:, :rank] - pn.unit_rms(whole[:, q_rank:q_rank + rank], 1e-5) * gk).abs().max()) < tol * 4
            turned = pn.rotate_pairs(whole[:, q_rank + rank:], pos, rotation)[:, halves]
            assert float((got[:, rank:] - turned).abs().max()) < tol * 5
            assert float(rows[0].abs().max()) == 0.0 and float(rows[3].abs().max()) == 0.0


# ------------------------------------------------------------------ xIELU and the plain feed-forward

@pytest.mark.parametrize("device", DEVICES)
def test_xielu_on_both_sides_of_zero(device):
    ops = ops_for(device)
    z = torch.cat([torch.linspace(-12, 12, 4001), torch.linspace(-0.3, 0.3, 4001), torch.tensor([0.0, -0.0, -1e-6, 1e-6, -80.0, 40.0])])
    for pq in ([0.3, -1.2], [-4.0, 2.5], [0.0, 0.0]):
        t = torch.tensor(pq, dtype=torch.float64)
        factors = (float(torch.nn.functional.softplus(t[0])), 0.5 + float(torch.nn.functional.softplus(t[1])))
        for cols in (z.numel(), 8, 4):                                        # odd, 16-byte pieces, four at a time
            x = z[:z.numel() // cols * cols].view(-1, cols)
            for dtype in dtypes_of(device):
                xr = rounded(x, dtype)
                with pn.precision(torch.float64):
                    want = pn.xielu(xr.double(), t).float()
                got = ops.activation(x.to(device=device, dtype=dtype), dtype, "xielu", factors).float().cpu()
                err = (got - want).abs() - 1e-6
                assert float((err / (want.abs() + 1e-6)).max()) < (2e-6 if dtype == torch.float32 else 5e-3), (pq, cols, dtype)
            sums = torch.stack([0.25 * x, 0.75 * x]).to(device)
            with pn.precision(torch.float64):
                want = pn.xielu(x.double(), t).float()
            got = ops.activation(sums, torch.float32, "xielu", factors).cpu()
            assert float(((got - want).abs() / (want.abs() + 1.0)).max()) < 1e-5


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("rows", [1, 5, 70, 300])
@pytest.mark.parametrize("width,ff", [(64, 200), (40, 24), (256, 512), (33, 17)])
def test_dense_feed_forward(device, rows, width, ff):
    """Few tokens (partial sums), many (the activation in the product's epilogue on the GPU), odd widths."""
    g = torch.Generator().manual_seed(ff)
    w = {"p.up": 1.5 * torch.randn(ff, width, generator=g) / math.sqrt(width), "p.down": torch.randn(width, ff, generator=g) / math.sqrt(ff),
         "p.act": torch.tensor([0.7, -0.9])}
    h = torch.randn(rows, width, generator=g)
    for dtype in dtypes_of(device):
        part = build_part("feed_forward", DenseMLPSpec(width, ff, activation="xielu", names=(("up", "up"), ("down", "down"), ("act", "act"))),
                          "p", context(device, dtype))
        part.load(loader(w, device, dtype))
        y = part.forward(h.to(device=device, dtype=dtype), None)
        got = (y.sum(0) if y.dim() == 3 else y).float().cpu()
        want = pn.dense_ff(rounded(h, dtype), {k: rounded(v, dtype) for k, v in w.items()}, "p")
        assert float((got - want).abs().max()) < (2e-5 if dtype == torch.float32 else 2e-2) * float(want.abs().max())


# ------------------------------------------------------------------ experts

class _Batch:
    def __init__(self, device):
        self.workspace = Workspace(torch.device(device))


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("experts,top,ff,width,shared", [(5, 2, 24, 40, 56), (12, 3, 64, 72, None), (4, 1, 10, 33, 7), (1, 1, 7, 20, 9),
                                                         (40, 8, 16, 48, 128), (6, 6, 128, 256, 256)])
def test_routed_experts_with_weights_on_their_inputs(device, experts, top, ff, width, shared):
    """Sigmoid scores taken as they are, a weight on what an expert is given (far from the same on what it gives: the gate is
    not linear), the shared expert times its gate; one token, a few and many, alone and in a batch."""
    g = torch.Generator().manual_seed(experts * 10 + top)
    n = lambda *shape: torch.randn(*shape, generator=g)
    w = {"p.router": 2 * n(experts, width) / math.sqrt(width)}
    for name, f in [(f"e{e}", ff) for e in range(experts)] + ([("shared", shared)] if shared else []):
        w.update({f"p.{name}.gate": 3 * n(f, width) / math.sqrt(width), f"p.{name}.up": 2 * n(f, width) / math.sqrt(width),
                  f"p.{name}.down": n(width, f) / math.sqrt(f)})
    c = {"router": {"experts": experts, "top": top}}
    if shared:
        w["p.shared.sg"] = n(1, width) / math.sqrt(width)
        c["shared"] = {"ff": shared}
    h = n(77, width)
    spec = RoutedExpertsSpec(width, ff, experts, 0, top, scores="sigmoid", correction=False, renormalise=False, activation="silu",
                             weight_on="input", shared_size=shared or 0)
    for dtype in dtypes_of(device):
        part = build_part("feed_forward", spec, "p", context(device, dtype))
        assert {k: tuple(s.shape) for k, s in part.tensors().items()} == {k: tuple(v.shape) for k, v in w.items()}
        part.load(loader(w, device, dtype))
        wr = {k: rounded(v, dtype) for k, v in w.items()}
        x = rounded(h, dtype)
        want = pn.moe_ff(x, wr, "p", c)
        for rows in (slice(0, 77), slice(5, 6), slice(40, 49)):
            xs = h[rows].to(device=device, dtype=dtype).contiguous()
            y = part.forward(xs, _Batch(device))
            assert y.dtype == torch.float32 and y.shape[0] == 1
            tol = 2e-5 if dtype == torch.float32 else 2e-2
            assert float((y[0].cpu() - want[rows]).abs().max()) < tol * max(1.0, float(want.abs().max())), (dtype, rows)
        ops = ops_for(device)
        big = n(1100, width)                                                  # several tokens share a block on the GPU
        routing = ops.moe_route(big.to(device=device, dtype=dtype), part.router, None, top, experts, scores="sigmoid", renormalise=False,
                                shared_gate=bool(shared), outputs=experts)
        chosen, weights = pn.route(rounded(big, dtype), wr, "p", top)
        assert torch.equal(routing.chosen.cpu().long().sort(-1).values, chosen.sort(-1).values)
        order = routing.chosen.cpu().long().argsort(-1)
        assert float((routing.weights.cpu().gather(1, order) - weights.gather(1, chosen.argsort(-1))).abs().max()) < 1e-5
        if shared:
            assert float((routing.gate.cpu() - torch.sigmoid(rounded(big, dtype) @ wr["p.shared.sg"].t())[:, 0]).abs().max()) < 1e-5
    # the construction does what it says: on the other side of the expert the weight gives something else
    chosen, weights = pn.route(h, w, "p", top)
    t = int(weights[:, -1].argmin())
    e, a = int(chosen[t, -1]), float(weights[t, -1])
    inside, outside = pn.gated_expert(a * h[t:t + 1], w, f"p.e{e}"), a * pn.gated_expert(h[t:t + 1], w, f"p.e{e}")
    assert float((inside - outside).abs().max()) > 0.05 * float(outside.abs().max()) and a < 0.9


# ------------------------------------------------------------------ the add of a normed sublayer, the stream as an input

@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("tokens", [1, 9, 80])
@pytest.mark.parametrize("hidden", [48, 321, 1024, 1000, 4096])
def test_add_of_a_normed_sublayer(device, tokens, hidden):
    """``x + g y / rms(y)`` into the float32 stream and, rounded, to the next sublayer: the cluster's, the register and the
    plain form of the kernel; deltas whole and as partial sums; one gain for all columns."""
    ops = ops_for(device)
    g = torch.Generator().manual_seed(hidden)
    resid = torch.randn(tokens, hidden, generator=g) * 3
    y, parts = torch.randn(tokens, hidden, generator=g), torch.randn(3, tokens, hidden, generator=g)
    norm_w = torch.tensor(0.37)
    for dtype in dtypes_of(device):
        norm = build_part("norm", RMSNormSpec(hidden, 1e-5, suffix="", single_gain=True), "n", context(device, dtype))
        assert tuple(norm.tensors()["n"].shape) == ()
        norm.load(lambda name: norm_w.to(device=device, dtype=dtype))
        gain = rounded(norm_w, dtype)
        for delta, value in ((y.to(device=device, dtype=dtype), rounded(y, dtype)), (parts.to(device), parts.sum(0))):
            stream = resid.clone().to(device)
            want = resid + pn.single_gain_norm(value, gain, 1e-5)
            got = enter_stream(ops, stream, NormedDelta(delta, norm.weight, 1e-5), dtype)
            assert float((stream.cpu() - want).abs().max()) < 2e-5
            assert got.dtype == dtype and float((got.float().cpu() - want).abs().max()) < (2e-5 if dtype == torch.float32 else 5e-3 * float(want.abs().max()))
            if dtype == torch.float32:
                assert got.data_ptr() == stream.data_ptr()
            rows = i32([tokens - 1, 0], device)                              # and the model's last norm over gathered rows
            final = norm.forward(stream, NormedDelta(delta, norm.weight, 1e-5), rows=rows).float().cpu()
            both = (want + pn.single_gain_norm(value, gain, 1e-5))[rows.cpu().long()]
            assert float((final - pn.single_gain_norm(both, gain, 1e-5)).abs().max()) < (1e-5 if dtype == torch.float32 else 1e-2)
    # a stream with nothing pending, and one with plain deltas (as another kind of block hands them on)
    stream = resid.clone().to(device)
    assert torch.equal(enter_stream(ops, stream, None, torch.float32).cpu(), resid)
    got = enter_stream(ops, stream, (y.to(device), None, parts.to(device)), torch.float32)
    assert float((got.cpu() - (resid + y + parts.sum(0))).abs().max()) < 2e-5
