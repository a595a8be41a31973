"""Razevik's mechanisms one at a time.  The kernels that came with the design against the formulas of
tests/plain_razevik.py on inputs of the tests' own making, and small models through the engine with weights made so that a
fault shows: a softmax so sharp that one far key carries a row, latents of every width the decode kernel takes, portions
around the length from which keys and values are rebuilt per head."""
from __future__ import annotations

import math
import random

import pytest
import torch

import plain_razevik as plain
import razevik_tiny as rt
import tiny

pytestmark = pytest.mark.gpu
DEV = "cuda:0"


def _close(got, want, tol, what=""):
    err = (got.double().cpu() - want.double()).abs().max().item() / max(want.abs().max().item(), 1e-30)
    assert err <= tol, f"{what}: {err:.3e} of the scale (limit {tol})"


# ---------------------------------------------------------------- the router
ROUTES = [(12, 3, (4, 2)), (6, 6, (3, 3)), (5, 2, (5, 4)), (24, 4, (8, 3)), (64, 8, (8, 4)), (16, 1, None), (40, 5, (2, 1)), (1, 1, (1, 1)), (130, 6, (10, 3))]


@pytest.mark.parametrize("E,top,groups", ROUTES)
@pytest.mark.parametrize("shared", [False, True])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_router_by_ranked_groups(E, top, groups, shared, dtype):
    """Sigmoid scores, corrections that make the choice scores negative, groups ranked by two values; weights, places and
    the shared expert's gate - for the few tokens of a decode step (outputs shared by a cluster) and for many."""
    from reinfer_b200 import ops
    g = torch.Generator().manual_seed(E + top)
    h, scale = 72, 0.7
    n = E + int(shared)
    w = (torch.randn(n, h, generator=g) * 0.3).to(dtype)
    corr = torch.randn(E, generator=g) * 0.4 - 1.0
    x = torch.randn(150, h, generator=g).to(dtype)
    z = x.double() @ w.double().t()
    want = torch.zeros(150, E, dtype=torch.float64)
    for t in range(150):
        chosen, wt = plain.route(z[t, :E], corr.double(), top, {"count": groups[0], "keep": groups[1]} if groups else None)
        want[t, chosen] = wt * scale
    gate = torch.sigmoid(z[:, E:]) * scale
    full = {}
    for T in (1, 6, 64, 150):
        gates, second = ops.moe_router(x[:T].contiguous().to(DEV), w.to(DEV), corr.to(DEV), E, top, mode="group_sigmoid", groups=groups,
                                       scale=scale, shared=shared)
        _close(gates, want[:T], 1e-5, "weights")
        assert ((gates > 0).sum(1) == top).all()
        side, none = ops.moe_router(x[:T].contiguous().to(DEV), w.to(DEV), corr.to(DEV), E, top, mode="group_sigmoid", groups=groups,
                                    scale=scale, shared=shared, side_by_side=True)
        assert none is None and torch.equal(side[:, :E], gates)
        if shared:
            _close(second, gate[:T], 1e-5, "shared gate")
            assert torch.equal(side[:, E:], second)
        else:
            assert second is None
        full[T] = side.cpu()
    for T in (1, 6, 64):                                            # the same bits whatever the batch
        assert torch.equal(full[T], full[150][:T])
    zf = torch.randn(9, n, generator=g)
    gates, second = ops.moe_route(zf.to(DEV), corr.to(DEV), E, top, mode="group_sigmoid", groups=groups, shared=shared)
    for t in range(9):
        chosen, wt = plain.route(zf[t, :E].double(), corr.double(), top, {"count": groups[0], "keep": groups[1]} if groups else None)
        _close(gates[t], torch.zeros(E, dtype=torch.float64).index_put((torch.tensor(chosen),), wt), 1e-6, "from logits")


def test_an_expert_of_a_dropped_group_is_never_chosen():
    """All choice scores are far below zero: an excluded expert must not win by standing at zero."""
    from reinfer_b200 import ops
    E, groups, top = 12, (4, 1), 3
    z = torch.zeros(1, E)
    corr = torch.full((E,), -40.0)
    corr[3:6] = -39.0                                              # the second group is the best
    gates, _ = ops.moe_route(z.to(DEV), corr.to(DEV), E, top, mode="group_sigmoid", groups=groups)
    assert (gates[0, 3:6] > 0.3).all() and gates[0].sum().item() == pytest.approx(1.0, abs=1e-6)


@pytest.mark.parametrize("mode", ["scores", "chosen_logits"])
def test_other_routes_over_a_cluster_give_the_same_bits(mode):
    from reinfer_b200 import ops
    g = torch.Generator().manual_seed(2)
    x, w, corr = torch.randn(100, 64, generator=g).to(DEV), torch.randn(20, 64, generator=g).to(DEV), torch.randn(20, generator=g).to(DEV)
    many, ident = ops.moe_router(x, w, corr, 18 if mode == "scores" else 20, 4, mode=mode)
    few, ident2 = ops.moe_router(x[:7].contiguous(), w, corr, 18 if mode == "scores" else 20, 4, mode=mode)
    assert torch.equal(many[:7], few) and (ident is None or torch.equal(ident[:7], ident2))


# ---------------------------------------------------------------- the pointwise end of a product
ACTS = {"none": lambda z: z, "relu2": plain.relu_squared, "gelu": plain.gelu_erf, "gelu_tanh": plain.gelu_tanh}


def _end(g, T, F, ff, blocks, vocab=9):
    tail = blocks * ff < F
    gates = torch.rand(T, blocks + int(tail), generator=g) * (torch.rand(T, blocks + int(tail), generator=g) < 0.6)
    rows = torch.randn(vocab, F + 16, generator=g)
    idx = torch.randint(0, vocab, (T,), generator=g, dtype=torch.int32)
    per_col = torch.cat([gates[:, :blocks].repeat_interleave(ff, dim=1), gates[:, blocks:].repeat_interleave(F - blocks * ff, dim=1)], dim=1) \
        if tail else gates.repeat_interleave(ff, dim=1)
    return gates, per_col, rows, idx


@pytest.mark.parametrize("act", list(ACTS))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_activation_with_block_factors_and_token_rows(act, dtype):
    from reinfer_b200 import ops
    g = torch.Generator().manual_seed(3)
    T, ff, blocks, F = 11, 12, 4, 4 * 12 + 20
    u = torch.randn(T, F + 3, generator=g) * 2
    gates, per_col, rows, idx = _end(g, T, F, ff, blocks)
    rows = rows.to(dtype)
    base = ACTS[act](u[:, :F].double()) * 0.7
    for with_gates, with_rows in ((False, False), (True, False), (False, True), (True, True)):
        out = torch.empty(T, F, dtype=dtype, device=DEV)
        ops.act_rows(u.to(DEV)[:, :F], out, act, scale=0.7, gates=gates.to(DEV) if with_gates else None, ff=ff, blocks=blocks,
                     mul=(rows.to(DEV)[:, 8:8 + F], idx.to(DEV)) if with_rows else None)
        want = base * (per_col.double() if with_gates else 1.0) * (rows[idx.long(), 8:8 + F].double() if with_rows else 1.0)
        _close(out.float(), want, 1e-5 if dtype == torch.float32 else 1e-2, f"{act} gates {with_gates} rows {with_rows}")


@pytest.mark.parametrize("T", [1, 8, 20, 60, 100, 200, 300, 700])
@pytest.mark.parametrize("act,F,ff,blocks", [("relu2", 264, 0, 0), ("gelu", 5 * 72 + 136, 72, 5), ("gelu", 300, 300, 1), ("gelu_tanh", 24, 0, 0), ("gelu_tanh", 256, 0, 0)])
def test_product_with_the_pointwise_end_in_its_epilogue(T, act, F, ff, blocks):
    """At the token counts of the tensor-core kernels (reduced in a cluster, one tile, persistent): factors per block with a
    tail block of another size, token rows - at a column offset that is and one that is not a multiple of 16 bytes."""
    from reinfer_b200 import ops
    g = torch.Generator().manual_seed(T + F)
    K = 200
    x = torch.randn(T, K, generator=g).to(torch.bfloat16)
    w = (torch.randn(F, K, generator=g) * K ** -0.5).to(torch.bfloat16)
    gates, per_col, rows, idx = _end(g, T, F, ff or F, blocks or 1)
    rows = rows.to(torch.bfloat16)
    base = ACTS[act](x.double() @ w.double().t()) * 1.3
    for off in (None, 8, 5):
        out = torch.empty(T, F, dtype=torch.bfloat16, device=DEV)
        assert ops.gemm_bf16_act(x.to(DEV), w.to(DEV), out, act, scale=1.3, gates=gates.to(DEV) if blocks else None, ff=ff, blocks=blocks,
                                 mul=(rows.to(DEV)[:, off:off + F], idx.to(DEV)) if off is not None else None)
        want = base * (per_col.double() if blocks else 1.0) * (rows[idx.long(), off:off + F].double() if off is not None else 1.0)
        _close(out.float(), want, 1e-2, f"{act} offset {off}")
        if blocks:
            assert (out.float().cpu()[per_col == 0] == 0).all()
    assert ops.status_word() == 0


@pytest.mark.parametrize("T,E,top,h,ff,tail", [(300, 8, 2, 64, 72, 40), (257, 4, 1, 128, 128, 0), (1000, 16, 4, 192, 200, 136), (130, 6, 3, 64, 8, 8)])
def test_ungated_experts_over_rows_sorted_by_expert(T, E, top, h, ff, tail):
    """The grouped form of experts without a gate matrix, their matrices being a slice of wider ones (a shared expert's
    follow), with an expert that nobody chose."""
    from reinfer_b200 import ops
    g = torch.Generator().manual_seed(T + E)
    x = torch.randn(T, h, generator=g).to(torch.bfloat16)
    wu = (torch.randn(E * ff + tail, h, generator=g) * h ** -0.5).to(torch.bfloat16)
    wd = (torch.randn(h, E * ff + tail, generator=g) * ff ** -0.5).to(torch.bfloat16)
    z = torch.randn(T, E, generator=g)
    z[:, 1] = -50.0
    val, idx = torch.topk(z, top, dim=-1)
    gates = torch.zeros(T, E).scatter_(1, idx, torch.softmax(val, -1))
    want = torch.zeros(T, h, dtype=torch.float64)
    for e in range(E):
        rows = (gates[:, e] > 0).nonzero().flatten()
        if len(rows):
            inner = plain.gelu_erf(x[rows].double() @ wu[e * ff:(e + 1) * ff].double().t()).to(torch.bfloat16).double()
            want[rows] += gates[rows, e:e + 1].double() * (inner @ wd[:, e * ff:(e + 1) * ff].double().t())
    base = torch.randn(T, h, generator=g)
    for store in (False, True):
        dst = base.clone().to(DEV)
        assert ops.moe_grouped_experts(x.to(DEV), gates.to(DEV), top, wu.to(DEV)[:E * ff], wd.to(DEV)[:, :E * ff], ff, "gelu", dst, store=store, gated=False)
        _close(dst, want if store else want + base.double(), 5e-3, f"store {store}")
    assert ops.status_word() == 0


# ---------------------------------------------------------------- norms
@pytest.mark.parametrize("h", [52, 64, 330, 1024, 4096, 5120])
@pytest.mark.parametrize("wdtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_two_norms_of_one_stream(h, wdtype, dtype):
    from reinfer_b200 import ops
    g = torch.Generator().manual_seed(h)
    x = torch.randn(7, h, generator=g) * 3
    w1, w2 = (torch.randn(h, generator=g).to(wdtype) for _ in range(2))
    a, b = ops.rmsnorm_pair(x.to(DEV), w1.to(DEV), w2.to(DEV), 1e-3, dtype)
    n = plain.rms(x.double(), 1e-3)
    tol = 1e-5 if dtype == torch.float32 else 5e-3
    _close(a.float(), n * w1.double(), tol, "first")
    _close(b.float(), n * w2.double(), tol, "second")
    one, none = ops.rmsnorm_pair(x.to(DEV), w1.to(DEV), None, 1e-3, dtype)
    assert none is None and torch.equal(one, a)


@pytest.mark.parametrize("h", [52, 64, 1024, 4096])
@pytest.mark.parametrize("parts", [1, 3])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_output_norm_that_leaves_the_next_two_norms_rows(h, parts, dtype):
    """x += m rms(y) w, and the rows of the two norms that read the new x - the same bits as those norms run by themselves."""
    from reinfer_b200 import ops
    g = torch.Generator().manual_seed(h + parts)
    x, y = torch.randn(5, h, generator=g), torch.randn(parts, 5, h, generator=g)
    w, w1, w2 = (torch.randn(h, generator=g).to(DEV) for _ in range(3))
    xd = x.clone().to(DEV)
    a, b = ops.residual_outnorm(xd, (y if parts > 1 else y[0]).to(DEV), w, 1e-5, 0.6, next_pair=(w1, w2, 1e-3, dtype))
    new = x.double() + 0.6 * plain.rms(y.double().sum(0), 1e-5) * w.double().cpu()
    _close(xd, new, 1e-5, "stream")
    n = plain.rms(new, 1e-3)
    tol = 2e-5 if dtype == torch.float32 else 5e-3
    _close(a.float(), n * w1.double().cpu(), tol, "first")
    _close(b.float(), n * w2.double().cpu(), tol, "second")


@pytest.mark.parametrize("rows,h", [(1, 5), (3, 52), (7, 1024), (65, 330)])
def test_rounded_rows(rows, h):
    from reinfer_b200 import ops
    x = torch.randn(rows, h)
    assert torch.equal(ops.round_rows(x.to(DEV)).cpu(), x.to(torch.bfloat16))


# ---------------------------------------------------------------- latent attention's small kernels
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_per_head_maps_with_one_gate_a_head_and_a_factor(dtype):
    from reinfer_b200 import ops
    g = torch.Generator().manual_seed(8)
    T, H, n_in, n_out = 70, 3, 24, 20
    x = torch.randn(T, H, n_in, generator=g).to(dtype)
    w = (torch.randn(H, n_out, n_in, generator=g) * 0.3).to(dtype)
    gate = torch.randn(T, H + 5, generator=g) * 2
    y = torch.empty(T, H, n_out, dtype=dtype, device=DEV)
    ops.heads_linear(x.to(DEV), w.to(DEV), y, gate=gate.to(DEV)[:, 2:2 + H], out_scale=0.6)
    want = 0.6 * torch.einsum("thi,hoi->tho", x.double(), w.double()) * torch.sigmoid(gate[:, 2:2 + H].double())[:, :, None]
    _close(y.float(), want, 1e-5 if dtype == torch.float32 else 1e-2, "gated maps")


def test_bottleneck_alone():
    """A layer without a latent of its own: the queries' bottleneck is normalised, nothing is stored."""
    from reinfer_b200 import ops
    g = torch.Generator().manual_seed(4)
    x, w = torch.randn(6, 30, generator=g), torch.randn(24, generator=g)
    a = torch.empty(6, 24, device=DEV)
    cache = torch.full((3, 8, 16), 7.0, device=DEV)
    ops.latent_prep(x.to(DEV), 24, 0, 0, w.to(DEV), None, 1e-5, torch.arange(6, dtype=torch.int32, device=DEV), None, 0, 1.0,
                    torch.arange(6, dtype=torch.int32, device=DEV), a, cache, 8)
    _close(a, plain.rms(x[:, :24].double(), 1e-5) * w.double(), 1e-5, "bottleneck")
    assert (cache == 7.0).all()


# ---------------------------------------------------------------- small models through the engine
def _run_cuts(tmp_path, cfg, seqs, page, dtype, tol, seed=3, cuts=None, edit=None, tail=40, sizes=(37, 2, 64, 3, 70, 5, 2, 11)):
    from reinfer_b200.engine import Engine, StepEntry
    store = torch.float32 if dtype == "float32" else torch.bfloat16
    d = rt.make_model_dir(str(tmp_path / f"m{dtype}"), "X", store, cfg=cfg, seed=seed, edit=edit)
    raw, w = plain.read_model(d)
    want = {r: plain.forward(raw, w, t) for r, t in seqs.items()}
    worst = []
    for steps in cuts or (tiny.cut_whole(seqs), tiny.cut_tail_one_by_one(seqs, tail=tail), tiny.cut_portions(seqs, sizes=sizes), tiny.cut_mixed(seqs, seed=seed)):
        e = Engine.from_model_dir(d, dtype=dtype, page_size=page, max_tokens=tiny.pool_tokens_needed(steps, page), max_num_seqs=4)
        done, errs = {}, []
        for entries, end in steps:
            lg = e.step([StepEntry(r, t, wnt) for r, t, wnt in entries]).double().cpu()
            row = 0
            for r, t, wnt in entries:
                for kk in wnt:
                    ref = want[r][done.get(r, 0) + kk]
                    errs.append((lg[row] - ref).abs().max().item() / ref.abs().max().item())
                    row += 1
                done[r] = done.get(r, 0) + len(t)
            for r in end:
                e.finish(r)
                done.pop(r, None)
        e.check_guards()
        e.check_status()
        assert e.cache.free_pages() == e.cache.total_pages()
        errs = torch.tensor(errs)
        if dtype == "float32":
            assert errs.max().item() <= tol, f"worst row {errs.max().item():.3e} at {int(errs.argmax())}"
        else:
            assert torch.isfinite(errs).all() and errs.median().item() <= tol / 3 and (errs <= tol).float().mean().item() >= 0.95, \
                f"median {errs.median().item():.3e}, within tolerance {(errs <= tol).float().mean().item():.3f}"
        worst.append(errs)
    return worst


def _seqs(vocab, lengths, seed):
    rnd = random.Random(seed)
    return {f"r{i}": [rnd.randrange(vocab) for _ in range(n)] for i, n in enumerate(lengths)}


def _model(layers, width=64, vocab=101, positions=800, mult=0.7, side=12, cap=15.0):
    return rt._cfg(vocab, width, positions, 1e-5, mult, side, layers, cap)


FFS = {"none": None, "dense": rt._dense(40), "moe": rt._moe(16, 12, 3, (4, 2), shared=24), "moe_free": rt._moe(16, 6, 2), "moe_odd": rt._moe(10, 6, 4, (3, 2), shared=7)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("ff", list(FFS))
def test_one_layer_and_one_feed_forward(tmp_path, ff, dtype):
    cfg = _model([rt._layer(rt._lat(4, 16, 24, 24, 40, 0.3), FFS[ff])], width=52 if ff == "moe_odd" else 64)
    _run_cuts(tmp_path, cfg, _seqs(101, [1, 9, 50, 90, 37], 5), 8, dtype, 1e-4 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("ff,experts,top,groups,shared", [(24, 12, 3, (4, 2), 40), (24, 12, 3, (4, 2), 7), (10, 16, 2, (4, 3), 8), (32, 16, 8, (2, 2), 16),
                                                          (16, 16, 9, None, 24), (8, 32, 4, (8, 2), None), (264, 4, 1, (2, 1), 300)])
def test_mixtures_over_long_portions(tmp_path, ff, experts, top, groups, shared):
    """Portions beyond the token count from which only the chosen pairs are computed, with inner sizes the grouped products take
    and sizes they refuse (the stacked form serves then), few and many experts chosen."""
    cfg = _model([rt._layer(rt._lat(2, 16, 16, 24, 24, 0.3), rt._moe(ff, experts, top, groups, shared))])
    seqs = _seqs(101, [310, 290], ff)
    steps = [([("r0", seqs["r0"][:300], list(range(300)))], []),
             ([("r0", seqs["r0"][300:301], [0]), ("r1", seqs["r1"][:280], list(range(280)))], []),
             ([("r0", seqs["r0"][301:], list(range(9))), ("r1", seqs["r1"][280:], list(range(10)))], ["r0", "r1"])]
    _run_cuts(tmp_path, cfg, seqs, 16, "bfloat16", 6e-2, cuts=[steps])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shared", [False, True])
def test_a_far_key_among_hundreds(tmp_path, shared, dtype):
    """A softmax so sharp that single keys carry a row, over 600 tokens: a key that is lost, shifted or read from the wrong page
    or the wrong layer changes rows outright.  Prompts, portions and decoded tokens; with `shared` the second layer reads
    the first one's latents, and only what it puts out counts (the first one's output matrix is small)."""
    layers = [rt._layer(rt._lat(4, 16, 16, 24, 32, 2.0), None)]
    if shared:
        layers.append(rt._layer(rt._lat(3, 24, 16, 20, 32, 2.0, kv_from=0), None))

    def edit(w):
        if shared:
            w["l0.mix.o"] = w["l0.mix.o"] * 0.05
            w["l1.mix.o"] = w["l1.mix.o"] * 3.0
        return w
    cfg = _model(layers)
    _run_cuts(tmp_path, cfg, _seqs(101, [600, 333], 9), 16, dtype, 3e-4 if dtype == "float32" else 6e-2, tail=48,
              sizes=(130, 2, 64, 3, 257, 5), edit=edit)


def _names(d, dtype, page, steps):
    """The kernel families of some steps, eagerly."""
    from reinfer_b200 import ops
    from reinfer_b200.engine import Engine, StepEntry
    e = Engine.from_model_dir(d, dtype=dtype, page_size=page, max_tokens=2048, max_num_seqs=3, cuda_graphs=False)
    out = []
    for entries in steps:
        prof = ops.SegmentProfiler()
        old = ops.set_profiler(prof)
        try:
            prof.begin()
            e.step([StepEntry(r, t, []) for r, t in entries])
        finally:
            ops.set_profiler(old)
        out.append(set(prof.summary()))
    return out


@pytest.mark.parametrize("rank", [8, 24, 64, 72, 128, 136, 192, 200, 256, 264])
@pytest.mark.parametrize("page", [8, 16, 64])
def test_decoding_over_latents_of_every_width(tmp_path, rank, page):
    """Decode steps over latents from one 16-byte piece to beyond the widest the tensor-core kernels take, in pages of each
    kind, with a softmax sharp enough that a single lost key shows: two requests of unequal length, page borders crossed."""
    cfg = _model([rt._layer(rt._lat(5 if rank == 72 else 16, 16, 16, 24, rank, 0.9), None)], positions=400)
    seqs = _seqs(101, [330, 61], rank + page)
    _run_cuts(tmp_path, cfg, seqs, page, "bfloat16", 6e-2, cuts=[tiny.cut_tail_one_by_one(seqs, tail=45)])
    names = _names(str(tmp_path / "mbfloat16"), "bfloat16", page, [[("a", seqs["r0"][:90])], [("a", seqs["r0"][90:91])]])
    assert ("fa_decode_tma" in names[1]) == (rank <= 256), names[1]


@pytest.mark.parametrize("heads,rank", [(3, 64), (2, 200), (16, 136)])
def test_prompts_whose_keys_and_values_are_rebuilt_per_head(tmp_path, heads, rank):
    """Heads of 128: portions of 64 tokens and more take the tcgen05 kernel over rebuilt keys and values, shorter ones and single
    tokens the latent form, also side by side in a step; the second layer rebuilds from the first one's latents.  A sharp
    softmax; portions that start inside a page, at a page's border, and end one token before and behind a key tile."""
    from reinfer_b200.parts import latent_attention as la
    layers = [rt._layer(rt._lat(heads, 128, 128, 32, rank, 0.3), None), rt._layer(rt._lat(2, 128, 128, 48, rank, 0.3, kv_from=0), FFS["moe"])]
    cfg = _model(layers, positions=700)
    seqs = _seqs(101, [500, 203, 64, 190], heads)
    mixed = [([("r0", seqs["r0"][:127], list(range(127))), ("r1", seqs["r1"][:65], list(range(65)))], []),
             ([("r0", seqs["r0"][127:128], [0]), ("r1", seqs["r1"][65:200], list(range(135))), ("r2", seqs["r2"], list(range(64)))], ["r2"]),
             ([("r0", seqs["r0"][128:399], list(range(271))), ("r1", seqs["r1"][200:201], [0]), ("r3", seqs["r3"][:2], [0, 1])], []),
             ([("r0", seqs["r0"][399:], list(range(101))), ("r1", seqs["r1"][201:], [0, 1]), ("r3", seqs["r3"][2:], list(range(188)))], ["r0", "r1", "r3"])]
    _run_cuts(tmp_path, cfg, seqs, 16, "bfloat16", 6e-2, cuts=[tiny.cut_whole(seqs), mixed, tiny.cut_portions(seqs, sizes=(70, 3, 64, 63, 1, 129, 2, 200)),
                                                               tiny.cut_tail_one_by_one(seqs, tail=40)])
    d = str(tmp_path / "mbfloat16")
    names = _names(d, "bfloat16", 16, [[("a", seqs["r0"][:100])], [("a", seqs["r0"][100:101]), ("b", seqs["r1"][:80])], [("a", seqs["r0"][101:120])]])
    assert {"latent_gather", "fa_prefill_tc"} <= names[0] and any(n.startswith("gemm+pages") for n in names[0]) and "fa_prefill" not in names[0], names[0]
    assert {"fa_decode_tma", "fa_prefill_tc"} <= names[1], names[1]
    assert "fa_prefill" in names[2] and "fa_prefill_tc" not in names[2], names[2]
    # the two forms agree
    from reinfer_b200.engine import Engine, StepEntry
    got = []
    try:
        for la.REBUILD in (True, False):
            e = Engine.from_model_dir(d, dtype="bfloat16", page_size=16, max_tokens=512, max_num_seqs=1)
            got.append(e.step([StepEntry("a", seqs["r0"], list(range(500)))]).double().cpu())
    finally:
        la.REBUILD = True
    err = (got[0] - got[1]).abs().amax(1) / got[1].abs().amax(1)
    assert err.median().item() <= 2e-2, err.median().item()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_token_rows_of_every_layer(tmp_path, dtype):
    """Every layer takes its own part of its token's row: with a table in which one token's rows are large in one layer only,
    that token's logits move and nobody else's do (the attention sees no other token: its output matrices are zero)."""
    from reinfer_b200.engine import Engine, StepEntry
    cfg = _model([rt._layer(rt._lat(2, 8, 8, 16, 16, 0.3), None) for _ in range(3)], side=8, width=64)

    def base(w):
        for i in range(3):
            w[f"l{i}.mix.o"] = torch.zeros_like(w[f"l{i}.mix.o"])
        return w
    toks = [5, 9, 5, 70, 9]
    out = {}
    for layer in (None, 0, 1, 2):
        def edit(w, layer=layer):
            w = base(w)
            if layer is not None:
                w["side.embed"][9, layer * 8:(layer + 1) * 8] *= -4.0
            return w
        store = torch.float32 if dtype == "float32" else torch.bfloat16
        d = rt.make_model_dir(str(tmp_path / f"{layer}{dtype}"), "X", store, cfg=cfg, seed=6, edit=edit)
        e = Engine.from_model_dir(d, dtype=dtype, page_size=8, max_tokens=64, max_num_seqs=1)
        out[layer] = e.step([StepEntry("a", toks, list(range(5)))]).double().cpu()
        raw, w = plain.read_model(d)
        _close(out[layer], plain.forward(raw, w, toks), 1e-4 if dtype == "float32" else 4e-2, f"layer {layer}")
    for layer in (0, 1, 2):
        moved = (out[layer] - out[None]).abs().amax(1)
        assert (moved[[0, 2, 3]] == 0).all() and (moved[[1, 4]] > 1e-2).all(), (layer, moved)
