"""The CUDA kernels and kernel options that the Bidinex family brought, each alone against its plain restatement in
tests/torch_kernels.py: the norm without statistics with a branch added in each of its three forms, the embedding with that norm, the
rows of the stream join, capped logits, routing among the best groups with weights that sum to one, plain silu experts with the
weighted sum left to the reader, and the gate's numbers behind a latent row's projection."""
import pytest
import torch

import torch_kernels as R
from test_rodapel_kernels_gpu import close, flat_plan, meta_for, paged, rnd

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
SIZES = [(1, 8), (5, 200), (3, 2050), (2, 4099), (7, 1028), (600, 96)]


@pytest.fixture(scope="module")
def K():
    from iitj_llm_coopt_b200 import kernels
    return kernels.load()


def norm_of(width, seed, alpha=0.8):
    return torch.tensor([alpha]).cuda(), rnd(width, seed=seed) + 1.0, rnd(width, seed=seed + 1)


def check(K, res, delta, summed, norm, dtype, factor=0.3):
    """out and the new stream for a delta given in some form, `summed` its float32 tensor; with and without storing, chosen rows,
    a column range as output, and no norm."""
    T, width = res.shape
    want = res + factor * summed if summed is not None else res
    for store in (True, False):
        r, out = res.clone(), torch.full((T, width), 9.0, dtype=dtype, device="cuda")
        K.add_dynamic_tanh(r, delta, factor, norm, out, store=store)
        close(out, R.ref_dynamic_tanh(want, norm), dtype)
        close(r, want if store else res, torch.float32)
    wide = torch.full((T, 2 * width + 3), 9.0, dtype=dtype, device="cuda")
    K.add_dynamic_tanh(res.clone(), delta, factor, None, wide[:, width:2 * width], store=False)
    close(wide[:, width:2 * width], want, dtype)
    assert (wide[:, :width] == 9.0).all() and (wide[:, 2 * width:] == 9.0).all()
    rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32).cuda()
    r, out = res.clone(), torch.full((3, width), 9.0, dtype=dtype, device="cuda")
    K.add_dynamic_tanh(r, delta, factor, norm, out, rows=rows)
    close(out, R.ref_dynamic_tanh(want[rows.long()], norm), dtype)
    assert torch.equal(r, res)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,width", SIZES)
def test_add_dynamic_tanh(K, dtype, tokens, width):
    from iitj_llm_coopt_b200.kernels import PartialSums
    res, norm = rnd(tokens, width, seed=1, s=2.0), norm_of(width, 3)
    check(K, res, None, None, norm, dtype)
    branch = rnd(tokens, width, dtype=dtype, seed=2, s=3.0)
    check(K, res, branch, branch.float(), norm, dtype)
    for splits in (2, 8) + ((9,) if dtype == torch.float32 else ()):      # more than eight parts are added up as the engine's type first
        parts = rnd(splits, tokens, width, seed=splits)
        sums = PartialSums(K, parts, torch.empty(tokens, width, dtype=dtype, device="cuda"))
        check(K, res, sums, parts.sum(0), norm, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,width,top", [(1, 8, 1), (6, 200, 3), (3, 2050, 4), (5, 99, 5), (300, 64, 9)])
def test_routed_sums_are_added_on_the_way(K, dtype, tokens, width, top):
    g = torch.Generator().manual_seed(top)
    place = torch.randperm(tokens * top, generator=g).to(torch.int32).cuda()
    y, w = rnd(tokens * top, width, dtype=dtype, seed=4), torch.rand(tokens, top, generator=g).cuda()
    chosen = torch.zeros(tokens, top, dtype=torch.int32, device="cuda")
    res, norm = rnd(tokens, width, seed=1), norm_of(width, 5)
    x, out = rnd(tokens, width, dtype=dtype, seed=6), torch.empty(tokens, width, dtype=dtype, device="cuda")
    for weights in (w, None):
        delta = K.moe_combine(y, {"place": place}, chosen, weights, x, 1, out, defer=True)
        rows = y.float()[place.long()].view(tokens, top, width)
        summed = (rows * weights.unsqueeze(2)).sum(1) if weights is not None else rows.sum(1)
        check(K, res, delta, summed, norm, dtype)
        close(delta.sum(), summed, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,width", SIZES)
def test_embed_dynamic_tanh(K, dtype, tokens, width):
    table, norm = rnd(50, width, dtype=dtype, seed=7, s=2.0), norm_of(width, 8, alpha=1.3)
    ids = torch.randint(0, 50, (tokens,), dtype=torch.int32, generator=torch.Generator().manual_seed(1)).cuda()
    want = R.ref_dynamic_tanh(R.ref_embed(ids, table, 0.7), norm)
    out = torch.empty(tokens, width, device="cuda")
    K.embed_dynamic_tanh(ids, table, 0.7, norm, out)
    close(out, want, torch.float32)
    wide = torch.full((tokens, 2 * width), 9.0, dtype=dtype, device="cuda")
    K.embed_dynamic_tanh(ids, table, 0.7, norm, out, cast_out=wide[:, width:])
    assert torch.equal(wide[:, width:], out.to(dtype)) and (wide[:, :width] == 9.0).all()


@pytest.mark.parametrize("shape", [(1, 1), (3, 77), (2, 4096), (5, 1001)])
def test_softcap(K, shape):
    x = rnd(*shape, s=30.0)
    want = 12.5 * torch.tanh(x / 12.5)
    close(K.softcap_(x.clone(), 12.5), want, torch.float32)
    assert want.abs().max() <= 12.5


@pytest.mark.parametrize("outputs,top,groups", [(12, 2, (3, 1)), (12, 3, (3, 2)), (6, 4, (6, 4)), (8, 8, (2, 2)), (1, 1, (1, 1)), (96, 6, (48, 5)),
                                                (256, 8, (8, 4)), (40, 5, None)])
def test_route_topk_in_groups(K, outputs, top, groups):
    for sigmoid in (False, True):
        scores = rnd(70, outputs, s=2.0, seed=top)
        chosen = torch.empty(70, top, dtype=torch.int32, device="cuda")
        weights = torch.empty(70, top, dtype=torch.float32, device="cuda")
        K.route_topk(scores, None, chosen, weights, sigmoid=sigmoid, groups=groups, renormalize=1e-20)
        c, w = R.ref_route_topk(scores, None, top, sigmoid=sigmoid, groups=groups, renormalize=1e-20)
        assert torch.equal(chosen, c)
        close(weights, w, torch.float32)
        assert (weights.sum(1) - 1).abs().max() < 1e-6
        if groups and groups[1] < groups[0]:
            assert all(len(set((row // (outputs // groups[0])).tolist())) <= groups[1] for row in chosen)


def test_a_closed_group_keeps_its_second_best_out(K):
    """The best group holds one large score and three of the smallest; the second best output overall is in a closed group."""
    scores = torch.tensor([[5.0, -9.0, -8.0, -7.0, 4.0, 3.9, 3.8, 3.7]]).cuda()
    chosen, weights = torch.empty(1, 2, dtype=torch.int32, device="cuda"), torch.empty(1, 2, device="cuda")
    K.route_topk(scores, None, chosen, weights, groups=(2, 1), renormalize=1e-20)
    assert chosen.tolist() == [[0, 3]]
    K.route_topk(scores, None, chosen, weights, groups=(2, 2), renormalize=1e-20)
    assert chosen.tolist() == [[0, 4]]
    # a correction moves the choice, not the weights
    corr = torch.tensor([0.0] * 7 + [2.0]).cuda()
    K.route_topk(scores, corr, chosen, weights, groups=(2, 1), renormalize=1e-20)
    c, w = R.ref_route_topk(scores, corr, 2, groups=(2, 1), renormalize=1e-20)
    assert chosen.tolist() == c.tolist() == [[7, 4]]
    close(weights, w, torch.float32)


def test_groups_that_do_not_fit_are_refused(K):
    from iitj_llm_coopt_b200.kernels import KernelError
    scores = rnd(2, 12)
    chosen, weights = torch.empty(2, 5, dtype=torch.int32, device="cuda"), torch.empty(2, 5, device="cuda")
    for groups in ((5, 2), (3, 4), (3, 1), (3, 0)):
        with pytest.raises(KernelError):
            K.route_topk(scores, None, chosen, weights, groups=groups)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens,top,experts,width,ff", [(11, 2, 10, 40, 24), (150, 3, 3, 64, 100), (9, 1, 1, 16, 8), (33, 4, 6, 33, 17)])
def test_plain_silu_experts(K, dtype, tokens, top, experts, width, ff):
    g = torch.Generator().manual_seed(tokens)
    chosen = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(tokens)]).to(torch.int32).cuda()
    weights = torch.rand(tokens, top, generator=g).cuda()
    x = rnd(tokens, width, dtype=dtype, seed=1)
    w1 = rnd(experts, 2 * ff, width, dtype=dtype, seed=2, s=2 * width ** -0.5)
    w2 = rnd(experts, width, ff, dtype=dtype, seed=3, s=ff ** -0.5)
    rows, outs = tokens * top, []
    for kern in (K, R.TorchKernels()):
        plan = kern.moe_plan(chosen, experts, *(torch.zeros(rows, dtype=torch.int32, device="cuda") for _ in range(2)),
                             torch.zeros(kern.moe_tile_bound(rows, experts) + 1, 4, dtype=torch.int32, device="cuda"))
        act = torch.zeros(rows, ff, dtype=dtype, device="cuda")
        kern.moe_linear(x, w1, act, plan, gather=True, glu="silu")
        y = torch.zeros(rows, width, dtype=dtype, device="cuda")
        kern.moe_linear(act, w2, y, plan)
        outs.append(kern.moe_combine(y, plan, chosen, weights, x, experts, torch.zeros(tokens, width, dtype=dtype, device="cuda")))
    close(outs[0], outs[1], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,rot,rotary,rank,pad", [(3, 12, 8, 8, 24, 5), (1, 20, 6, 6, 10, 0), (32, 32, 64, 64, 512, 0),
                                                           (9, 6, 8, 4, 16, 7), (5, 16, 16, 0, 32, 3)])
def test_gate_behind_the_latent_row(K, dtype, heads, dim, rot, rotary, rank, pad):
    """The gate's numbers and the rest of the projection, then the attention with that gate on its heads (one and two key splits)."""
    T, page, row = 50, 16, rank + rot
    cache, table = paged(dtype, 1, [T], page, row, seed=rank)
    ref_cache, pos = cache.clone(), list(range(T))
    gain = rnd(rank, seed=9) * 0.1 + 1.0
    slots = torch.tensor([int(table[0, p // page]) * page + p % page for p in pos], dtype=torch.int32).cuda()
    at = heads * (dim + rot) + row
    qd = rnd(T, at + heads + pad, dtype=dtype, seed=3)
    tables = None
    if rotary:
        ang = torch.tensor(pos).float().unsqueeze(1) * (1.0 / 100.0 ** (torch.arange(0, rotary, 2).float() / rotary)).unsqueeze(0)
        tables = (ang.cos().cuda().contiguous(), ang.sin().cuda().contiguous())
    qa = rnd(T, heads * row, dtype=dtype, seed=5)
    qb, gate = qa.clone(), torch.full((T, heads), 9.0, device="cuda")
    RK = R.TorchKernels()
    K.latent_prepare(qd, tables, rotary, False, gain, 1e-5, qa, cache, slots, heads, dim, rot, rank, gate_out=gate)
    RK.latent_prepare(qd[:, :at].contiguous(), tables, rotary, False, gain, 1e-5, qb, ref_cache, slots, heads, dim, rot, rank)
    close(qa, qb, dtype)
    assert torch.equal(cache.isnan(), ref_cache.isnan())                  # rows of the pool that nothing wrote
    close(cache.nan_to_num(), ref_cache.nan_to_num(), dtype)
    assert torch.equal(gate, qd[:, at:at + heads].float())
    meta = meta_for(table, [0] * T, pos)
    want = torch.empty(T, heads * rank, device="cuda")
    RK.attention_flat(qb, ref_cache, meta, want, heads, 1, row, rank, shared_value=True, scale=0.2, gate=gate)
    for plan in (None, flat_plan(K, [0] * T, pos, heads, 1, row, rank, 0), flat_plan(K, [0] * T, pos, heads, 1, row, rank, 0, splits=2)):
        out = torch.full((T, heads * rank), float("nan"), dtype=dtype, device="cuda")
        K.attention_flat(qa, cache, meta, out, heads, 1, row, rank, shared_value=True, scale=0.2, gate=gate, plan=plan)
        close(out, want, dtype)
