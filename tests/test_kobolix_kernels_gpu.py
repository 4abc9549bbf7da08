"""The CUDA kernels and kernel options that the Kobolix family brought, each alone against its plain restatement in
tests/torch_kernels.py: the matrix memory and the gated delta rule as single tokens, as portions walked token by token and as portions
cut into chunks, continued over several steps with requests of unequal length in slots of their own; states that decay at once or
not at all; the branch norm with every form of the branch; routing by the two best scores of a group."""
import math

import pytest
import torch

import torch_kernels as R
from test_rodapel_kernels_gpu import close, rnd

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def K():
    from iitj_llm_coopt_b200 import kernels
    return kernels.load()


def i32(x):
    return torch.tensor(x, dtype=torch.int32).cuda()


def step_arrays(K, done, portion, slots):
    """Index arrays of a step that brings portion[r] tokens of every request r that has `done[r]` behind it."""
    from iitj_llm_coopt_b200.parts.base import StepShape
    from iitj_llm_coopt_b200.parts.state_plan import plan_state_chunks
    live = [r for r, n in enumerate(portion) if n]
    lens = [portion[r] for r in live]
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    shape = StepShape(lens, [done[r] + portion[r] for r in live], cu[-1], False, False, "cuda")
    plan = plan_state_chunks(K, shape)
    if plan is not None:
        plan.bind({k: i32(v) for k, v in plan.arrays.items()})
    pos = [done[r] + i for r in live for i in range(portion[r])]
    treq = [j for j, n in enumerate(lens) for _ in range(n)]
    return dict(T=cu[-1], longest=max(lens), plan=plan, cu=i32(cu), slots=i32([slots[r] for r in live]), pos=i32(pos), treq=i32(treq))


# portions of three requests, step after step: whole prompts, portions down to two tokens, single tokens beside portions, single tokens
PORTIONS = {
    "chunks": [[130, 64, 200], [1, 65, 2], [1, 1, 1], [70, 1, 64]],
    "walks": [[3, 17, 0], [2, 1, 40], [1, 1, 1], [0, 16, 1], [33, 2, 5]],
    "decode": [[1, 1, 1]] * 6,
}


def tolerance(dtype):
    return 2e-5 if dtype == torch.float32 else 2e-2


def check_state(got, want, scale=1e-4):
    assert torch.isfinite(got).all()
    assert (got - want).abs().max().item() <= scale * max(want.abs().max().item(), 1e-3), (got - want).abs().max().item()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portions", list(PORTIONS))
@pytest.mark.parametrize("H,D,V,cap", [(3, 16, 24, 5.0), (2, 64, 128, 12.0), (1, 7, 5, 3.0), (2, 48, 64, 8.0), (5, 32, 40, 15.0),
                                       (2, 128, 200, 10.0), (1, 256, 96, 6.0), (1, 320, 30, 6.0)])
def test_matrix_memory(K, dtype, portions, H, D, V, cap):
    from iitj_llm_coopt_b200.parts.matrix_memory import record
    g = torch.Generator().manual_seed(D + V)
    n = record(H, D, V)
    state = torch.zeros(6, n).cuda()
    want_state = state.clone()
    bias, gain = rnd(2 * H, seed=1), 1.0 + 0.2 * rnd(H * V, seed=2)
    bias[H:] += 2.0                                  # forget gates near one, as trained ones are
    done, slots = [0, 0, 0], [4, 1, 3]
    for step, portion in enumerate(PORTIONS[portions]):
        a = step_arrays(K, done, portion, slots)
        T = a["T"]
        proj = torch.randn(T, 2 * H * (D + V), generator=g).to(dtype).cuda()
        gates = (torch.randn(T, 2 * H, generator=g) * 3.0).cuda()
        out = torch.empty(T, H * V, dtype=dtype, device="cuda")
        want = R.ref_matrix_memory(proj, gates, bias, cap, gain, 1e-5, 1e-6, want_state, a["slots"], a["cu"], H, D, V)
        K.matrix_memory(proj, gates, bias, cap, gain, 1e-5, 1e-6, state, a["slots"], a["cu"], out, H, D, V, longest=a["longest"], plan=a["plan"])
        assert (out.float() - want).abs().max().item() <= tolerance(dtype) * want.abs().max().item(), (step, portion)
        check_state(state[slots], want_state[slots])
        done = [d + n for d, n in zip(done, portion)]
    assert not state[0].any() and not state[2].any() and not state[5].any()          # nobody else's slot was touched


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portions", list(PORTIONS))
@pytest.mark.parametrize("H,G,D,V,taps", [(4, 2, 16, 24, 3), (2, 2, 64, 128, 4), (3, 1, 7, 5, 1), (6, 3, 32, 40, 2), (4, 1, 128, 72, 4),
                                          (2, 1, 96, 32, 7), (1, 1, 200, 30, 9)])
def test_gated_delta(K, dtype, portions, H, G, D, V, taps):
    from iitj_llm_coopt_b200.parts.delta_rule import record
    g = torch.Generator().manual_seed(D + V)
    C, n = 2 * G * D + H * V, record(H, G, D, V, taps)
    state = torch.zeros(6, n).cuda()
    want_state = state.clone()
    conv, rate = rnd(C, taps, seed=1) * 0.5, torch.exp(rnd(H, seed=2) - 1.5)
    dt, gain = rnd(H, seed=3), 1.0 + 0.2 * rnd(V, seed=4)
    done, slots = [0, 0, 0], [4, 1, 3]
    for step, portion in enumerate(PORTIONS[portions]):
        a = step_arrays(K, done, portion, slots)
        T = a["T"]
        proj = torch.randn(T, C + H * V, generator=g).to(dtype).cuda()
        gates = (torch.randn(T, 2 * H, generator=g) * 2.0).cuda()
        out = torch.empty(T, H * V, dtype=dtype, device="cuda")
        want = R.ref_gated_delta(proj, gates, conv, rate, dt, gain, 1e-5, 1e-6, want_state, a["slots"], a["pos"], a["cu"], H, G, D, V)
        K.gated_delta(proj, gates, conv, rate, dt, gain, 1e-5, 1e-6, state, a["slots"], a["pos"], a["treq"], a["cu"], out, H, G, D, V,
                      longest=a["longest"], plan=a["plan"])
        err = (out.float() - want).abs().amax(1) / want.abs().max()
        if dtype == torch.float32:
            assert err.max().item() <= tolerance(dtype), (step, portion)
        else:       # the convolved rows of portions are bfloat16: a head whose output nearly cancels is normed up to size with its rounding
            assert err.median().item() <= tolerance(dtype) and err.max().item() <= 8 * tolerance(dtype), (step, portion, err.max().item())
        check_state(state[slots], want_state[slots], 1e-4 if dtype == torch.float32 else 2e-2)
        done = [d + n for d, n in zip(done, portion)]
    assert not state[0].any() and not state[2].any() and not state[5].any()


@pytest.mark.parametrize("mixer", ["memory", "delta"])
def test_chunks_and_walk_agree(K, monkeypatch, mixer):
    """The same bfloat16 portion cut into chunks and walked token by token: the two forms differ by the split halves' rounding alone, at
    every chunk's edge and behind it."""
    H, G, D, V, taps, T = 4, 2, 64, 96, 4, 64 * 5 + 17
    g = torch.Generator().manual_seed(9)
    outs, states = [], []
    for size_from in (64, 1 << 30):
        monkeypatch.setattr(K, "state_chunk_from", size_from)
        a = step_arrays(K, [0], [T], [1])
        g.manual_seed(9)
        gates = (torch.randn(T, 2 * H, generator=g) * 2.0).cuda()
        out = torch.empty(T, H * V, dtype=torch.bfloat16, device="cuda")
        if mixer == "memory":
            from iitj_llm_coopt_b200.parts.matrix_memory import record
            proj = torch.randn(T, 2 * H * (D + V), generator=g).bfloat16().cuda()
            state = torch.zeros(2, record(H, D, V)).cuda()
            K.matrix_memory(proj, gates, rnd(2 * H, seed=1) + 1.0, 8.0, torch.ones(H * V).cuda(), 1e-6, 1e-6, state, a["slots"], a["cu"], out, H,
                            D, V, longest=T, plan=a["plan"])
        else:
            from iitj_llm_coopt_b200.parts.delta_rule import record
            C = 2 * G * D + H * V
            proj = torch.randn(T, C + H * V, generator=g).bfloat16().cuda()
            state = torch.zeros(2, record(H, G, D, V, taps)).cuda()
            K.gated_delta(proj, gates, rnd(C, taps, seed=1) * 0.5, torch.full((H,), 0.05).cuda(), rnd(H, seed=3), torch.ones(V).cuda(), 1e-6, 1e-6,
                          state, a["slots"], a["pos"], a["treq"], a["cu"], out, H, G, D, V, longest=T, plan=a["plan"])
        outs.append(out.float())
        states.append(state[1].clone())
    assert (outs[0] - outs[1]).abs().max().item() <= 1e-2 * outs[1].abs().max().item()        # one bfloat16 step of the output
    check_state(states[0], states[1], 1e-4)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("f_bias", [-40.0, 40.0])
def test_matrix_memory_at_the_gates_ends(K, dtype, f_bias):
    """Forget gates capped at either end: nothing of the past is kept, or all of it for 200 tokens; one input gate far above the rest."""
    from iitj_llm_coopt_b200.parts.matrix_memory import record
    H, D, V, T = 2, 32, 48, 200
    a = step_arrays(K, [0], [T], [0])
    g = torch.Generator().manual_seed(4)
    proj = torch.randn(T, 2 * H * (D + V), generator=g).to(dtype).cuda()
    gates = torch.randn(T, 2 * H, generator=g).cuda()
    gates[70, :H] = 60.0
    bias, gain = torch.tensor([0.0] * H + [f_bias] * H).cuda(), torch.ones(H * V).cuda()
    state = torch.zeros(1, record(H, D, V)).cuda()
    want_state = state.clone()
    out = torch.empty(T, H * V, dtype=dtype, device="cuda")
    want = R.ref_matrix_memory(proj, gates, bias, 15.0, gain, 1e-6, 1e-6, want_state, a["slots"], a["cu"], H, D, V)
    K.matrix_memory(proj, gates, bias, 15.0, gain, 1e-6, 1e-6, state, a["slots"], a["cu"], out, H, D, V, longest=T, plan=a["plan"])
    err = (out.float() - want).abs().amax(1) / want.abs().max()
    assert err.median().item() <= tolerance(dtype) and err.max().item() <= 10 * tolerance(dtype)
    check_state(state, want_state)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,width", [(1, 64), (5, 320), (9, 4096), (600, 384), (7, 50), (600, 50)])
@pytest.mark.parametrize("form", ["rows", "float32 rows", "parts", "routed", "routed and rows", "routed and parts"])
def test_add_branch_rmsnorm(K, dtype, T, width, form):
    from iitj_llm_coopt_b200.kernels import PartialSums
    if "parts" in form and width % 4:
        pytest.skip("a product's parts come in rows of four numbers")
    res, gain = rnd(T, width, seed=1), 1.0 + 0.2 * rnd(width, seed=2)
    E, top, factor = 6, 3, 0.7
    x = rnd(T, width, dtype=dtype, seed=3)
    out_t = torch.empty(T, width, dtype=dtype, device="cuda")
    parts = PartialSums(K, rnd(5, T, width, seed=4), torch.empty_like(out_t))
    if form == "rows":
        delta = rnd(T, width, dtype=dtype, seed=5)
        plain = delta.float()
    elif form == "float32 rows":
        delta = plain = rnd(T, width, seed=5)
    elif form == "parts":
        delta, plain = parts, parts.parts.sum(0)
    else:
        chosen = torch.stack([torch.randperm(E)[:top] for _ in range(T)]).to(torch.int32).cuda()
        weights = rnd(T, top, seed=6).abs()
        rows = T * top
        plan = K.moe_plan(chosen, E, i32([0] * rows), i32([0] * rows), torch.zeros(K.moe_tile_bound(rows, E) + 1, 4, dtype=torch.int32, device="cuda"))
        y = rnd(rows, width, dtype=dtype, seed=7)
        extra, more = None, 0.0
        if form == "routed and rows":
            extra = rnd(T, width, dtype=dtype, seed=8)
            more = extra.float()
        elif form == "routed and parts":
            extra, more = parts, parts.parts.sum(0)
        delta = K.moe_combine(y, plan, chosen, weights, x, E, out_t, defer=True, extra=extra)
        place = plan["place"].view(T, top).long()
        plain = (weights.unsqueeze(2) * y.float()[place]).sum(1) + more
    out = torch.empty(T, width, dtype=dtype, device="cuda")
    want_res = res + factor * plain
    want = want_res * torch.rsqrt(want_res.pow(2).mean(-1, keepdim=True) + 1e-5) * gain
    got_res = res.clone()
    K.add_branch_rmsnorm(got_res, delta, factor, gain, 1e-5, out)
    assert (got_res - want_res).abs().max().item() <= 1e-5 * want_res.abs().max().item()
    close(out, want, dtype)
    rows = i32([T - 1, 0])
    picked, kept = torch.empty(2, width, dtype=dtype, device="cuda"), res.clone()
    K.add_branch_rmsnorm(kept, delta, factor, gain, 1e-5, picked, rows=rows)
    assert torch.equal(kept, res)                      # chosen rows are read only
    close(picked, want[rows.long()], dtype)
    if form.startswith("routed"):           # a part that does not take the sums by itself gets them added up
        close(delta.sum(), plain, dtype)


@pytest.mark.parametrize("E,groups,top,scale", [(15, (3, 2), 5, 1.0), (8, (4, 1), 2, 2.5), (6, (6, 4), 3, 0.3), (40, (5, 5), 7, 1.2), (9, None, 2, 1.7)])
def test_route_topk_two_best_of_a_group(K, E, groups, top, scale):
    z = rnd(33, E, seed=E)
    chosen, weights = torch.empty(33, top, dtype=torch.int32, device="cuda"), torch.empty(33, top, device="cuda")
    K.route_topk(z, None, chosen, weights, sigmoid=True, groups=groups, worth=2, scale=scale)
    c, w = R.ref_route_topk(z, None, top, sigmoid=True, groups=groups, worth=2, scale=scale)
    assert torch.equal(chosen.cpu(), c.cpu())
    assert (weights - w).abs().max().item() < 1e-6


def test_a_group_with_one_good_score_loses_to_two_fair_ones(K):
    z = torch.tensor([[3.0, -4.0, -4.0, 1.0, 1.1, -4.0]]).cuda()          # the best single score stands in the first group
    for worth, want in ((2, [4, 3]), (1, [0, 1])):
        chosen, weights = torch.empty(1, 2, dtype=torch.int32, device="cuda"), torch.empty(1, 2, device="cuda")
        K.route_topk(z, None, chosen, weights, sigmoid=True, groups=(2, 1), worth=worth)
        assert chosen[0].tolist() == want
        assert math.isclose(weights[0, 0].item(), 1 / (1 + math.exp(-z[0, want[0]].item())), rel_tol=1e-6)
