"""The Kobolix family through the engine's step function, cache manager and entry points, against the plain restatement of
tests/plain_kobolix.py: every way of cutting the same requests into steps (whole, the last tokens one by one, portions down to two
tokens, mixed batches over a pool so small that pages and slots are used again), the first tokens, long decoding, a token far away
that every later query and state must still hold, the stream after every layer, each mechanism alone, restatements that are wrong in
one thing, and greedy generation through `LLM.generate`.
CPU cases run the host logic with the plain-torch kernel double; `-m gpu` cases run the CUDA kernels.

bfloat16 and routed experts.  A token whose best router scores lie closer together than bfloat16 rounding moves them may pick another
expert than the float64 restatement does, and everything after it in the request then differs by far more than rounding.  So in
bfloat16 the configurations run with softer attention scales, once with every expert chosen (`soft_variant`: nothing is left to choose,
and there the ways of cutting must also agree with one another) and once as they are; both under bounds on the median and the ninth
decile of the error.  float32 is compared at every position, with the configurations as they are."""
import copy

import pytest
import torch

import plain_kobolix as plain
import replay_cases as cases
from helpers import make_engine, rel_err, run_steps
from kobolix_models import CONFIGS, config, dense, make_tensors, mlstm, moe, parallel, plant_needle, write_model

FP32_TOL, BF16_TOL = 3e-4, 5e-2
# lengths around the page sizes (16, 8, 16, 4), the attention's key tiles of 32 and the states' chunks of 64
LENGTHS = {"A": [1, 15, 16, 17, 33, 130], "B": [2, 8, 31, 33, 97], "C": [3, 16, 63, 64, 65, 200], "D": [7, 17, 64, 129]}

GPU = pytest.mark.gpu
CASES = [pytest.param("cpu", "float32", n, id=f"cpu-fp32-{n}") for n in "ABCD"] + \
        [pytest.param("cuda:0", dt, n, marks=GPU, id=f"gpu-{dt}-{n}") for dt in ("float32", "bfloat16") for n in "ABCD"]


def soft_variant(cfg, all_experts=True):
    """Attention scales a quarter as large (a peaked softmax magnifies bfloat16's rounding of queries and keys far beyond a
    rounding-sized tolerance) and, with `all_experts`, routers that choose every expert."""
    cfg = copy.deepcopy(cfg)
    for lay in cfg["layers"]:
        if lay["type"] == "parallel":
            lay["mixer"]["left"]["scale"] *= 0.25
        if all_experts and lay["mlp"] is not None and lay["mlp"]["kind"] == "moe":
            r = lay["mlp"]["router"]
            r["top"] = r["experts"]
            if "groups" in r:
                r["groups"]["keep"] = r["groups"]["count"]
    return cfg


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    out = {}
    for name, (cfg, seed, _) in CONFIGS.items():
        for key, c in ((name, cfg), (name + "-all", soft_variant(cfg)), (name + "-soft", soft_variant(cfg, all_experts=False))):
            out[key] = write_model(c, str(tmp_path_factory.mktemp("kob_" + key)), seed)
    return out


@pytest.fixture(scope="module")
def refs(dirs):
    cache = {}

    def get(key):
        if key not in cache:
            cfg, seed, _ = CONFIGS[key[0]]
            reqs = cases.requests_for(cfg["vocab"], LENGTHS[key[0]], seed + 10)
            c, w = plain.read_model_dir(dirs[key])
            cache[key] = (reqs, {rid: plain.forward(c, w, toks).float() for rid, toks in reqs.items()})
        return cache[key]
    return get


def errors(rows, ref, reqs):
    """Per position: largest difference of the logits row over the largest logit of the request."""
    out = []
    for rid, toks in reqs.items():
        got = torch.stack([rows[(rid, i)] for i in range(len(toks))])
        top = max(ref[rid].abs().max().item(), 1e-30)
        out += ((got.float().cpu() - ref[rid]).abs().amax(dim=1) / top).tolist()
    return out


def compare(rows, ref, reqs, tol, strict=True):
    """float32 (`strict`): every position within `tol`.  bfloat16: the median within `tol` and nine positions in ten within twice that."""
    e = sorted(errors(rows, ref, reqs))
    if strict:
        assert e[-1] <= tol, e[-1]
    else:
        assert e[len(e) // 2] <= tol and e[int(0.9 * (len(e) - 1))] <= 2 * tol, (e[len(e) // 2], e[int(0.9 * (len(e) - 1))], e[-1])


def agree(rows, base, ref, tol):
    """Two ways of cutting the same requests give the same logits (relative to each request's largest logit)."""
    worst = max(((rows[k].float() - base[k].float()).abs().max() / ref[k[0]].abs().max()).item() for k in base)
    assert worst <= tol, worst


def variants(name, dtype):
    """(model key, compared at every position, whether different cuts must agree closely) for a configuration and type."""
    return [(name, True, True)] if dtype == "float32" else [(name + "-all", False, True), (name + "-soft", False, False)]


@pytest.mark.parametrize("device,dtype,name", CASES)
def test_every_way_of_cutting(dirs, refs, device, dtype, name):
    page = CONFIGS[name][2]
    tol = FP32_TOL if dtype == "float32" else BF16_TOL
    for key, strict, cuts_agree in variants(name, dtype):
        reqs, ref = refs(key)
        mixed_steps, peak = cases.mixed(reqs, live=3, seed=2)
        eng = make_engine(dirs[key], dtype, page, peak // page, device=device, max_num_seqs=3, max_num_batched_tokens=peak)
        base = None
        for steps in (cases.whole(reqs), cases.last_one_by_one(reqs, tail=12), cases.portions(reqs), mixed_steps):
            rows = run_steps(eng, steps)
            eng.cache.check()
            assert all(eng.cache.groups[i].pool.num_free == eng.cache.groups[i].pool.num_pages for i in eng.cache.paged)
            assert len(eng.cache.free_slots) == 3
            compare(rows, ref, reqs, tol, strict)
            if cuts_agree and base is not None:
                agree(rows, base, ref, tol if strict else 3e-2)
            base = base or rows


@pytest.mark.parametrize("device,dtype,name", CASES)
def test_first_tokens_and_token_by_token(dirs, refs, device, dtype, name):
    """A whole request one token a step, from the first on."""
    page = CONFIGS[name][2]
    for key, strict, _ in variants(name, dtype):
        reqs, ref = refs(key)
        rid, toks = max(reqs.items(), key=lambda kv: len(kv[1]) if len(kv[1]) <= 40 else 0)
        eng = make_engine(dirs[key], dtype, page, 16, device=device, max_num_seqs=2)
        rows = run_steps(eng, [([(rid, toks[i:i + 1], [0])], []) for i in range(len(toks))])
        compare(rows, ref, {rid: toks}, FP32_TOL if dtype == "float32" else BF16_TOL, strict)


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda:0", marks=GPU)])
@pytest.mark.parametrize("name", ["A", "B", "D"])
def test_stream_after_every_layer(dirs, refs, device, name):
    """The residual stream behind every layer, with the pending branch added."""
    from iitj_llm_coopt_b200.kernels import materialize
    reqs, _ = refs(name)
    rid, toks = next((r, t) for r, t in reqs.items() if 16 <= len(t) <= 50)
    c, w = plain.read_model_dir(dirs[name])
    want = []
    plain.forward(c, w, toks, want)
    eng = make_engine(dirs[name], "float32", CONFIGS[name][2], 16, device=device, max_num_seqs=2)
    got = []

    def watched(inner):
        def forward(ctx, residual, delta, call):
            res, d = inner(ctx, residual, delta, call)
            got.append((res + c.get("residual_mult", 1.0) * materialize(d).float()).double().cpu())
            return res, d
        return forward
    for block in eng.runner.model.layers:
        block.forward = watched(block.forward)
    run_steps(eng, [([(rid, toks, [])], [rid])])
    assert len(got) == len(want)
    assert max(rel_err(g, x) for g, x in zip(got, want)) < FP32_TOL


NEEDLE = 7
FAR = {"attention beside a delta rule": [(parallel((4, 2, 16, 24, 0.8, 8, 1000.0), (4, 2, 32, 40, 3)), None)],
       "matrix memory": [(mlstm(2, 32, 24, 9.0), dense(20))],
       "both": [(mlstm(3, 16, 32, 6.0), None), (parallel((2, 1, 24, 16, 0.9, 12, 300.0), (2, 1, 64, 24, 4)), dense(28)), (mlstm(1, 24, 16, 11.0), None)]}


@pytest.mark.parametrize("device,dtype", [("cpu", "float32"), pytest.param("cuda:0", "float32", marks=GPU),
                                          pytest.param("cuda:0", "bfloat16", marks=GPU)])
@pytest.mark.parametrize("what", list(FAR))
def test_one_far_token_among_many(tmp_path, device, dtype, what):
    """A token that every later query scores far above all others and that every state holds against all others stands at the start, at
    both sides of a page's and of a chunk's border, or in the middle: the logits of all later positions hang on it, in a prompt, in
    portions and in single decoded tokens."""
    cfg, seed, page = config(56, 99, 1e-5, FAR[what], mult=0.9, scale=1.0), 81, 16
    d = write_model(cfg, str(tmp_path / "m"), seed, tensors=plant_needle(cfg, make_tensors(cfg, seed), NEEDLE))
    c, w = plain.read_model_dir(d)
    total = 150 if device == "cpu" else 500
    base = [t if t != NEEDLE else NEEDLE + 1 for t in cases.requests_for(cfg["vocab"], [total], seed)["r0"]]
    without = plain.forward(c, w, base)
    eng = make_engine(d, dtype, page, -(-total // page) + 1, device=device, max_num_seqs=2, max_num_batched_tokens=total)
    for at in (0, page - 1, page, 63, 64, total // 2 - 1):
        toks = base[:at] + [NEEDLE] + base[at + 1:]
        ref = plain.forward(c, w, toks)
        moved = (ref - without)[at + 1:].abs().amax(dim=1) / ref.abs().max()
        assert moved.median() > 0.1, moved.median()                      # the needle decides what comes behind it
        reqs = {"r0": toks}
        for steps in (cases.whole(reqs), cases.last_one_by_one(reqs, tail=10), cases.portions(reqs)):
            rows = run_steps(eng, steps)
            compare(rows, {"r0": ref.float()}, reqs, FP32_TOL if dtype == "float32" else BF16_TOL, dtype == "float32")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding(dirs, dtype, name):
    """A short prompt, then hundreds of tokens one by one through many pages."""
    cfg, seed, page = CONFIGS[name]
    total = 330
    for key, strict, _ in variants(name, dtype):
        reqs = cases.requests_for(cfg["vocab"], [total], seed + 20)
        c, w = plain.read_model_dir(dirs[key])
        ref = {rid: plain.forward(c, w, toks).float() for rid, toks in reqs.items()}
        eng = make_engine(dirs[key], dtype, page, -(-total // page) + 1, max_num_seqs=2)
        compare(run_steps(eng, cases.last_one_by_one(reqs, tail=total - 21)), ref, reqs, FP32_TOL if dtype == "float32" else BF16_TOL, strict)


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_float32_cuts_agree_closely(dirs, refs, name):
    reqs, _ = refs(name)
    eng = make_engine(dirs[name], "float32", CONFIGS[name][2], 128, max_num_seqs=4)
    a, b = run_steps(eng, cases.whole(reqs)), run_steps(eng, cases.portions(reqs))
    assert max(rel_err(b[k], a[k]) for k in a) < 1e-4


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda:0", marks=GPU)])
@pytest.mark.parametrize("name", ["A", "B"])
def test_greedy_generation_through_llm(dirs, device, name):
    """Prompts of unequal length generate together through the scheduler (small token budget: prompts are cut into portions, the pool is
    small enough that requests wait; on the GPU decode steps replay from CUDA graphs); float32 must choose the plain implementation's
    tokens."""
    from iitj_llm_coopt_b200 import LLM, SamplingParams
    cfg, seed, page = CONFIGS[name]
    c, w = plain.read_model_dir(dirs[name])
    v = cfg["vocab"]
    prompts = [[5, 17, 3, v - 1, 9], [i % v for i in range(40, 77)], [v // 2], [i % v for i in range(20, 39)]]
    want = [plain.greedy(c, w, p, 8) for p in prompts]
    kernels = None
    if device == "cpu":
        from torch_kernels import TorchKernels
        kernels = TorchKernels()
    llm = LLM(dirs[name], dtype="float32", page_size=page, num_pages=128 // page, max_num_seqs=3, max_num_batched_tokens=24,
              device=device, kernels=kernels)
    outs = llm.generate(prompts, SamplingParams(max_tokens=8, ignore_eos=True))
    assert [o.token_ids for o in outs] == want


@pytest.mark.gpu
def test_graphs_and_eager_steps_agree(dirs):
    """Decode steps replayed from captured graphs (padded batches too: their padding rows have a state slot of their own) against a
    generation without graphs, bfloat16: the same tokens, request by request."""
    from iitj_llm_coopt_b200 import LLM, SamplingParams
    cfg, seed, page = CONFIGS["C"]
    prompts = list(cases.requests_for(cfg["vocab"], [5, 70, 12, 33, 64, 3, 20, 9, 41, 17, 2], seed + 5).values())
    outs = []
    for graphs in (True, False):
        llm = LLM(dirs["C-all"], dtype="bfloat16", page_size=page, num_pages=64, max_num_seqs=11, max_num_batched_tokens=300, cuda_graphs=graphs)
        outs.append([o.token_ids for o in llm.generate(prompts, SamplingParams(max_tokens=24, ignore_eos=True))])
    assert outs[0] == outs[1]


@pytest.mark.gpu
def test_command_line_serves_a_model_folder(dirs, tmp_path):
    """The serving command line on a Kobolix folder (continuous batching under a small token budget, float32, greedy): every request's
    ids equal the plain implementation's; and on a named shape of the family with random weights."""
    import json
    import os
    import subprocess
    import sys
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg, seed, page = CONFIGS["B"]
    prompts = list(cases.requests_for(cfg["vocab"], [3, 40, 17, 70, 5], seed + 60).values())
    work, out = tmp_path / "w.jsonl", tmp_path / "res.json"
    work.write_text("\n".join(json.dumps({"id": f"p{i}", "prompt_token_ids": p, "max_tokens": 5 + i}) for i, p in enumerate(prompts)))
    proc = subprocess.run([sys.executable, "-m", "iitj_llm_coopt_b200.cli", "--model", dirs["B"], "--workload", str(work), "--out", str(out),
                           "--num-pages", "64", "--page-size", str(page), "--max-num-seqs", "3", "--max-num-batched-tokens", "48",
                           "--dtype", "float32", "--save-tokens"], cwd=root, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    res = json.loads(out.read_text())
    assert res["summary"]["completed"] == len(prompts) and res["summary"]["failed"] == 0
    c, w = plain.read_model_dir(dirs["B"])
    for i, (p, rec) in enumerate(zip(prompts, res["requests"])):
        assert rec["token_ids"] == plain.greedy(c, w, p, 5 + i), i
    proc = subprocess.run([sys.executable, "-m", "iitj_llm_coopt_b200.cli", "--shape", "kobolix-toy", "--random-seed", "5", "--workload",
                           "synthetic:10:4-300:3-20", "--out", str(out), "--num-pages", "128", "--max-num-seqs", "4",
                           "--max-num-batched-tokens", "96", "--save-tokens"], cwd=root, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    res = json.loads(out.read_text())
    assert res["summary"]["completed"] == 10 and res["summary"]["failed"] == 0
    assert all(len(r["token_ids"]) == r["output_tokens"] == r["max_tokens"] for r in res["requests"])


# ---- each mechanism alone, and restatements that are wrong in one thing -------------------------------------------------
def one(mixer=None, mlp=None, mult=1.0, scale=1.0):
    return config(56, 101, 1e-5, [(mixer or mlstm(3, 10, 14, 6.0), mlp)], mult, scale)


PAR = parallel((4, 2, 12, 10, 0.9, 8, 100.0), (6, 3, 10, 14, 4))
ALONE = {"matrix memory": one(), "attention beside a delta rule": one(PAR), "experts": one(mlp=moe(8, 3, 20, groups=(4, 2), scale=1.7)),
         "experts of any group": one(mlp=moe(8, 3, 20)), "shared expert": one(mlp=moe(4, 1, 12, shared=30)), "dense": one(mlp=dense(36)),
         "embedding scale": one(scale=3.0), "branch factor": one(mult=0.35, mlp=dense(20)), "no rotation": one(parallel(
             (2, 2, 8, 8, 1.0, None, 0.0), (2, 1, 8, 8, 2)))}


def _whole_logits(tmp_path, cfg, device, seed=71, n=60, change=lambda t: t):
    d = write_model(cfg, str(tmp_path / "m"), seed, tensors=change(make_tensors(cfg, seed)))
    c, w = plain.read_model_dir(d)
    reqs = cases.requests_for(cfg["vocab"], [n], seed)
    rows = run_steps(make_engine(d, "float32", 16, 8, device=device, max_num_seqs=1), cases.last_one_by_one(reqs, tail=15))
    return torch.stack([rows[("r0", i)] for i in range(n)]), c, w, reqs["r0"]


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda:0", marks=GPU)])
@pytest.mark.parametrize("what", list(ALONE))
def test_mechanism_alone(tmp_path, device, what):
    got, c, w, toks = _whole_logits(tmp_path, ALONE[what], device)
    assert rel_err(got, plain.forward(c, w, toks)) < FP32_TOL


def _weights(tensors, names, change):
    return {k: (change(v) if any(k.endswith(n) for n in names) else v) for k, v in tensors.items()}


def _memory_walk_without_a_floor(q, k, v, i, f):
    S, n, out = torch.zeros(q.shape[1], v.shape[1], dtype=torch.float64), torch.zeros(q.shape[1], dtype=torch.float64), torch.zeros_like(v)
    for t in range(q.shape[0]):
        S, n = torch.exp(f[t]) * S + torch.exp(i[t]) * torch.outer(k[t], v[t]), torch.exp(f[t]) * n + torch.exp(i[t]) * k[t]
        out[t] = (q[t] @ S) / ((n @ q[t]).abs() + 1e-6)
    return out


def _delta_walk(first="decay", write_first=True):
    def walk(q, k, v, g, beta):
        S = torch.zeros(q.shape[1], v.shape[1], dtype=torch.float64)
        out = torch.zeros_like(v)
        for t in range(q.shape[0]):
            if not write_first:
                out[t] = q[t] @ S
            u = beta[t] * (v[t] - k[t] @ (S if first == "read" else g[t] * S))
            S = g[t] * S + torch.outer(k[t], u)
            if write_first:
                out[t] = q[t] @ S
        return out
    return walk


def _route(worth=2, scaled=True, normed=False):
    def route(h, w, p, r):
        s = torch.sigmoid(h @ w[p + "router"].T)
        g, E = r["groups"], s.shape[1]
        size = E // g["count"]
        best = torch.topk(torch.topk(s.view(-1, g["count"], size), worth, dim=-1).values.sum(-1), g["keep"], dim=-1).indices
        kept = torch.zeros(s.shape[0], g["count"], dtype=torch.bool).scatter_(1, best, True).repeat_interleave(size, dim=1)
        chosen = torch.topk(s.masked_fill(~kept, -1.0), r["top"], dim=-1).indices
        c = torch.gather(s, 1, chosen)
        c = c / c.sum(-1, keepdim=True) if normed else c
        return chosen, c * r["scale"] if scaled else c
    return route


def _halves(x, dims, base):
    """Halves rotate instead of neighbours."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = torch.arange(x.shape[0], dtype=torch.float64).view(-1, 1, 1) * f
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), x[..., dims:]], -1)


def _patch(name, value):
    return lambda c, w, mp: (mp.setattr(plain, name, value), (c, w))[1]


def _silu_gate(h, w, p, m, eps):
    """The matrix memory with silu where its output gate has a sigmoid."""
    inner, z = _MEMORY(h, {**w, p + "o": torch.eye(m["heads"] * m["vdim"], dtype=torch.float64)}, p, m, eps), h @ w[p + "g"].T
    return (inner * z) @ w[p + "o"].T


_MEMORY = plain.matrix_memory
MISTAKES = {
    "an open output gate": lambda c, w, mp: (c, _weights(w, [".mix.g"], torch.zeros_like)),
    "silu in the memory's gate": lambda c, w, mp: (mp.setitem(plain.MIXERS, "mlstm", _silu_gate), (c, w))[1],
    "no gate biases": lambda c, w, mp: (c, _weights(w, [".mix.i.b", ".mix.f.b"], torch.zeros_like)),
    "no cap on the gates": lambda c, w, mp: ({**c, "layers": [{**l, "mixer": {**l["mixer"], "gate_cap": 1e6}} for l in c["layers"]]}, w),
    "no unit lengths": _patch("unit_vectors", lambda x: x),
    "no decay": lambda c, w, mp: (c, _weights(w, [".A_log"], lambda v: v - 60.0)),
    "no decay bias": lambda c, w, mp: (c, _weights(w, [".dt_bias"], torch.zeros_like)),
    "the correction before the decay": _patch("delta_walk", _delta_walk(first="read")),
    "the read before the write": _patch("delta_walk", _delta_walk(write_first=False)),
    "the convolution's taps turned round": lambda c, w, mp: (c, _weights(w, [".conv"], lambda v: v.flip(1))),
    "no convolution": lambda c, w, mp: (c, _weights(w, [".conv"], lambda v: torch.cat([torch.zeros_like(v[:, :-1]), torch.ones_like(v[:, -1:])], 1))),
    "one plus the plain gains": lambda c, w, mp: (c, _weights(w, [".left.out"], lambda v: v + 1.0)),
    "the plain norms' gains as they are": _patch("stream_norm", lambda x, w, n, eps: plain.unit_rms(x, eps) * w[n]),
    "no branch factor": lambda c, w, mp: ({**c, "residual_mult": 1.0}, w),
    "no embedding scale": lambda c, w, mp: ({**c, "embedding": {"scale": 1.0}}, w),
    "the scaled table as the head": lambda c, w, mp: (mp.setattr(plain, "forward", _scaled_head(plain.forward)), (c, w))[1],
    "halves rotate": _patch("rotate_neighbours", _halves),
    "groups by their best score": _patch("route", _route(worth=1)),
    "no scale on the weights": _patch("route", _route(scaled=False)),
    "weights that sum to the scale": _patch("route", _route(normed=True)),
    "no shared expert": lambda c, w, mp: (c, _weights(w, [".shared.down"], torch.zeros_like)),
}


def _scaled_head(inner):
    return lambda cfg, w, tokens, layer_outputs=None: inner(cfg, w, tokens, layer_outputs) * cfg["embedding"]["scale"]


@pytest.fixture(scope="module")
def everything(tmp_path_factory):
    cfg = config(56, 101, 1e-5, [(mlstm(3, 10, 14, 6.0), moe(8, 3, 20, groups=(4, 2), scale=1.7, shared=16)), (PAR, dense(24))], 0.6, 1.5)
    return _whole_logits(tmp_path_factory.mktemp("kob_all"), cfg, "cpu",
                         change=lambda t: _weights(t, [".A_log"], lambda v: v + 2.5))        # decays fast enough to show


@pytest.mark.parametrize("mistake", list(MISTAKES))
def test_a_restatement_that_is_wrong_in_one_thing_is_told_apart(everything, monkeypatch, mistake):
    got, c, w, toks = everything
    assert rel_err(got, plain.forward(c, w, toks)) < FP32_TOL
    wrong_c, wrong_w = MISTAKES[mistake](c, w, monkeypatch)
    assert rel_err(got, plain.forward(wrong_c, wrong_w, toks)) > 30 * FP32_TOL


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda:0", marks=GPU)])
def test_the_floor_under_the_memory_s_divisor(tmp_path, monkeypatch, device):
    """Input gates far below zero, behind a head norm whose eps is large: what the divisor's floor does shows."""
    cfg = config(48, 60, 0.05, [(mlstm(2, 12, 10, 8.0), None)], 1.0, 1.0)
    t = make_tensors(cfg, 91)
    t["l0.mix.i.b"][:] = -6.0
    t["l0.mix.v"] = t["l0.mix.v"] * 8
    d = write_model(cfg, str(tmp_path / "m"), 91, tensors=t)
    c, w = plain.read_model_dir(d)
    toks = cases.requests_for(60, [50], 3)["r0"]
    rows = run_steps(make_engine(d, "float32", 16, 8, device=device, max_num_seqs=1), cases.last_one_by_one({"r0": toks}, tail=15))
    got = torch.stack([rows[("r0", i)] for i in range(50)])
    assert rel_err(got, plain.forward(c, w, toks)) < FP32_TOL
    monkeypatch.setattr(plain, "memory_walk", _memory_walk_without_a_floor)
    assert rel_err(got, plain.forward(c, w, toks)) > 30 * FP32_TOL
