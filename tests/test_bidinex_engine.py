"""The Bidinex family through the engine's step function, cache manager and entry points, against the plain restatement of
tests/plain_bidinex.py: every way of cutting the same requests into steps (whole, the last tokens one by one, portions down to two
tokens, mixed batches over a pool so small that pages and slots are used again), the first tokens, long decoding, keys far away that
every later query must see, the stream after every layer run, and greedy generation through `LLM.generate`.
CPU cases run the host logic with the plain-torch kernel double; `-m gpu` cases run the CUDA kernels.

bfloat16 and routed experts.  A token whose best router scores lie closer together than bfloat16 rounding moves them may pick another
expert than the float64 restatement does, and everything after it in the request then differs by far more than rounding.  So in
bfloat16 the configurations run with softer attention scales, once with every expert chosen (`soft_variant`: nothing is left to choose,
and there the ways of cutting must also agree with one another) and once as they are; both under bounds on the median and the ninth
decile of the error.  float32 is compared at every position, with the configurations as they are."""
import copy

import pytest
import torch

import plain_bidinex as plain
import replay_cases as cases
from bidinex_models import CONFIGS, make_tensors, plant_needle, write_model
from helpers import make_engine, rel_err, run_steps

FP32_TOL, BF16_TOL = 3e-4, 5e-2
# lengths around the page sizes (16, 8, 16, 4) and the key tiles of 32
LENGTHS = {"A": [1, 15, 16, 17, 33, 70], "B": [2, 8, 31, 32, 33, 97], "C": [3, 16, 40, 65], "D": [7, 15, 16, 17, 70, 130]}

GPU = pytest.mark.gpu
CASES = [pytest.param("cpu", "float32", n, id=f"cpu-fp32-{n}") for n in "ABCD"] + \
        [pytest.param("cuda:0", dt, n, marks=GPU, id=f"gpu-{dt}-{n}") for dt in ("float32", "bfloat16") for n in "ABCD"]


def soft_variant(cfg, all_experts=True):
    """Attention scales a quarter as large (a peaked softmax magnifies bfloat16's rounding of queries and keys far beyond a
    rounding-sized tolerance) and, with `all_experts`, routers that choose every expert."""
    cfg = copy.deepcopy(cfg)
    for lay in cfg["layers"]:
        lay["mixer"]["scale"] *= 0.25
        if all_experts and lay["mlp"] is not None:
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
            out[key] = write_model(c, str(tmp_path_factory.mktemp("bid_" + key)), seed)
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
                agree(rows, base, ref, tol if strict else 2e-2)
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
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_stream_after_every_layer_run(dirs, refs, device, name):
    """The residual stream behind every layer run (each pass through a repeated layer counts), with the pending branch added."""
    from iitj_llm_coopt_b200.kernels import materialize
    reqs, _ = refs(name)
    rid, toks = next((r, t) for r, t in reqs.items() if 30 <= len(t) <= 50)
    c, w = plain.read_model_dir(dirs[name])
    want = []
    plain.forward(c, w, toks, want)
    eng = make_engine(dirs[name], "float32", CONFIGS[name][2], 16, device=device, max_num_seqs=2)
    got = []

    def watched(inner):
        def forward(ctx, residual, delta, call):
            res, d = inner(ctx, residual, delta, call)
            got.append((res + c["residual_mult"] * materialize(d).float()).double().cpu())
            return res, d
        return forward
    for block in eng.runner.model.layers:
        block.forward = watched(block.forward)
    run_steps(eng, [([(rid, toks, [])], [rid])])
    assert len(got) == len(want)
    assert max(rel_err(g, x) for g, x in zip(got, want)) < FP32_TOL


NEEDLE = 7


@pytest.mark.parametrize("device,dtype", [("cpu", "float32"), pytest.param("cuda:0", "float32", marks=GPU),
                                          pytest.param("cuda:0", "bfloat16", marks=GPU)])
@pytest.mark.parametrize("name", ["A", "C"])
def test_one_far_key_among_many(tmp_path, device, dtype, name):
    """A token whose key every later query of every layer scores far above all others stands at the start, at both sides of a page's
    border, or in the middle: the logits of all later positions hang on it, in a prompt, in portions and in single decoded tokens."""
    cfg, seed, page = CONFIGS[name]
    cfg = copy.deepcopy(cfg) if dtype == "float32" else soft_variant(cfg)
    for lay in cfg["layers"]:
        lay["mixer"]["scale"] *= 0.5 if dtype == "float32" else 2.0
    d = write_model(cfg, str(tmp_path / "m"), seed, tensors=plant_needle(cfg, make_tensors(cfg, seed), NEEDLE))
    c, w = plain.read_model_dir(d)
    total = 150 if device == "cpu" else 700
    base = [t if t != NEEDLE else NEEDLE + 1 for t in cases.requests_for(cfg["vocab"], [total], seed)["r0"]]
    without = plain.forward(c, w, base)
    eng = make_engine(d, dtype, page, -(-total // page) + 1, device=device, max_num_seqs=2, max_num_batched_tokens=total)
    for at in (0, page - 1, page, total // 2 - 1):
        toks = base[:at] + [NEEDLE] + base[at + 1:]
        ref = plain.forward(c, w, toks)
        moved = (ref - without)[at + 1:].abs().amax(dim=1) / ref.abs().max()
        assert moved.median() > 0.1                                  # the needle decides what comes behind it
        reqs = {"r0": toks}
        for steps in (cases.whole(reqs), cases.last_one_by_one(reqs, tail=10), cases.portions(reqs)):
            rows = run_steps(eng, steps)
            compare(rows, {"r0": ref.float()}, reqs, FP32_TOL if dtype == "float32" else BF16_TOL, dtype == "float32")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B"])
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
    assert max(rel_err(b[k], a[k]) for k in a) < 1e-5


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
def test_command_line_serves_a_model_folder(dirs, tmp_path):
    """The serving command line on a Bidinex folder (continuous batching under a small token budget, float32, greedy): every request's
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
    proc = subprocess.run([sys.executable, "-m", "iitj_llm_coopt_b200.cli", "--shape", "bidinex-toy", "--random-seed", "5", "--workload",
                           "synthetic:10:4-300:3-20", "--out", str(out), "--num-pages", "128", "--max-num-seqs", "4",
                           "--max-num-batched-tokens", "64", "--save-tokens"], cwd=root, capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    res = json.loads(out.read_text())
    assert res["summary"]["completed"] == 10 and res["summary"]["failed"] == 0
    assert all(len(r["token_ids"]) == r["output_tokens"] == r["max_tokens"] for r in res["requests"])


# ---- each mechanism alone, and restatements that are wrong in one thing -------------------------------------------------
def one(mlp=True, loop=None, softcap=None, scale=1.0, mult=1.0, groups=(4, 2)):
    from bidinex_models import config, latent, layer, moe
    return config(56, 101, 1e-5, [layer(latent(3, 10, 6, 14, 18, 0.6, base=100.0), moe(8, 3, 20, groups=groups) if mlp else None)], mult, scale,
                  loop=loop, softcap=softcap)


ALONE = {"attention": one(mlp=False), "experts": one(), "experts of any group": one(groups=None), "join": one(mlp=False, loop=(0, 1, 1)),
         "repeated layer": one(mlp=False, loop=(0, 1, 4)), "cap": one(mlp=False, softcap=3.0), "embedding scale": one(mlp=False, scale=0.4),
         "branch factor": one(mult=0.35)}


def _whole_logits(tmp_path, cfg, device, seed=71, n=60):
    d = write_model(cfg, str(tmp_path / "m"), seed)
    c, w = plain.read_model_dir(d)
    reqs = cases.requests_for(cfg["vocab"], [n], seed)
    rows = run_steps(make_engine(d, "float32", 16, 8, device=device, max_num_seqs=1), cases.last_one_by_one(reqs, tail=15))
    return torch.stack([rows[("r0", i)] for i in range(n)]), c, w, reqs["r0"]


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda:0", marks=GPU)])
@pytest.mark.parametrize("what", list(ALONE))
def test_mechanism_alone(tmp_path, device, what):
    got, c, w, toks = _whole_logits(tmp_path, ALONE[what], device)
    assert rel_err(got, plain.forward(c, w, toks)) < FP32_TOL


def _drop(tensors, names, value):
    return {k: (torch.full_like(v, value) if any(k.endswith(n) for n in names) else v) for k, v in tensors.items()}


def _wrong_pairs(v, dims, base):
    """Neighbours rotate instead of halves."""
    T = v.shape[0]
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = torch.arange(T, dtype=torch.float64).view(T, 1, 1) * f.view(1, 1, -1)
    out, e, o = v.clone(), v[..., 0:dims:2], v[..., 1:dims:2]
    out[..., 0:dims:2], out[..., 1:dims:2] = e * torch.cos(a) - o * torch.sin(a), o * torch.cos(a) + e * torch.sin(a)
    return out


MISTAKES = {
    "a gate that is always open by half": lambda c, w, mp: (c, _drop(w, [".mix.g"], 0.0)),
    "no shift in the norms": lambda c, w, mp: (c, _drop(w, ["norm1.b", "norm2.b", "final.norm.b", "embed.norm.b"], 0.0)),
    "alpha of one": lambda c, w, mp: (c, _drop(w, [".alpha"], 1.0)),
    "no norm of the latent row": lambda c, w, mp: (mp.setattr(plain, "rms_norm", lambda x, g, e: x * g), (c, w))[1],
    "no cap": lambda c, w, mp: ({**c, "logit_softcap": None}, w),
    "no embedding scale": lambda c, w, mp: ({**c, "embedding": {"scale": 1.0}}, w),
    "no branch factor": lambda c, w, mp: ({**c, "residual_mult": 1.0}, w),
    "one pass too few": lambda c, w, mp: ({**c, "loop": {**c["loop"], "times": c["loop"]["times"] - 1}}, w),
    "the join's halves swapped": lambda c, w, mp: (mp.setattr(plain, "enter_pass", lambda x, x0, w_: torch.cat([x0, x], -1) @ w_["loop.in"].T), (c, w))[1],
    "the join at the first pass alone": lambda c, w, mp: (mp.setattr(plain, "run_order", lambda c_: [(0, True), (0, False), (0, False)]), (c, w))[1],
    "the join from the second pass on": lambda c, w, mp: (mp.setattr(plain, "run_order", lambda c_: [(0, False), (0, True), (0, True)]), (c, w))[1],
    "neighbours rotate": lambda c, w, mp: (mp.setattr(plain, "rotate_halves", _wrong_pairs), (c, w))[1],
    "every group open": lambda c, w, mp: (mp.setattr(plain, "route", _route_variant(groups=False)), (c, w))[1],
    "weights as they are": lambda c, w, mp: (mp.setattr(plain, "route", _route_variant(normed=False)), (c, w))[1],
}


def _route_variant(groups=True, normed=True):
    inner = plain.route

    def route(h, w, p, r):
        r = r if groups else {**r, "groups": None}
        chosen, weights = inner(h, w, p, r)
        if not normed:
            weights = torch.gather(torch.softmax(h @ w[p + "router"].T, dim=-1), 1, chosen)
        return chosen, weights
    return route


@pytest.fixture(scope="module")
def everything(tmp_path_factory):
    return _whole_logits(tmp_path_factory.mktemp("bid_all"), one(loop=(0, 1, 3), softcap=8.0, scale=0.5, mult=0.6), "cpu")


@pytest.mark.parametrize("mistake", list(MISTAKES))
def test_a_restatement_that_is_wrong_in_one_thing_is_told_apart(everything, monkeypatch, mistake):
    got, c, w, toks = everything
    assert rel_err(got, plain.forward(c, w, toks)) < FP32_TOL
    wrong_c, wrong_w = MISTAKES[mistake](c, w, monkeypatch)
    assert rel_err(got, plain.forward(wrong_c, wrong_w, toks)) > 30 * FP32_TOL
