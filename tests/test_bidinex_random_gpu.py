"""Bidinex configurations drawn at random from fixed seeds (layer counts, layers of different sizes, repeated runs anywhere or none, head
counts, unrotated, rotated and value sizes, latent widths, expert counts, groups and choices, layers without a feed-forward, branch
factors, embedding scales, caps, widths and vocabularies that are no multiples of 8, page sizes), each through the engine in float32
and bfloat16, whole, in portions and in mixed batches over reused pages and slots, against the plain restatement.  Sizes that are
multiples of 16 take the tensor-core attention and the streamed grouped products in bfloat16, the others the plain forms; both are drawn.

The matrices are scaled by the inverse root of their input width, so scores and activations are of order one as in a trained model:
float32 is then compared at (nearly) every position (99 positions in 100 within 3e-4 and all within 1e-2 leaves room for a router's
close call), bfloat16 by its median and ninth decile, and the ways of cutting must agree with one another (in bfloat16 only where the
routers choose every expert: a close call moves a whole request)."""
import random

import pytest
import torch

import plain_bidinex as plain
import replay_cases as cases
from bidinex_models import config, latent, layer, make_tensors, moe, write_model
from helpers import make_engine, run_steps
from test_bidinex_engine import agree, errors

pytestmark = pytest.mark.gpu


def draw(seed):
    rng = random.Random(seed)
    width = rng.choice([64, 96, 100, 128, 160, 256, 384])
    layers = []
    for _ in range(rng.randint(1, 5)):
        dim, rot = rng.choice([8, 16, 32, 48, 80]), rng.choice([2, 4, 8, 16, 64])
        m = latent(rng.choice([1, 2, 3, 5, 6, 8, 16]), dim, rot, rng.choice([8, 16, 24, 48, 80]), rng.choice([16, 32, 40, 48, 96, 128]),
                   (dim + rot) ** -0.5 * rng.choice([1.0, 1.5, 0.5]), base=rng.choice([100.0, 1e4, 1e6]))
        mlp = None
        if rng.random() < 0.85:
            count = rng.choice([1, 2, 3, 4, 5])
            experts, keep = count * rng.choice([1, 2, 3, 4]), rng.randint(1, count)
            room = experts // count * keep
            mlp = moe(experts, rng.choice([1, room, rng.randint(1, room)]), rng.choice([16, 24, 33, 64, 128]),
                      groups=rng.choice([(count, keep), None]) if keep == count else (count, keep))
        layers.append(layer(m, mlp))
    n = len(layers)
    a = rng.randrange(n)
    loop = rng.choice([None, (a, rng.randint(a + 1, n), rng.randint(1, 4)), (0, n, 2)])
    cfg = config(width, rng.choice([64, 131, 300, 1000]), rng.choice([1e-5, 1e-6]), layers, rng.choice([1.0, 0.5, 0.2]), rng.choice([1.0, 0.4, 3.0]),
                 loop=loop, softcap=rng.choice([None, 5.0, 40.0]))
    return cfg, rng.choice([4, 8, 16, 32])


def trained_like(cfg, seed):
    """Random tensors of the family's writer with every matrix scaled by the inverse root of its input width."""
    t = make_tensors(cfg, seed)
    for name, w in t.items():
        if w.dim() == 2 and name != "embed":
            f = w.float()
            t[name] = (f / f.std().clamp_min(1e-6) * w.shape[1] ** -0.5).to(torch.bfloat16).contiguous()
    return t


@pytest.mark.parametrize("seed", range(600, 616))
def test_random_configuration(tmp_path, seed):
    cfg, page = draw(seed)
    d = write_model(cfg, str(tmp_path / "m"), seed, tensors=trained_like(cfg, seed))
    c, w = plain.read_model_dir(d)
    reqs = cases.requests_for(cfg["vocab"], [1, 19, 66, 150], seed)
    ref = {rid: plain.forward(c, w, toks).float() for rid, toks in reqs.items()}
    mixed_steps, peak = cases.mixed(reqs, live=3, seed=seed, decode_tail=12)
    choice = any(l["mlp"] is not None and l["mlp"]["router"]["top"] < l["mlp"]["router"]["experts"] for l in cfg["layers"])
    for dtype, tol in (("float32", 3e-4), ("bfloat16", 5e-2)):
        eng = make_engine(d, dtype, page, max(peak // page, 1), max_num_seqs=3, max_num_batched_tokens=peak)
        base = None
        for steps in (cases.whole(reqs), cases.portions(reqs), mixed_steps):
            rows = run_steps(eng, steps)
            eng.cache.check()
            e = sorted(errors(rows, ref, reqs))
            if dtype == "float32":
                assert e[int(0.99 * (len(e) - 1))] <= tol and e[-1] <= 1e-2, (seed, e[int(0.99 * (len(e) - 1))], e[-1])
            else:
                assert e[len(e) // 2] <= tol and e[int(0.9 * (len(e) - 1))] <= 3 * tol, (seed, e[len(e) // 2], e[int(0.9 * (len(e) - 1))])
            if base is not None and (dtype == "float32" or not choice):
                agree(rows, base, ref, tol if dtype == "float32" else 2e-2)
            base = base or rows
