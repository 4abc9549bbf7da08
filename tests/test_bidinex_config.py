"""Bidinex's configuration, its layers and run order as data, its checkpoint names, and the trace replay's protocol on a Bidinex
folder (CPU)."""
import copy
import io
import json
import os

import numpy as np
import pytest
import torch

import plain_bidinex as plain
from bidinex_models import BID_A, BID_B, BID_C, BID_D, CONFIGS, make_tensors, write_model

from iitj_llm_coopt_b200.config import ConfigError, load_config
from iitj_llm_coopt_b200.config.bidinex import BidinexConfig
from iitj_llm_coopt_b200.models.decoder import cache_needs
from iitj_llm_coopt_b200.weights.loader import WeightError, expected_tensors


def test_layers_as_data(tmp_path):
    arch, typed = load_config(write_model(BID_A, str(tmp_path / "m"), 1))
    assert arch.name == "Bidinex"
    spec = typed.model_spec()
    # layers 1 and 2 twice: six runs, each with a cache entry of its own; both passes enter through the join
    assert [c.layer for c in spec.order] == [0, 1, 2, 1, 2, 3]
    assert [c.cache for c in spec.order] == list(range(6)) and all(c.write and c.state is None for c in spec.order)
    assert [c.join for c in spec.order] == [False, True, False, True, False, False]
    assert [l.arrangement for l in spec.layers] == ["prenorm", "prenorm_mixer", "prenorm", "prenorm"]
    needs = cache_needs(spec)
    assert len(needs) == 6 and all(n.kind == "paged_kv" and n.shared_value and n.window == 0 for n in needs)
    assert [(n.head_dim, n.value_dim) for n in needs] == [(32, 24), (56, 40), (20, 16), (56, 40), (20, 16), (24, 12)]
    m = spec.layers[2].part("mixer")
    assert (m.heads, m.head_dim, m.value_dim, m.softmax_scale) == (5, 6, 10, 0.6) and m.option("gate") == "head"
    assert (m.position.pairing, m.position.rotary_dim, m.position.theta) == ("half", 4, 50.0)
    f = spec.layers[2].part("feed_forward")
    assert (f.kind, f.experts, f.experts_per_token, f.inner, f.option("groups")) == ("routed_glu", 4, 3, 12, (4, 3))
    assert spec.layers[3].part("feed_forward").option("groups") is None
    norm = spec.layers[0].part("mixer_norm")
    assert norm.kind == "dynamic_tanh" and dict(norm.options)["branch_factor"] == 0.7 and spec.final_norm == norm
    assert spec.tie_embeddings and spec.embedding.scale == 1.5 and dict(spec.head.options)["softcap"] == 6.0
    c, d = BidinexConfig.from_dict(BID_C).model_spec(), BidinexConfig.from_dict(BID_D).model_spec()
    assert [x.join for x in c.order] == [True, False] and c.head.options == ()
    assert [x.join for x in d.order] == [False, False] and d.join is None
    b = BidinexConfig.from_dict(BID_B).model_spec()
    assert [x.layer for x in b.order] == [0, 1, 1, 1] and [x.join for x in b.order] == [False, True, True, True]
    for cfg in (BID_A, BID_B, BID_C, BID_D):
        assert BidinexConfig.from_dict(BidinexConfig.from_dict(cfg).to_dict()).model_spec() == BidinexConfig.from_dict(cfg).model_spec()


def test_optional_keys_may_be_null():
    cfg = copy.deepcopy(BID_D)
    cfg.update(loop=None, logit_softcap=None)
    cfg["layers"][0]["mlp"]["router"]["groups"] = None
    del cfg["embedding"]
    spec = BidinexConfig.from_dict(cfg).model_spec()
    assert spec.join is None and spec.head.options == () and spec.embedding.scale == 1.0


def test_checkpoint_names_are_the_family_s(tmp_path):
    for name, (cfg, seed, _) in CONFIGS.items():
        arch, typed = load_config(write_model(cfg, str(tmp_path / name), seed))
        want = expected_tensors(arch, arch.model_spec(typed))
        have = make_tensors(cfg, seed)
        assert set(want) == set(have)
        assert all(tuple(want[k][0]) == tuple(have[k].shape) for k in want)


@pytest.mark.parametrize("change,text", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda c: c["loop"].pop("times"), "times"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0].update(type="attention"), "not known"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"].update(heads=0), "positive"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "mlp.kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "router takes"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=3), "router takes"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "groups"),
])
def test_bad_configurations_are_refused(change, text):
    cfg = copy.deepcopy(BID_A)
    change(cfg)
    with pytest.raises(ConfigError, match=text):
        BidinexConfig.from_dict(cfg)


def test_missing_and_unexpected_tensors_are_listed(tmp_path):
    from helpers import make_engine
    t = make_tensors(BID_A, 1)
    t["l0.mlp.e6.up"] = t["l0.mlp.e5.up"].clone()               # the layer has six experts: e0 .. e5
    t["l1.norm2"] = t["l1.norm1"].clone()                       # the layer has no feed-forward
    t["head"] = t["embed"].clone()                              # the embedding's table is the head
    del t["l1.mix.g"], t["loop.in"], t["embed.norm.alpha"], t["l3.norm2.b"]
    with pytest.raises(WeightError) as e:
        make_engine(write_model(BID_A, str(tmp_path / "m"), 1, tensors=t), "float32", device="cpu")
    assert e.value.missing == ["embed.norm.alpha", "l1.mix.g", "l3.norm2.b", "loop.in"]
    assert e.value.unexpected == ["head", "l0.mlp.e6.up", "l1.norm2"]


def test_a_run_order_that_joins_needs_a_stream_join():
    import dataclasses

    from iitj_llm_coopt_b200.models.decoder import build_model
    from torch_kernels import TorchKernels
    spec = dataclasses.replace(BidinexConfig.from_dict(BID_C).model_spec(), join=None)
    with pytest.raises(ValueError, match="stream join"):
        build_model(spec, TorchKernels(), torch.float32, device="cpu")


def test_trace_replay_protocol(tmp_path):
    """bin/trace_run's program on a Bidinex folder (CPU kernel double): files only for steps that want something, a `done` line after
    every step, a request left out of a step that goes on later, two state slots that three requests share."""
    from iitj_llm_coopt_b200 import replay
    from torch_kernels import TorchKernels
    cfg, seed, page = CONFIGS["A"]
    d = write_model(cfg, str(tmp_path / "m"), seed)
    c, w = plain.read_model_dir(d)
    a, b = list(range(3, 40)), list(range(90, 111))
    lines = [json.dumps(x) for x in (
        {"step": 0, "entries": [{"id": "a", "tokens": a[:17], "want": [16]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": a[17:19], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "b", "tokens": b[2:], "want": [0, 18]}, {"id": "a", "tokens": a[19:20], "want": [0]}], "end": ["b"]},
        {"step": 3, "entries": [{"id": "c", "tokens": b, "want": [20]}, {"id": "a", "tokens": a[20:], "want": [16]}], "end": ["a", "c"]})]
    out = io.StringIO()
    args = replay.parse_args(["--model", d, "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "128",
                              "--max-requests", "2", "--device", "cpu"])
    assert replay.run(args, lines, out=out, kernels=TorchKernels()) == 0
    assert out.getvalue().split() == ["done", "0", "done", "1", "done", "2", "done", "3"]
    assert sorted(os.listdir(tmp_path / "o")) == ["0.f32", "2.f32", "3.f32"]
    ra, rb = plain.forward(c, w, a), plain.forward(c, w, b)
    got = {s: np.fromfile(tmp_path / "o" / f"{s}.f32", dtype="<f4").reshape(-1, cfg["vocab"]) for s in (0, 2, 3)}
    want = {0: [ra[16]], 2: [rb[2], rb[20], ra[19]], 3: [rb[20], ra[36]]}
    for s, rows in want.items():
        ref = torch.stack(rows).float().numpy()
        assert np.abs(got[s] - ref).max() <= 1e-4 * np.abs(ref).max()
