"""Kobolix's configuration, its layers and run order as data, its checkpoint names, and the trace replay's protocol on a Kobolix
folder (CPU)."""
import copy
import io
import json
import os

import numpy as np
import pytest

import plain_kobolix as plain
from kobolix_models import CONFIGS, KOB_A, KOB_B, KOB_C, KOB_D, make_tensors, write_model

from iitj_llm_coopt_b200.config import ConfigError, load_config
from iitj_llm_coopt_b200.config.kobolix import KobolixConfig
from iitj_llm_coopt_b200.models.decoder import cache_needs
from iitj_llm_coopt_b200.parts.delta_rule import record as delta_record
from iitj_llm_coopt_b200.parts.matrix_memory import record as memory_record
from iitj_llm_coopt_b200.weights.loader import WeightError, expected_tensors


def test_layers_as_data(tmp_path):
    arch, typed = load_config(write_model(KOB_A, str(tmp_path / "m"), 1))
    assert arch.name == "Kobolix"
    spec = typed.model_spec()
    assert [c.layer for c in spec.order] == [0, 1, 2, 3]
    assert [(c.cache, c.state) for c in spec.order] == [(0, None), (1, 2), (3, None), (4, 5)] and all(c.write for c in spec.order)
    assert [l.arrangement for l in spec.layers] == ["prenorm", "prenorm", "prenorm_mixer", "prenorm"]
    needs = cache_needs(spec)
    assert [n.kind for n in needs] == ["state", "paged_kv", "state", "state", "paged_kv", "state"]
    assert needs[0].state_shape == (memory_record(3, 12, 20),) and needs[2].state_shape == (delta_record(4, 2, 12, 10, 3),)
    assert memory_record(3, 12, 20) == 760 and memory_record(1, 7, 5) == 52        # 3 * 21 * 12 + 3, 6 * 8 + 1, up to a multiple of four
    assert delta_record(4, 2, 12, 10, 3) == 4 * 10 * 12 + 3 * (48 + 40)
    assert (needs[1].kv_heads, needs[1].head_dim, needs[1].value_dim, needs[1].window) == (2, 16, 24, 0)
    m = spec.layers[0].part("mixer")
    assert (m.kind, m.heads, m.head_dim, m.value_dim, m.option("gate_cap")) == ("matrix_memory", 3, 12, 20, 5.0)
    p = spec.layers[1].part("mixer")
    left, right = p.option("left"), p.option("right")
    assert p.kind == "parallel" and p.option("scale") == 0.5 and p.position == left.position
    assert (left.softmax_scale, left.position.pairing, left.position.rotary_dim, left.position.theta) == (0.8, "interleaved", 8, 1000.0)
    assert (right.kind, right.heads, right.kv_heads, right.head_dim, right.value_dim, right.option("conv_taps")) == ("gated_delta", 4, 2, 12, 10, 3)
    f = spec.layers[1].part("feed_forward")
    assert (f.kind, f.experts, f.experts_per_token, f.inner) == ("routed_glu", 6, 2, 20)
    assert [f.option(k) for k in ("groups", "group_worth", "weight_scale", "shared", "router")] == [(3, 2), 2, 1.3, 28, "sigmoid"]
    assert spec.layers[0].part("feed_forward").kind == "swiglu"
    norm = spec.layers[0].part("mixer_norm")
    assert norm.kind == "rmsnorm_one_plus" and dict(norm.options)["branch_factor"] == 0.6 and spec.final_norm == norm
    assert spec.tie_embeddings and spec.embedding.scale == 2.0
    b = KobolixConfig.from_dict(KOB_B).model_spec()
    assert b.layers[0].part("mixer").position is None and b.embedding.scale == 1.0
    assert dict(b.layers[0].part("mixer_norm").options)["branch_factor"] == 1.0
    f = b.layers[0].part("feed_forward")
    assert [f.option(k) for k in ("groups", "weight_scale", "shared")] == [None, 1.0, 0]
    for cfg in (KOB_A, KOB_B, KOB_C, KOB_D):
        assert KobolixConfig.from_dict(KobolixConfig.from_dict(cfg).to_dict()).model_spec() == KobolixConfig.from_dict(cfg).model_spec()


def test_optional_keys_may_be_null():
    cfg = copy.deepcopy(KOB_A)
    cfg.update(embedding=None, residual_mult=None)
    cfg["layers"][1]["mixer"]["left"]["rot"] = None
    cfg["layers"][1]["mlp"]["router"].update(groups=None, scale=None)
    cfg["layers"][1]["mlp"]["shared"] = None
    spec = KobolixConfig.from_dict(cfg).model_spec()
    assert spec.layers[1].part("mixer").position is None
    assert [spec.layers[1].part("feed_forward").option(k) for k in ("groups", "weight_scale", "shared")] == [None, 1.0, 0]


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
    (lambda c: c["norm"].update(eps=0), "eps"),
    (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c["layers"][0].update(type="attention"), "not known"),
    (lambda c: c["layers"][0]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda c: c["layers"][0]["mixer"].update(gate_cap=0), "gate_cap"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=0), "positive"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"]["right"].pop("conv"), "conv"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["left"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mlp"].update(kind="glu"), "mlp.kind"),
    (lambda c: c["layers"][0]["mlp"].pop("ff"), "ff"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "router takes"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "router takes"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "groups"),
    (lambda c: c["layers"][1]["mlp"]["shared"].update(ff=0), "positive"),
])
def test_bad_configurations_are_refused(change, text):
    cfg = copy.deepcopy(KOB_A)
    change(cfg)
    with pytest.raises(ConfigError, match=text):
        KobolixConfig.from_dict(cfg)


def test_missing_and_unexpected_tensors_are_listed(tmp_path):
    from helpers import make_engine
    t = make_tensors(KOB_A, 1)
    t["l1.mlp.e6.up"] = t["l1.mlp.e5.up"].clone()               # the layer has six experts: e0 .. e5
    t["l2.norm2"] = t["l2.norm1"].clone()                       # the layer has no feed-forward
    t["head"] = t["embed"].clone()                              # the embedding's table is the head
    del t["l0.mix.f.b"], t["l1.mix.right.dt_bias"], t["l1.mlp.shared.down"], t["l3.mix.left.out"]
    with pytest.raises(WeightError) as e:
        make_engine(write_model(KOB_A, str(tmp_path / "m"), 1, tensors=t), "float32", device="cpu")
    assert e.value.missing == ["l0.mix.f.b", "l1.mix.right.dt_bias", "l1.mlp.shared.down", "l3.mix.left.out"]
    assert e.value.unexpected == ["head", "l1.mlp.e6.up", "l2.norm2"]


def test_the_step_s_plan_of_walks_and_chunks():
    """Which requests of a step go by chunks, and where their chunks lie."""
    from types import SimpleNamespace

    from iitj_llm_coopt_b200.parts.base import StepShape
    from iitj_llm_coopt_b200.parts.state_plan import plan_state_chunks
    k = SimpleNamespace(STATE_CHUNK=64, state_chunk_from=64)
    plan = plan_state_chunks(k, StepShape([5, 130, 1, 64, 63], [9, 130, 7, 70, 63], 263, False, False, "cpu"))
    assert plan.arrays["walks"] == [0, 2, 4]
    assert plan.arrays["chunks"] == [1, 5, 64, 0, 1, 69, 64, 1, 1, 133, 2, 2, 3, 136, 64, 0]
    assert plan.arrays["longs"] == [1, 0, 3, 3, 3, 1] and plan.counts == plan.graph_key == (3, 4, 2)
    assert plan_state_chunks(k, StepShape([1, 1], [4, 5], 2, True, True, "cpu")) is None
    assert plan_state_chunks(SimpleNamespace(), StepShape([90], [90], 90, False, False, "cpu")) is None
    short = plan_state_chunks(k, StepShape([3, 1], [4, 5], 4, False, False, "cpu"))
    assert short.arrays["walks"] == [0, 1] and short.counts == (2, 0, 0) and len(short.arrays["chunks"]) == 1


def test_trace_replay_protocol(tmp_path):
    """bin/trace_run's program on a Kobolix folder (CPU kernel double): files only for steps that want something, a `done` line after
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
        ref = torch_stack(rows)
        assert np.abs(got[s] - ref).max() <= 1e-4 * np.abs(ref).max()


def torch_stack(rows):
    import torch
    return torch.stack(rows).float().numpy()
