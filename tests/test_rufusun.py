"""Rufusun on CPU: configuration and tensor names, coverage, and that the plain evaluation the GPU tests compare
with would show the faults they look for."""
import json

import numpy as np
import pytest

from dyninfer_b200 import checkpoint as ck, registry as reg, rufusun, synth
from dyninfer_b200.runtime import DynInferError, ModelLoader
import rufusun_cases as cases
import rufusun_ref as ref


def test_catalog_lists_runs_and_reads_every_size(tmp_path):
    doc = cases.mixed()
    cat = ck.open_catalog(synth.write_rufusun(str(tmp_path / "m"), doc, seed=1))
    c = cat.config
    assert (c["layers"], c["hidden"], c["vocab"], c["tied"]) == (9, 44, 101, False) and c["eps"] == 1e-5
    assert c["norm_offset"] == 1.0 and c["logit_scale"] == 0.7
    assert [m["tensors"] for m in c["mixers"]] == [0, 1, 2, 3, 1, 2, 3, 7, 8]
    assert c["mixers"][4] == {"type": "gated_delta", "tensors": 1, "ff": 0, "parallel": 1, "heads": 4, "kv_heads": 2, "dim": 12,
                              "vdim": 20, "taps": 3, "experts": 5, "top": 2, "expert_ff": 28, "expert_limit": 0.8,
                              "shared_ff": 36, "shared_limit": 1.7}
    assert c["mixers"][8]["rot_dims"] == 4 and c["mixers"][8]["softcap"] == 30.0 and c["mixers"][8]["scale"] == 0.3
    assert c["kv_elements_per_token"] == 2 * 32 + 2 * 5 * 36 + 28          # every run caches
    delta = lambda h, g, d, e, t: h * d * e + t * (2 * g * d + h * e)      # noqa: E731
    assert c["state_bytes_per_slot"] == 4 * (2 * delta(4, 2, 12, 20, 3) + 2 * delta(3, 1, 28, 8, 5) + delta(2, 2, 16, 24, 1))
    assert set(cat.parameters) == set(rufusun.tensor_names(doc).values()) and len(cat.parameters) == len(synth.rufusun_shapes(doc))
    assert cat.parameters["blk.1.expert_4_down.weight"].shape == (44, 28) and cat.parameters["blk.7.attn_q.weight"].shape == (32, 44)
    assert not any(p.startswith(("blk.4.", "blk.5.", "blk.6.")) for p in cat.parameters)
    assert len(ck.build_runtime_provider_plan(cat).parameters) == len(cat.parameters)


@pytest.mark.parametrize("loop, order", [(None, [0, 1, 2]), (cases.span(0, 2, 2), [0, 1, 0, 1, 2]), (cases.span(2, 3, 3), [0, 1, 2, 2, 2]),
                                         (cases.span(1, 1, 4), [0, 1, 2]), (cases.span(0, 3, 1), [0, 1, 2])])
def test_run_order(loop, order):
    doc = cases.model([cases.delta()] * 3, loop=loop)
    assert rufusun.run_order(doc) == order == ref.run_order(doc)
    assert rufusun.first_runs(doc) == {i: order.index(i) for i in range(3)}


def test_bad_checkpoints_are_refused(tmp_path):
    doc = cases.model([cases.delta(mlp=cases.moe())])
    path = synth.write_rufusun(str(tmp_path / "m"), doc)
    t = cases.weights(doc)
    del t["l0.mlp.e3.up"]
    with pytest.raises(ck.CheckpointError, match="lacks tensor l0.mlp.e3.up"):
        ck.open_catalog(synth.write_rufusun(str(tmp_path / "missing"), doc, tensors=t))
    layer = doc["layers"][0]
    for change, match in (({"layers": [dict(layer, type="conv")]}, "unknown mixer"), ({"width": None}, "config.json"),
                          ({"loop": cases.span(0, 2, 2)}, "loop of layers"), ({"layers": [dict(layer, mlp={"kind": "other"})]}, "feed-forward"),
                          ({"layers": [dict(layer, mlp=cases.moe(3, 4))]}, "4 of 3 experts")):
        with open(f"{path}/config.json", "w") as f:
            json.dump(dict(doc, architecture="Rufusun", **{k: v for k, v in change.items() if k not in doc}) | change, f)
        with pytest.raises(ck.CheckpointError, match=match):
            ck.open_catalog(path)


def test_every_operation_is_covered_in_both_modes(tmp_path):
    loader = ModelLoader()
    cat = loader.bind(synth.write_rufusun(str(tmp_path / "m"), cases.mixed()))
    rep = loader.kernel_coverage(cat, loader.resolve_target("cuda")[0])
    assert not rep.missing
    ids = {k for _, _, k in rep.selected}
    assert {"gated_delta.cuda_sm100.f32", "attention.gqa.cuda_sm100", "short_conv.cuda_sm100.f32", "moe.choice.cuda_sm100.f32",
            "bias.cuda_sm100.f32", "plain.bf16.matmul.cuda_sm100", "plain.bf16.lm_head.cuda_sm100"} <= ids
    other = loader.kernel_coverage(cat, reg.TargetProfile.llvm_cpu_host())       # never another target's kernels
    assert {op for op, _, _ in other.missing} >= {"blk.1.delta", "blk.1.expert_choice", "blk.0.qkv_bias"}


def test_tensor_parallel_is_refused(tmp_path):
    path = synth.write_rufusun(str(tmp_path / "m"), cases.mixed())
    with pytest.raises(DynInferError, match="tensor parallelism"):
        ModelLoader().load(path, tp=(0, 2))


# ---- the plain evaluation ------------------------------------------------------------------------

def test_delta_rule_replaces_the_value_of_a_key():
    rng = np.random.default_rng(0)
    k = rng.normal(size=6)
    k /= np.linalg.norm(k)
    S = ref.delta_state(rng.normal(size=(6, 4)), k, np.arange(4.0), 0.8, 1.0)
    assert np.allclose(S.T @ k, np.arange(4.0))                        # beta 1: the key now reads its value exactly
    other = np.linalg.svd(k[None])[2][1]
    S2 = ref.delta_state(S, other, np.ones(4), 1.0, 1.0)
    assert np.allclose(S2.T @ k, np.arange(4.0))                       # and an orthogonal key does not disturb it


def test_rotation_keeps_relative_positions_and_passes_the_rest():
    rng = np.random.default_rng(1)
    a, b = rng.normal(size=10), rng.normal(size=10)
    at = lambda p, r: ref.rotate_half(a, p, 6, 50.0) @ ref.rotate_half(b, r, 6, 50.0)   # noqa: E731
    assert np.isclose(at(3, 1), at(12, 10)) and not np.isclose(at(3, 1), at(3, 2))
    assert np.array_equal(ref.rotate_half(a, 9, 6, 50.0)[6:], a[6:])


def test_convolution_is_causal_with_the_last_tap_on_the_current_token():
    x = np.arange(12.0).reshape(6, 2)
    w = np.array([[1.0, 10.0, 100.0], [2.0, 20.0, 200.0]])
    tail, out = np.zeros((2, 2)), []
    for row in x:
        out.append(ref.causal_conv(row, tail, w))
    assert np.allclose(out[0], x[0] * w[:, 2])
    assert np.allclose(out[4], x[2] * w[:, 0] + x[3] * w[:, 1] + x[4] * w[:, 2])


def test_router_keeps_the_scores_of_the_best():
    chosen, s = ref.route(np.array([1.0]), np.array([[0.1], [2.0], [-3.0], [1.0]]), 2)
    assert chosen.tolist() == [1, 3] and np.allclose(s, 1 / (1 + np.exp([-2.0, -1.0])))


def test_capped_scores_stay_inside_the_cap():
    assert np.allclose(ref.capped(np.array([0.01, -0.02]), 5.0), [0.01, -0.02], atol=1e-6)
    assert np.abs(ref.capped(np.array([1e3, -1e3]), 5.0)).max() <= 5.0


FAULTS = {
    "newest key hidden": ("visible", lambda n: np.arange(n) < max(1, n - 1)),
    "oldest key hidden": ("visible", lambda n: np.arange(n) >= (n > 1)),
    "rotation one position off": ("rotate_half", lambda v, p, d, b, f=ref.rotate_half: f(v, p + (p > 3), d, b)),
    "scores not capped": ("capped", lambda s, cap: s),
    "convolution tail dropped": ("causal_conv", lambda x, tail, w, f=ref.causal_conv: f(x, np.zeros_like(tail), w)),
    "state not decayed": ("decay", lambda a, A, dt: np.ones_like(a)),
    "state not corrected": ("delta_state", lambda S, k, v, g, beta: g * S + np.outer(k, beta * v)),
    "correction from the state before its decay": ("delta_state", lambda S, k, v, g, beta: g * S + np.outer(k, beta * (v - S.T @ k))),
    "keys of any length": ("unit", lambda x: x),
    "norm weights as they are": ("rms_norm", lambda x, w, eps: ref.rms(x, eps) * w),
    "scores renormalised": ("route", lambda h, w, top, f=ref.route: (f(h, w, top)[0], f(h, w, top)[1] / f(h, w, top)[1].sum())),
    "the next best expert": ("route", lambda h, w, top, f=ref.route: tuple(np.roll(f(h, w, top + 1)[i], -1)[:top] for i in (0, 1))),
    "experts not clamped": ("clamped_ff", lambda x, w, limit, f=ref.clamped_ff: f(x, w, 1e9)),
}


@pytest.mark.parametrize("fault", FAULTS)
def test_faults_show_in_the_logits(fault, monkeypatch):
    """Each planted fault moves the logits by far more than the tolerances of the GPU tests."""
    doc = cases.mixed()
    ids = cases.tokens(12, doc["vocab"])
    want = ref.Model(doc, cases.weights(doc)).forward(ids)
    name, wrong = FAULTS[fault]
    monkeypatch.setattr(ref, name, wrong)
    assert cases.error(ref.Model(doc, cases.weights(doc)).forward(ids), want)[4:].max() > 0.05
