"""Refolix without a GPU: configuration, description, tensor names, cache layout, the rotation's frequencies, and the plain
implementation's own mechanisms against closed forms."""

import copy
import math

import pytest
import torch

from llm_runtime_study_b200.config import RefolixConfig, architecture_for
from llm_runtime_study_b200.errors import ConfigError
from llm_runtime_study_b200.models.description import tensor_schema
from llm_runtime_study_b200.models.model import DecoderModel
from llm_runtime_study_b200.models.refolix import describe_refolix
from llm_runtime_study_b200.parts import FEED_FORWARDS, FixedState, Runtime
from llm_runtime_study_b200.parts.rope import RotaryEmbedding
from tests import helpers
from tests.plain import refolix_plain as plain


def test_the_registry_finds_the_design_by_its_architecture_key():
    assert architecture_for(helpers.REFOLIX_A).name == "Refolix"


def test_every_size_and_constant_is_read_from_the_dict():
    cfg = RefolixConfig.from_dict(helpers.REFOLIX_A)
    assert (cfg.vocab, cfg.width, cfg.eps, len(cfg.layers)) == (211, 64, 1e-5, 4)
    assert (cfg.postln_alpha, cfg.embedding_scale, cfg.logit_scale, cfg.logit_softcap) == (1.7, 2.5, 0.8, 3.0)
    left, right = cfg.layers[0].mixer.left, cfg.layers[0].mixer.right
    assert (left.heads, left.kv_heads, left.dim, left.vdim, left.scale, left.softcap, left.window) == (3, 1, 24, 20, 0.4, 2.0, 5)
    s = left.rot.scaling
    assert (left.rot.base, left.rot.dims, s.factor, s.original, s.fast, s.slow) == (500.0, 12, 4.0, 64.0, 8.0, 1.0)
    assert (right.heads, right.kv_heads, right.dim, right.vdim, right.conv) == (6, 2, 12, 10, 4)
    keep = cfg.layers[1]
    assert keep.mlp is None and keep.mixer.decay == (0.5, 0.97, 1.0) and (keep.mixer.rot.base, keep.mixer.rot.dims) == (100.0, 8)
    mlp = cfg.layers[0].mlp
    assert (mlp.experts, mlp.top, mlp.ff, mlp.groups, mlp.keep, mlp.shared_ff) == (9, 3, 24, 3, 2, 40)
    other = RefolixConfig.from_dict(helpers.REFOLIX_B)
    assert other.logit_softcap is None and other.layers[1].mlp.shared_ff is None and other.layers[1].mixer.left.window == 1


@pytest.mark.parametrize("patch,match", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("postln_alpha"), "postln_alpha"),
    (lambda c: c.__setitem__("logit_softcap", 0), "logit_softcap"),
    (lambda c: c.__setitem__("width", True), "width must be int, got bool"),
    (lambda c: c["layers"][0].__setitem__("type", "attention"), "not a layer of this design"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][0]["mixer"]["left"].__setitem__("kv_heads", 2), "not a multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"].__setitem__("softcap", -1), "softcap"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].__setitem__("size", 0), "mask.size"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].__setitem__("dims", 26), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].__setitem__("dims", 7), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][0]["mixer"]["right"].__setitem__("conv", 0), "conv"),
    (lambda c: c["layers"][1]["mixer"].__setitem__("decay", [0.5]), "one number per head"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "not a feed-forward of this design"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].__setitem__("count", 4), "do not fit"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].__setitem__("keep", 4), "do not fit"),
    (lambda c: c["layers"][2]["mlp"]["router"].__setitem__("top", 4), "exceeds"),
    (lambda c: c.__setitem__("layers", []), "layers must not be empty"),
])
def test_a_bad_config_is_refused_with_the_key_named(patch, match):
    raw = copy.deepcopy(helpers.REFOLIX_A)
    patch(raw)
    with pytest.raises(ConfigError, match=match):
        RefolixConfig.from_dict(raw)


def test_tensor_names_and_shapes_follow_the_description():
    schema = tensor_schema(describe_refolix(RefolixConfig.from_dict(helpers.REFOLIX_A)))
    assert schema["embed"].shape == (211, 64) and schema["head"].shape == (211, 64) and schema["final.norm"].shape == (64,)
    for name in ("norm1", "norm2", "ls1", "ls2", "mix.left.out", "mix.right.out"):
        assert schema[f"l0.{name}"].shape == (64,)
    assert "l1.norm2" not in schema and "l1.ls2" not in schema and schema["l1.ls1"].shape == (64,)
    assert schema["l0.mix.left.q"].shape == (72, 64) and schema["l0.mix.left.v"].shape == (20, 64) and schema["l0.mix.left.o"].shape == (64, 60)
    assert schema["l0.mix.left.q.norm"].shape == (24,) and schema["l0.mix.left.k.norm"].shape == (24,)
    assert schema["l0.mix.right.k"].shape == (24, 64) and schema["l0.mix.right.v.conv"].shape == (60, 4)
    assert schema["l0.mix.right.a"].shape == (6, 64) and schema["l0.mix.right.dt_bias"].shape == (6,) and schema["l0.mix.right.A_log"].shape == (6,)
    assert schema["l0.mix.right.g"].shape == (60, 64) and schema["l0.mix.right.norm"].shape == (10,) and "l0.mix.right.a1" not in schema
    assert schema["l2.mix.g"].shape == (40, 64) and schema["l2.mix.o"].shape == (64, 40) and "l2.mix.norm" not in schema
    assert schema["l0.mlp.router"].shape == (9, 64) and schema["l0.mlp.correction"].shape == (9,) and schema["l0.mlp.shared.sg"].shape == (1, 64)
    assert schema["l0.mlp.e8.down"].shape == (64, 24) and "l0.mlp.e9.down" not in schema and "l0.mlp.router.b" not in schema
    assert "l1.mlp.shared.sg" not in tensor_schema(describe_refolix(RefolixConfig.from_dict(helpers.REFOLIX_B)))


def test_the_cache_layout_comes_from_the_mixers():
    model = DecoderModel(describe_refolix(RefolixConfig.from_dict(helpers.REFOLIX_A)))
    layout = model.cache_layout()
    needs = {group.requirement.window: group.requirement.tensors for group in layout.groups}
    assert needs == {5: (("keys", (1, 24)), ("values", (1, 20))), 33: (("keys", (2, 10)), ("values", (2, 16)))}
    states = {(s.layer, s.requirement.name): s.requirement for s in layout.states}
    assert states[(0, "right.state")] == FixedState((6, 12, 10), torch.float32, "right.state")
    assert states[(0, "right.conv")].shape == (3, 108) and states[(3, "right.conv")].shape == (1, 120)
    assert states[(1, "state")].shape == (3, 20, 12)
    assert model.graph_safe()


def test_scores_over_all_outputs_belong_together():
    base = {"kind": "routed_experts", "hidden_size": 8, "intermediate_size": 4, "experts": 4, "top": 2, "act": "silu_glu", "router_bias": False}
    FEED_FORWARDS.build({**base, "score": "sigmoid_all", "correction": True, "groups": 2, "keep": 1, "group_best": 2, "renormalise": True})
    for wrong in ({"score": "sigmoid", "renormalise": True}, {"score": "sigmoid_all", "group_best": 3}, {"score": "sigmoid", "groups": 2}):
        with pytest.raises(ValueError):
            FEED_FORWARDS.build({**base, **wrong})


@pytest.mark.parametrize("dims,base,scaling", [
    (16, 250.0, {"factor": 8.0, "original": 512, "fast": 32.0, "slow": 1.0}),
    (12, 500.0, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}),
    (8, 50.0, {"factor": 3.0, "original": 4, "fast": 900.0, "slow": 800.0}),       # both ends below pair 0: every pair divided
    (2, 100.0, {"factor": 2.0, "original": 64, "fast": 4.0, "slow": 4.0}),
    (10, 7.0, None),
])
def test_stretched_frequencies(dims, base, scaling):
    rope = RotaryEmbedding(dims + 4, base, dims, scaling=scaling, interleaved=True)
    rope.load({}, Runtime(torch.device("cpu"), torch.float32))
    inv_freq, rotary_dim, interleaved, factor = rope.rotary_layout()
    want, want_factor = plain.frequencies(dims, base, scaling)
    assert rotary_dim == dims and interleaved and abs(factor - want_factor) < 1e-12
    assert torch.allclose(inv_freq.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6, atol=0)


def test_the_plain_rotations():
    x = torch.tensor([[[9.0, 9.0, 9.0, 9.0, 9.0]], [[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=torch.float64)
    c, s = 2 * math.cos(0.5), 2 * math.sin(0.5)
    e, t = 2 * math.cos(0.25), 2 * math.sin(0.25)
    y = plain.rotate(x, [0.5, 0.25], 2.0, interleaved=True)[1, 0]
    assert torch.allclose(y, torch.tensor([c - 2 * s, 2 * c + s, 3 * e - 4 * t, 4 * e + 3 * t, 5.0], dtype=torch.float64))
    y = plain.rotate(x, [0.5, 0.25], 2.0, interleaved=False)[1, 0]
    assert torch.allclose(y, torch.tensor([c - 3 * s, 2 * e - 4 * t, 3 * c + s, 4 * e + 2 * t, 5.0], dtype=torch.float64))
    assert torch.allclose(plain.rotate(x, [0.5, 0.25], 2.0, interleaved=True)[0, 0], torch.tensor([18.0, 18.0, 18.0, 18.0, 9.0], dtype=torch.float64))


def test_the_plain_window_and_cap():
    assert plain.window_mask(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]]
    # equal scores: the mean of the visible values; scores far apart: the cap leaves e^(2 cap) between the largest and the smallest
    v = torch.tensor([3.0, 6.0, 12.0], dtype=torch.float64).view(3, 1, 1)
    zero = torch.zeros(3, 1, 2, dtype=torch.float64)
    assert plain.window_attention(zero, zero, v, scale=1.0, cap=5.0, size=2)[:, 0, 0].tolist() == [3.0, 4.5, 9.0]
    q = torch.tensor([1.0, 1.0], dtype=torch.float64).view(2, 1, 1)
    k = torch.tensor([-1e6, 1e6], dtype=torch.float64).view(2, 1, 1)
    out = plain.window_attention(q, k, v[:2], scale=1.0, cap=0.5, size=None)
    assert abs(float(out[1, 0, 0]) - (3 + 6 * math.e) / (1 + math.e)) < 1e-12


def test_the_plain_delta_rule_overwrites():
    """With no decay and beta 1 a unit key's value is replaced, not added to; the read-out sees the current write; a decay acts
    ahead of the correction."""

    k = torch.tensor([[1.0, 0.0], [0.0, 1.0], [1.0, 0.0]], dtype=torch.float64).view(3, 1, 2)
    v = torch.tensor([5.0, 7.0, 11.0], dtype=torch.float64).view(3, 1, 1)
    one = torch.ones(3, 1, dtype=torch.float64)
    assert plain.delta_scan(k, k, v, one, one)[:, 0, 0].tolist() == [5.0, 7.0, 11.0]
    out = plain.delta_scan(torch.ones_like(k), k, v, 0.5 * one, 0.5 * one)[:, 0, 0].tolist()
    # S: (2.5, 0); (1.25, 3.5); first halved to 0.625, then + 0.5 (11 - 0.625)
    assert out == [2.5, 4.75, 0.625 + 0.5 * 10.375 + 1.75]
    z = torch.tensor([-700.0, 0.0, 700.0], dtype=torch.float64)
    g = plain.head_decay(z, torch.tensor(0.0, dtype=torch.float64), torch.tensor(0.0, dtype=torch.float64))
    assert torch.allclose(g, torch.tensor([1.0, 0.5, 0.0], dtype=torch.float64))


def test_the_plain_retention_and_convolution():
    k = torch.tensor([1.0, 1.0, 0.0], dtype=torch.float64).view(3, 1, 1)
    v = torch.tensor([8.0, 2.0, 100.0], dtype=torch.float64).view(3, 1, 1)
    assert plain.retention_scan(torch.ones_like(k), k, v, [0.25])[:, 0, 0].tolist() == [8.0, 4.0, 1.0]
    x = torch.tensor([[1.0], [10.0], [100.0]], dtype=torch.float64)
    assert plain.short_convolution(x, torch.tensor([[3.0, 2.0, 1.0]], dtype=torch.float64))[:, 0].tolist() == [1.0, 12.0, 123.0]


def test_the_plain_router_scores_a_group_by_its_two_best():
    """The first group holds the single best expert, the second the best pair; the weights know no correction; a group that is
    not kept cannot be chosen even where every choice score that remains is negative."""

    s = torch.tensor([0.9, 0.1, 0.2, 0.6, 0.7, 0.3], dtype=torch.float64)
    z = torch.log(s / (1 - s)).unsqueeze(0)
    none = torch.zeros(6, dtype=torch.float64)
    chosen, w = plain.route(z, none, top=2, groups=2, keep_groups=1)
    assert chosen.tolist() == [[4, 3]] and torch.allclose(w, torch.tensor([[0.7 / 1.3, 0.6 / 1.3]], dtype=torch.float64))
    assert plain.route(z, none, top=2, groups=2, keep_groups=2)[0].tolist() == [[0, 4]]
    low = torch.tensor([-5.0, -5.0, -5.0, -4.0, -4.0, -9.0], dtype=torch.float64)
    chosen, w = plain.route(z, low, top=3, groups=2, keep_groups=1)
    assert chosen.tolist() == [[4, 3, 5]] and torch.allclose(w, torch.tensor([[0.7, 0.6, 0.3]], dtype=torch.float64) / 1.6)


def test_the_plain_norm_behind_the_sum():
    x = plain.layer_norm(torch.tensor([[1.0, 3.0, 5.0, 7.0]], dtype=torch.float64), torch.tensor([1.0, 2.0, 1.0, 1.0], dtype=torch.float64), 4.0)
    assert torch.allclose(x, torch.tensor([[-1.0, -2.0 / 3, 1.0 / 3, 1.0]], dtype=torch.float64))       # variance 5, plus 4: a root of 3
