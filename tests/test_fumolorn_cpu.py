"""Fumolorn without a GPU: configuration, description, tensor names, cache layout, the rotation's frequencies, and the plain
implementation's own mechanisms against closed forms."""

import copy
import math

import pytest
import torch

from llm_runtime_study_b200.config import FumolornConfig, architecture_for
from llm_runtime_study_b200.errors import ConfigError, KernelError
from llm_runtime_study_b200.models.description import tensor_schema
from llm_runtime_study_b200.models.fumolorn import describe_for_checkpoint, describe_fumolorn
from llm_runtime_study_b200.models.model import DecoderModel
from llm_runtime_study_b200.parts import FixedState, PagedTensors, Runtime
from llm_runtime_study_b200.parts.rope import RotaryEmbedding
from tests import helpers
from tests.plain import fumolorn_plain as plain


def test_the_registry_finds_the_design_by_its_architecture_key():
    assert architecture_for(helpers.FUMOLORN_A).name == "Fumolorn"


def test_every_size_and_constant_is_read_from_the_dict():
    cfg = FumolornConfig.from_dict(helpers.FUMOLORN_A)
    assert (cfg.vocab, cfg.width, cfg.eps, len(cfg.layers)) == (211, 64, 1e-5, 5)
    assert (cfg.residual_mult, cfg.logit_softcap, cfg.embedding_scale) == (0.6, 4.0, 3.5)
    assert (cfg.bigram.buckets, cfg.bigram.mul_prev, cfg.bigram.mul_cur) == (13, 40_000_003, 11)
    memory, latent, linear, _, second = (layer.mixer for layer in cfg.layers)
    assert (memory.heads, memory.dim, memory.vdim, memory.gate_cap) == (1, 24, 40, 5.0)
    assert (latent.heads, latent.dim, latent.rot_dim, latent.vdim, latent.kv_rank, latent.q_rank, latent.scale) == (3, 16, 12, 24, 40, 48, 0.35)
    s = latent.rot_scaling
    assert (latent.rot_base, latent.rot_dims, s.factor, s.original, s.fast, s.slow) == (500.0, 12, 4.0, 64.0, 8.0, 1.0)
    assert (linear.heads, linear.dim, linear.vdim, linear.tau) == (3, 12, 20, 8.0)
    assert second.rot_scaling is None and cfg.layers[1].mlp is None and cfg.layers[2].mlp.ff == 50
    other = FumolornConfig.from_dict(helpers.FUMOLORN_B)
    assert other.logit_softcap is None and other.bigram is None and other.residual_mult == 1.0


@pytest.mark.parametrize("patch,match", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.pop("residual_mult"), "residual_mult"),
    (lambda c: c.__setitem__("logit_softcap", 0), "logit_softcap"),
    (lambda c: c.__setitem__("width", True), "width must be int, got bool"),
    (lambda c: c["layers"][0].__setitem__("type", "mamba"), "not a layer of this design"),
    (lambda c: c["layers"][0]["mixer"].__setitem__("gate_cap", 0), "gate_cap"),
    (lambda c: c["layers"][2]["mixer"].__setitem__("tau", -1), "tau"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 14), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"]["rot"].__setitem__("dims", 7), "rot.dims"),
    (lambda c: c["layers"][1]["mixer"].pop("rot"), "needs a rot entry"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].__setitem__("factor", 0), "factor"),
    (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "moe"), "not a feed-forward of this design"),
    (lambda c: c["embedding"]["bigram"].__setitem__("buckets", 0), "buckets"),
    (lambda c: c.__setitem__("layers", []), "layers must not be empty"),
])
def test_a_bad_config_is_refused_with_the_key_named(patch, match):
    raw = copy.deepcopy(helpers.FUMOLORN_A)
    patch(raw)
    with pytest.raises(ConfigError, match=match):
        FumolornConfig.from_dict(raw)


def test_tensor_names_and_shapes_follow_the_description():
    schema = tensor_schema(describe_fumolorn(FumolornConfig.from_dict(helpers.FUMOLORN_A), {2: 10}))
    assert schema["embed"].shape == (211, 64) and schema["bigram"].shape == (14, 64) and schema["head"].shape == (211, 64)
    assert schema["embed.norm"].shape == (64,) and schema["final.norm"].shape == (64,)
    assert "l1.norm2" not in schema and schema["l2.norm2"].shape == (64,)
    assert schema["l0.mix.q"].shape == (24, 64) and schema["l0.mix.v"].shape == (40, 64) and schema["l0.mix.g"].shape == (40, 64)
    assert schema["l3.mix.i"].shape == (5, 64) and schema["l3.mix.f.b"].shape == (5,) and schema["l3.mix.norm"].shape == (40,)
    assert schema["l1.mix.dq"].shape == (48, 64) and schema["l1.mix.uq"].shape == (84, 48) and schema["l1.mix.dkv"].shape == (52, 64)
    assert schema["l1.mix.g"].shape == (3, 64) and schema["l1.mix.sink"].shape == (3,) and schema["l1.mix.uv"].shape == (72, 40)
    assert schema["l2.mix.a1"].shape == (10, 64) and schema["l2.mix.a2"].shape == (36, 10) and schema["l2.mix.a2.b"].shape == (36,)
    assert schema["l2.mix.norm"].shape == (20,) and schema["l2.mlp.gate"].shape == (50, 64) and schema["l2.mlp.down"].shape == (64, 50)
    assert "bigram" not in tensor_schema(describe_fumolorn(FumolornConfig.from_dict(helpers.FUMOLORN_B)))


def test_low_rank_sizes_come_from_the_stored_shapes():
    raw = copy.deepcopy(helpers.FUMOLORN_A)
    del raw["layers"][1]["mixer"]["q_rank"]
    config = FumolornConfig.from_dict(raw)
    with pytest.raises(ConfigError, match="q_rank"):
        describe_fumolorn(config)
    schema = tensor_schema(describe_for_checkpoint(config, {"l1.mix.dq": (44, 64), "l2.mix.a1": (5, 64)}))
    assert schema["l1.mix.uq"].shape == (84, 44) and schema["l2.mix.a2"].shape == (36, 5)


def test_the_cache_layout_comes_from_the_mixers_and_the_embedding():
    model = DecoderModel(describe_fumolorn(FumolornConfig.from_dict(helpers.FUMOLORN_A)))
    layout = model.cache_layout()
    needs = {group.requirement: group.layers for group in layout.groups}
    assert all(isinstance(need, PagedTensors) and need.window is None for need in needs)
    assert sorted(need.tensors[0][1][0] for need in needs) == [28, 52]          # latent plus rotated key part
    states = {(s.layer, s.requirement.name): s.requirement for s in layout.states}
    assert states[(0, "state")] == FixedState((1, 24, 40), torch.float32, "state")
    assert states[(3, "normaliser")].shape == (5, 16) and states[(3, "maximum")].shape == (5,)
    assert states[(2, "state")].shape == (3, 12, 20)
    assert states[(5, "previous_token")] == FixedState((1,), torch.int32, "previous_token")
    assert model.graph_safe()


@pytest.mark.parametrize("dims,base,scaling", [
    (16, 10000.0, {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}),
    (64, 10000.0, {"factor": 40.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
    (12, 500.0, {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}),
    (8, 50.0, {"factor": 3.0, "original": 4, "fast": 900.0, "slow": 800.0}),       # both ends below pair 0: every pair divided
    (4, 10000.0, {"factor": 3.0, "original": 1 << 20, "fast": 2.0, "slow": 1.0}),  # both ends clamped or past the last pair
    (2, 100.0, {"factor": 2.0, "original": 64, "fast": 4.0, "slow": 4.0}),
])
def test_stretched_frequencies(dims, base, scaling):
    rope = RotaryEmbedding(dims, base, dims, scaling=scaling, interleaved=True)
    rope.load({}, Runtime(torch.device("cpu"), torch.float32))
    inv_freq, rotary_dim, interleaved, factor = rope.rotary_layout()
    want, want_factor = plain.ramp_frequencies(dims, base, scaling)
    assert rotary_dim == dims and interleaved and abs(factor - want_factor) < 1e-12
    assert torch.allclose(inv_freq.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6, atol=0)
    with pytest.raises(KernelError):           # kernels that know neither the pairing nor the factor are not handed the table
        rope.rotary_parameters()


def test_the_plain_rotation_and_frequencies():
    f, factor = plain.ramp_frequencies(8, 100.0, None)
    assert factor == 1.0 and all(abs(x - 100.0 ** (-i / 4)) < 1e-12 for i, x in enumerate(f))
    scaling = {"factor": 4.0, "original": 128, "fast": 8.0, "slow": 1.0}
    f, factor = plain.ramp_frequencies(8, 100.0, scaling)
    # pair indices of 8 and of 1 turns in 128 positions: 8 ln(128 / (16 pi)) / (2 ln 100) = 0.81 and 2.62: from pair 0 to pair 3
    for i, x in enumerate(f):
        r = min(i / 3, 1.0)
        assert abs(x - 100.0 ** (-i / 4) * (r / 4.0 + 1 - r)) < 1e-12
    assert abs(factor - (0.1 * math.log(4.0) + 1)) < 1e-12
    x = torch.tensor([[1.0, 0.0, 0.0, 2.0, 7.0]], dtype=torch.float64)
    y = plain.rotate_pairs(x, torch.tensor([3]), [0.5, 0.25], 2.0)
    want = [2 * math.cos(1.5), 2 * math.sin(1.5), -4 * math.sin(0.75), 4 * math.cos(0.75), 7.0]
    assert torch.allclose(y[0], torch.tensor(want, dtype=torch.float64))


def test_the_plain_sink_counts_once_and_is_not_scaled():
    w = plain.sink_softmax(torch.log(torch.tensor([[1.0, 2.0]], dtype=torch.float64)), torch.tensor(math.log(5.0), dtype=torch.float64))
    assert torch.allclose(w, torch.tensor([[1 / 8, 2 / 8]], dtype=torch.float64))
    q = torch.zeros(3, 1, 2, dtype=torch.float64)
    v = torch.tensor([3.0, 6.0, 12.0], dtype=torch.float64).view(3, 1, 1)
    out = plain.sink_attention(q, q, v, scale=9.0, sink=torch.tensor([0.0], dtype=torch.float64))
    assert torch.allclose(out[:, 0, 0], torch.tensor([3 / 2, 9 / 3, 21 / 4], dtype=torch.float64))


def test_the_plain_matrix_memory_equals_its_unscaled_form():
    """Without the running maximum: S = sum of products of sigmoids times e^i k v^T, divided by max(|n.q|, 1) (both sides of
    the quotient scaled alike by e^-m, but for the small constant)."""

    torch.manual_seed(0)
    T, d, dv = 9, 3, 4
    q, k, v = (torch.randn(T, 1, n, dtype=torch.float64) for n in (d, d, dv))
    li, lf = plain.mlstm_gates(3 * torch.randn(T, 1, dtype=torch.float64), 3 * torch.randn(T, 1, dtype=torch.float64), 2.0)
    assert li.abs().max() < 2.0 and lf.max() < 0
    out = plain.mlstm_scan(q, k, v, li, lf)
    S, n = torch.zeros(d, dv, dtype=torch.float64), torch.zeros(d, dtype=torch.float64)
    m = 0.0
    for t in range(T):
        S = torch.exp(lf[t, 0]) * S + torch.exp(li[t, 0]) * k[t, 0][:, None] * v[t, 0][None, :]
        n = torch.exp(lf[t, 0]) * n + torch.exp(li[t, 0]) * k[t, 0]
        m = max(float(lf[t, 0]) + m, float(li[t, 0]))
        want = S.T @ q[t, 0] / (max(abs(float(n @ q[t, 0])), 1.0) + 1e-6 * math.exp(m))
        assert torch.allclose(out[t, 0], want)
    # the first token: m starts at zero, so a small input gate leaves the floor at one
    small = plain.mlstm_scan(q[:1], k[:1], v[:1], torch.full((1, 1), -50.0, dtype=torch.float64), torch.full((1, 1), -1e-9, dtype=torch.float64))
    assert small.abs().max() < 1e-15


def test_the_plain_channel_decay_and_scan():
    z = torch.tensor([-40.0, 0.0, 40.0], dtype=torch.float64)
    a = plain.channel_decay(z, 4.0)
    assert torch.allclose(a, torch.tensor([math.exp(-10.0), 0.5 ** 0.25, 1.0], dtype=torch.float64))
    k = torch.tensor([[[1.0, 0.0]], [[0.0, 1.0]], [[0.0, 0.0]]], dtype=torch.float64)
    alpha = torch.tensor([[[0.5, 0.25]]], dtype=torch.float64).expand(3, 1, 2)
    v = torch.tensor([8.0, 16.0, 1.0], dtype=torch.float64).view(3, 1, 1)
    out = plain.gla_scan(torch.ones(3, 1, 2, dtype=torch.float64), k, v, alpha)
    assert out[:, 0, 0].tolist() == [8.0, 4.0 + 16.0, 2.0 + 4.0]
