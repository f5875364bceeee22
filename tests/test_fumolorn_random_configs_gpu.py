"""Fumolorn under random configurations: layers in any order, head and latent sizes on and off the tensor-core kernels'
steps, widths and vocabularies that are no power of two, rotations with and without stretched frequencies, every constant
drawn.  Each configuration is replayed whole, in portions and mixed, in both run types, against the plain implementation."""

import random

import numpy as np
import pytest
import torch

from tests import helpers
from tests.plain import fumolorn_plain as plain

pytestmark = pytest.mark.gpu

TOL32 = (3e-5, 2e-4)
BF16_USUAL, BF16_WORST = 6e-2, 3e-1


def _configuration(case: int):
    rng = random.Random(case)
    width = rng.choice([48, 63, 72, 100, 136, 200, 256])
    layers, ranks = [], {}
    for i in range(rng.choice([1, 2, 3, 4])):
        kind = rng.choice(["latent_attention", "mlstm", "gla"])
        heads = rng.choice([1, 2, 3, 5, 8])
        if kind == "latent_attention":
            rot = rng.choice([2, 8, 16, 16, 32])
            scaling = rng.choice([None, {"factor": rng.choice([1.0, 2.5, 32.0]), "original": rng.choice([16, 300, 4096]),
                                         "fast": rng.choice([4.0, 32.0]), "slow": rng.choice([0.5, 1.0, 4.0])}])
            mixer = {"heads": heads, "dim": rng.choice([7, 16, 24, 48, 64]), "rot_dim": rot, "vdim": rng.choice([5, 16, 32, 40, 64]),
                     "kv_rank": rng.choice([12, 16, 32, 48, 64]), "q_rank": rng.choice([9, 24, 64]), "scale": rng.choice([0.1, 0.25, 0.5]),
                     "rot": {"base": rng.choice([20.0, 1000.0, 500000.0]), "dims": rot, "scaling": scaling}}
        elif kind == "mlstm":
            mixer = {"heads": heads, "dim": rng.choice([5, 16, 32, 48, 136]), "vdim": rng.choice([3, 16, 31, 32, 64, 96]),
                     "gate_cap": rng.choice([1.0, 6.0, 15.0, 30.0])}
        else:
            mixer = {"heads": heads, "dim": rng.choice([6, 16, 32, 64, 144]), "vdim": rng.choice([9, 16, 32, 50, 64]), "tau": rng.choice([1.0, 4.0, 16.0])}
            ranks[i] = rng.choice([1, 5, 16, 24])
        mlp = None if rng.random() < 0.2 else {"kind": "dense", "ff": rng.choice([56, 96, 131, 272])}
        layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
    raw = {"architecture": "Fumolorn", "vocab": rng.choice([97, 256, 503, 1000, 2049]), "width": width,
           "norm": {"eps": rng.choice([1e-6, 1e-5, 3e-6])}, "residual_mult": rng.choice([0.25, 1.0, 1.4]),
           "logit_softcap": rng.choice([2.0, 15.0, 50.0]),
           "embedding": {"scale": rng.choice([0.5, 1.0, 16.0]),
                         "bigram": {"buckets": rng.choice([1, 37, 1013]), "mul_prev": rng.choice([0, 1, 29, 1_000_003]),
                                    "mul_cur": rng.choice([0, 1, 5, 999_983])}},
           "layers": layers}
    lengths = [rng.choice([1, 2, 5, 33, 64, 65, 130, 200]) for _ in range(5)]
    return raw, ranks, lengths, rng


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", range(1, 11))
def test_random_configuration(case, dtype, tmp_path):
    from llm_runtime_study_b200.engine.replay import TraceReplayer
    from llm_runtime_study_b200.engine.runtime import load

    raw, ranks, lengths, rng = _configuration(case)
    path, weights = helpers.make_fumolorn_dir(tmp_path / "model", raw, case, torch_dtype=dtype, ranks=ranks)
    requests = {f"r{i}": helpers.random_tokens(rng, raw["vocab"], n) for i, n in enumerate(lengths)}
    store = plain.round_bfloat16 if dtype == "bfloat16" else plain.keep
    expected = {rid: plain.forward(raw, weights, tokens, store=store) for rid, tokens in requests.items()}
    loaded = load(path, device="cuda:0", dtype=dtype, strict_dtype=False)
    traces = {
        "whole": helpers.trace_whole(requests),
        "mixed": helpers.trace_mixed(requests, random.Random(case), sizes=(2, 3, 8, 40, 130)),
        "portions": helpers.trace_chunked(requests, random.Random(case), sizes=(2, 17, 64, 128, 129)),
    }
    for kind, steps in traces.items():
        replayer = TraceReplayer(loaded, max_tokens=helpers.pool_tokens(steps), max_requests=4)
        outputs = {}
        for record in steps:
            rows = replayer.run_step(record)
            if rows is not None:
                outputs[record["step"]] = torch.from_numpy(np.array(rows))
        replayer.runner.manager.check()
        got = helpers.collect_logits(steps, outputs)
        for rid, tokens in requests.items():
            rows = torch.stack([got[rid][p] for p in range(len(tokens))]).double()
            want = expected[rid]
            if dtype == "float32":
                bad, err, top = helpers.first_wrong_row(rows, want, TOL32)
                assert bad is None, f"{kind}, request {rid}: first wrong position {bad} of {len(tokens)}, {err:.3e}, {top:.3e}; configuration {raw}"
                continue
            err = (rows - want).pow(2).mean(dim=1).sqrt() / want.pow(2).mean(dim=1).sqrt()
            assert torch.isfinite(err).all(), (kind, rid, raw)
            assert float(err.max()) <= BF16_WORST, (kind, rid, int(err.argmax()), float(err.max()), raw)
            assert int((err > BF16_USUAL).sum()) <= max(1, len(tokens) // 10), (kind, rid, err, raw)
