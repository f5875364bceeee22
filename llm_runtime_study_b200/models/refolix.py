"""Refolix, described as parts.

A decoder whose norms sit behind the sums (``x <- norm(alpha x + s * sublayer(x))``, layer norms, a scale per channel on every
sublayer's output) and whose layers carry one of two mixers: ``parallel`` (softmax attention with normed and rotated q and k,
YaRN's frequencies, capped scores and a sliding window, beside the delta rule with one decay per head; the mean of their normed
outputs) or ``retention`` (linear attention with a constant decay per head behind a rotation).  The feed-forward is a mixture of
gated units (sigmoid scores with a correction for the choice only, groups of neighbours scored by their two best, weights
renormalised over the chosen, a shared unit behind a sigmoid gate per token), or absent.  The embedding is scaled; the output
head has a matrix of its own, a scale and a soft cap on the logits.

Tensor names: ``embed``, ``final.norm``, ``head``; a layer's tensors start with ``l<i>.``: ``norm1``, ``norm2``, ``ls1``, ``ls2``, ``mix.*``
(``mix.left.*``, ``mix.right.*``), ``mlp.*``; a linear map's weight is stored under the map's own name (no ``.weight``).
"""

from __future__ import annotations

from dataclasses import asdict

from ..config.refolix import Experts, Parallel, RefolixConfig, RefolixLayer, Retention, Rotation
from ..config.registry import Architecture, register_architecture
from .description import LayerDescription, ModelDescription
from .sorulix import stored_name

# Fixed by the design (not in config.json): the constant under the unit vectors' root, how many choice scores a group sums.
UNIT_EPS = 1e-6
GROUP_BEST = 2


def _position(rot: Rotation | None, dim: int, interleaved: bool) -> dict | None:
    if rot is None:
        return None
    return {"kind": "rope", "head_dim": dim, "theta": rot.base, "rotary_dim": rot.dims, "interleaved": interleaved,
            "scaling": asdict(rot.scaling) if rot.scaling else None}


def _mixer(layer: RefolixLayer, config: RefolixConfig) -> dict:
    m = layer.mixer
    if isinstance(m, Parallel):
        left, right = m.left, m.right
        return {
            "kind": "parallel", "hidden_size": config.width, "eps": config.eps,
            "branches": [
                {"name": "left", "mixer": {
                    "kind": "capped_attention", "hidden_size": config.width, "num_heads": left.heads, "num_kv_heads": left.kv_heads,
                    "head_dim": left.dim, "value_dim": left.vdim, "scale": left.scale, "qk_norm_eps": config.eps,
                    "softcap": left.softcap, "window": left.window, "position": _position(left.rot, left.dim, True),
                }},
                {"name": "right", "mixer": {
                    "kind": "gated_delta_rule", "hidden_size": config.width, "num_heads": right.heads, "num_qk_heads": right.kv_heads,
                    "head_dim": right.dim, "value_dim": right.vdim, "taps": right.conv, "decay_rank": None, "gate_rank": None,
                    "gate_act": "silu", "eps": config.eps, "unit_eps": UNIT_EPS,
                }},
            ],
        }
    assert isinstance(m, Retention)
    return {"kind": "retention", "hidden_size": config.width, "num_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim,
            "decay": m.decay, "eps": config.eps, "position": _position(m.rot, m.dim, False)}


def _feed_forward(mlp: Experts | None, config: RefolixConfig) -> dict | None:
    if mlp is None:
        return None
    return {
        "kind": "routed_experts", "hidden_size": config.width, "intermediate_size": mlp.ff, "experts": mlp.experts, "top": mlp.top,
        "act": "silu_glu", "router_bias": False, "score": "sigmoid_all", "correction": True, "groups": mlp.groups, "keep": mlp.keep,
        "group_best": GROUP_BEST, "renormalise": True, "shared_size": mlp.shared_ff, "shared_gate": mlp.shared_ff is not None,
    }


def describe_refolix(config: RefolixConfig) -> ModelDescription:
    norm = {"kind": "layer_norm", "dim": config.width, "eps": config.eps}
    layers = []
    for i, layer in enumerate(config.layers):
        block = {
            "kind": "sum_norm", "hidden_size": config.width, "mixer_norm": norm, "mixer": _mixer(layer, config),
            "ffn_norm": norm if layer.mlp else None, "feed_forward": _feed_forward(layer.mlp, config),
            "names": {"mixer_norm": "norm1", "mixer": "mix", "ffn_norm": "norm2", "feed_forward": "mlp"},
            "alpha": config.postln_alpha, "layer_scale": True,
        }
        layers.append(LayerDescription(block=block, prefix=f"l{i}"))
    return ModelDescription(
        architecture=RefolixConfig.ARCHITECTURE, vocab_size=config.vocab, hidden_size=config.width,
        max_positions=RefolixConfig.MAX_POSITIONS, eos_token_ids=(),
        embedding={"prefix": "embed", "vocab_size": config.vocab, "hidden_size": config.width, "scale": config.embedding_scale},
        layers=tuple(layers), order=tuple(range(len(layers))),
        final_norm={"prefix": "final.norm", **norm},
        head={"prefix": "head", "vocab_size": config.vocab, "hidden_size": config.width, "softcap": config.logit_softcap,
              "scale": config.logit_scale},
        stored_name=stored_name,
    )


REFOLIX = Architecture(
    name=RefolixConfig.ARCHITECTURE, model_type=RefolixConfig.MODEL_TYPE,
    config_from_dict=RefolixConfig.from_dict, describe=describe_refolix,
)
register_architecture(REFOLIX, replace=True)
