"""Fumolorn, described as parts.

A decoder whose norms sit on the sublayers' outputs (``x <- x + m * norm(sublayer(x))`` with one factor ``m`` for the model) behind
an embedding that is a scaled token table plus a table of hashed bigrams, normed, and whose layers carry one of three mixers:
``latent_attention`` (attention over one low-rank latent per token with a rotated key part shared by the heads, interleaved
pairs with YaRN's frequencies, a sink and one sigmoid gate per head), ``mlstm`` (the matrix memory of xLSTM with capped exponential
gates) or ``gla`` (linear attention with a decay per key channel).  The feed-forward is a gated unit with the tanh form of gelu,
or absent.  The output head has a matrix of its own and a soft cap on the logits.

Tensor names: ``embed``, ``bigram``, ``embed.norm``, ``final.norm``, ``head``; a layer's tensors start with ``l<i>.``: ``norm1``,
``norm2``, ``mix.*``, ``mlp.*``; a linear map's weight is stored under the map's own name (no ``.weight``), its bias under ``<name>.b``.
"""

from __future__ import annotations

from dataclasses import asdict

from ..config.fumolorn import FumolornConfig, FumolornLayer, GatedLinear, LatentAttention, MatrixMemory
from ..config.registry import Architecture, register_architecture
from ..errors import ConfigError
from .description import LayerDescription, ModelDescription
from .tafisun import stored_name

MLP_ACT = "gelu_tanh"     # fixed by the design (not in config.json)


def _mixer(index: int, layer: FumolornLayer, config: FumolornConfig, ranks: dict[int, int]) -> dict:
    m = layer.mixer
    sizes = {"hidden_size": config.width, "num_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim, "eps": config.eps}
    if isinstance(m, MatrixMemory):
        return {"kind": "matrix_memory", **sizes, "gate_cap": m.gate_cap}
    if isinstance(m, GatedLinear):
        return {"kind": "gated_linear_attention", **sizes, "tau": m.tau, "decay_rank": ranks.get(index, max(1, m.dim // 4))}
    assert isinstance(m, LatentAttention)
    q_rank = m.q_rank or ranks.get(index, 0)
    if q_rank <= 0:
        raise ConfigError(f"layers[{index}].mixer.q_rank is neither in the configuration nor given by a stored tensor's shape")
    position = None
    if m.rot_dims:
        position = {"kind": "rope", "head_dim": m.rot_dim, "theta": m.rot_base, "rotary_dim": m.rot_dims, "interleaved": True,
                    "scaling": asdict(m.rot_scaling) if m.rot_scaling else None}
    return {"kind": "latent_attention", **sizes, "rot_dim": m.rot_dim, "kv_rank": m.kv_rank, "q_rank": q_rank, "scale": m.scale,
            "position": position, "sink": True, "gate": "head"}


def describe_fumolorn(config: FumolornConfig, ranks: dict[int, int] | None = None) -> ModelDescription:
    """``ranks``: per layer, the inner size of a low-rank map that config.json does not give (a gla layer's decay; a latent
    attention layer's query where the configuration leaves it out): the stored tensors' shapes do (``describe_for_checkpoint``).
    Without them a quarter of the key size is assumed for the decay, which is what random weights are drawn with."""

    norm = {"kind": "rms_norm", "dim": config.width, "eps": config.eps}
    layers = []
    for i, layer in enumerate(config.layers):
        block = {
            "kind": "output_norm", "mixer_norm": norm, "mixer": _mixer(i, layer, config, ranks or {}),
            "ffn_norm": norm if layer.mlp else None,
            "feed_forward": {"kind": "gated_mlp", "hidden_size": config.width, "intermediate_size": layer.mlp.ff, "act": MLP_ACT,
                             "names": ("gate", "up", "down")} if layer.mlp else None,
            "names": {"mixer_norm": "norm1", "mixer": "mix", "ffn_norm": "norm2", "feed_forward": "mlp"},
            "residual_factor": config.residual_mult,
        }
        layers.append(LayerDescription(block=block, prefix=f"l{i}"))
    bigram = config.bigram
    return ModelDescription(
        architecture=FumolornConfig.ARCHITECTURE, vocab_size=config.vocab, hidden_size=config.width,
        max_positions=FumolornConfig.MAX_POSITIONS, eos_token_ids=(),
        embedding={"prefix": "embed", "kind": "summed_embedding", "vocab_size": config.vocab, "hidden_size": config.width,
                   "scale": config.embedding_scale, "norm": norm,
                   "bigram": (bigram.buckets, bigram.mul_prev, bigram.mul_cur) if bigram else None},
        layers=tuple(layers), order=tuple(range(len(layers))),
        final_norm={"prefix": "final.norm", **norm},
        head={"prefix": "head", "vocab_size": config.vocab, "hidden_size": config.width, "softcap": config.logit_softcap},
        stored_name=stored_name,
    )


def describe_for_checkpoint(config: FumolornConfig, shapes) -> ModelDescription:
    """The description with the low-rank sizes read from the checkpoint's tensor shapes (``shapes``: name -> shape)."""

    ranks = {}
    for i, layer in enumerate(config.layers):
        name = {"gla": "a1", "latent_attention": "dq"}.get(layer.type)
        shape = shapes.get(f"l{i}.mix.{name}")
        if shape is not None and len(shape) == 2:
            ranks[i] = int(shape[0])
    return describe_fumolorn(config, ranks)


FUMOLORN = Architecture(
    name=FumolornConfig.ARCHITECTURE, model_type=FumolornConfig.MODEL_TYPE,
    config_from_dict=FumolornConfig.from_dict, describe=describe_fumolorn, describe_for_checkpoint=describe_for_checkpoint,
)
register_architecture(FUMOLORN, replace=True)
