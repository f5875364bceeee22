"""Plain, slow Fumolorn forward pass: whole sequences, no cache, CPU.

One function per mechanism, elementary torch operations only, nothing shared with the engine.  It takes a
``config.json`` dict and ``{tensor name: tensor}`` with the checkpoint's own names.  ``dtype`` is the arithmetic
type (float64 separates rounding from faults).

``store`` (optional) is applied wherever a serving engine with 16-bit activations keeps a tensor in memory
between two operations: the rows a sublayer reads, the results of projections, q and k as they enter the
attention, the gated read-outs, the hidden rows of a feed-forward.  The residual stream, the statistics, the gates
of the recurrences, their states and the logits stay in ``dtype`` either way.

Notation: ``T`` tokens at positions ``0..T-1``; ``unit(x) = x / sqrt(mean(x^2) + eps)`` over the last axis;
every linear map is ``x @ W.T`` with ``W`` stored ``[out, in]``.
"""

from __future__ import annotations

import math
from typing import Mapping

import torch


# ----------------------------------------------------------------- elementary
def keep(x: torch.Tensor) -> torch.Tensor:
    return x


def round_bfloat16(x: torch.Tensor) -> torch.Tensor:
    return x.to(torch.bfloat16).to(x.dtype)


def unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit(x, eps) * w


def sigmoid(x: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-x))


def log_sigmoid(x: torch.Tensor) -> torch.Tensor:
    """``ln sigmoid(x) = min(x, 0) - ln(1 + e^-|x|)``."""

    return torch.clamp(x, max=0.0) - torch.log1p(torch.exp(-x.abs()))


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * sigmoid(x)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def soft_cap(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


# ------------------------------------------------------------------ embedding
def bigram_rows(tokens: list[int], *, buckets: int, mul_prev: int, mul_cur: int) -> list[int]:
    """The row of the bigram table for every position: a hash of (previous token, token); the table's last row
    (number ``buckets``) where there is no previous token."""

    rows = []
    for t, token in enumerate(tokens):
        rows.append(buckets if t == 0 else (tokens[t - 1] * mul_prev + token * mul_cur) % buckets)
    return rows


def embedding(tokens: list[int], weights: Mapping[str, torch.Tensor], config: Mapping, dtype) -> torch.Tensor:
    """The scaled token table plus the bigram table, then a norm."""

    e = config["embedding"]
    x = weights["embed"].to(dtype)[torch.tensor(tokens)] * e["scale"]
    if e.get("bigram"):
        x = x + weights["bigram"].to(dtype)[torch.tensor(bigram_rows(tokens, **e["bigram"]))]
    return rms_norm(x, weights["embed.norm"].to(dtype), config["norm"]["eps"])


# ------------------------------------------------------------------- rotation
def ramp_frequencies(dims: int, base: float, scaling: Mapping | None) -> tuple[list[float], float]:
    """Frequencies ``f_i`` of the ``dims / 2`` pairs and the factor on cosine and sine.

    Without ``scaling``: ``base^(-2i/dims)`` and 1.  With it (YaRN): between the pair indices at which a wavelength fits
    ``fast`` and ``slow`` times into ``original`` positions, ``f_i`` moves linearly from itself to ``f_i / factor``."""

    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return plain, 1.0
    factor, original = scaling["factor"], scaling["original"]

    def index_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(scaling["fast"])), 0)
    hi = min(math.ceil(index_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, freq: list[float], factor: float) -> torch.Tensor:
    """Columns ``2i`` and ``2i + 1`` of the last axis are a pair: ``(u, v) -> (u cos a - v sin a, v cos a + u sin a)`` with
    ``a = p f_i``, cosine and sine multiplied by ``factor``; columns behind the last pair pass unchanged."""

    out = x.clone()
    for i, f in enumerate(freq):
        a = positions.to(torch.float64) * f
        c, s = (factor * torch.cos(a)).to(x.dtype), (factor * torch.sin(a)).to(x.dtype)
        shape = [x.shape[0]] + [1] * (x.dim() - 2)
        c, s = c.view(shape), s.view(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


# ------------------------------------------------------------------ attention
def sink_softmax(scores: torch.Tensor, sink: float | torch.Tensor) -> torch.Tensor:
    """Rows of weights ``e^s_j / (e^sink + sum_k e^s_k)``: a further term in the sum that belongs to no key."""

    top = torch.clamp(scores.max(dim=-1, keepdim=True).values, min=float(sink))
    e = torch.exp(scores - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(torch.as_tensor(sink, dtype=scores.dtype) - top))


def sink_attention(q, k, v, *, scale: float, sink: torch.Tensor) -> torch.Tensor:
    """q ``[T, H, d]``, k ``[T, H or 1, d]``, v ``[T, H or 1, dv]`` -> ``[T, H, dv]``; position i sees every ``j <= i``."""

    T, H, _ = q.shape
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h if k.shape[1] > 1 else 0
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~seen, -math.inf)
        out[:, h] = sink_softmax(s, sink[h]) @ v[:, g]
    return out


def latent_attention_mixer(h, w: Mapping[str, torch.Tensor], m: Mapping, eps: float, store=keep) -> torch.Tensor:
    """Keys and values made from one normed latent per token, a rotated key part shared by the heads, a sink per head and
    one sigmoid gate per head."""

    T = h.shape[0]
    H, d, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions = torch.arange(T)
    freq, factor = ramp_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    cq = store(rms_norm(store(h @ w["dq"].T), w["dq.norm"], eps))
    q = store(cq @ w["uq"].T).view(T, H, d + dr)
    down = store(h @ w["dkv"].T)
    c = store(rms_norm(down[:, :r], w["dkv.norm"], eps))
    k_rot = store(rotate_pairs(down[:, r:], positions, freq, factor))
    q_rot = store(rotate_pairs(q[..., d:], positions, freq, factor))
    k_plain = store(c @ w["uk"].T).view(T, H, d)
    v = store(c @ w["uv"].T).view(T, H, dv)
    k = torch.cat([k_plain, k_rot[:, None, :].expand(T, H, dr)], dim=-1)
    o = sink_attention(torch.cat([q[..., :d], q_rot], dim=-1), k, v, scale=m["scale"], sink=w["sink"])
    gate = sigmoid(store(h @ w["g"].T))            # [T, H]
    o = store(store(o) * gate[:, :, None])
    return o.reshape(T, H * dv) @ w["o"].T


# ---------------------------------------------------------------- recurrences
def mlstm_gates(zi: torch.Tensor, zf: torch.Tensor, cap: float) -> tuple[torch.Tensor, torch.Tensor]:
    """Logarithms of the input gate and of the forget gate from their logits."""

    return soft_cap(zi, cap), log_sigmoid(soft_cap(zf, cap))


def mlstm_scan(q, k, v, log_i, log_f) -> torch.Tensor:
    """q, k ``[T, H, d]``, v ``[T, H, dv]``, gates ``[T, H]`` -> read-outs ``[T, H, dv]``, token after token.  The running
    maximum ``m`` starts at zero and only rescales the state."""

    T, H, d = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(d, v.shape[2], dtype=q.dtype)
        n = torch.zeros(d, dtype=q.dtype)
        m = torch.zeros((), dtype=q.dtype)
        for t in range(T):
            m_new = torch.maximum(log_f[t, h] + m, log_i[t, h])
            forget, take = torch.exp(log_f[t, h] + m - m_new), torch.exp(log_i[t, h] - m_new)
            S = forget * S + take * k[t, h][:, None] * v[t, h][None, :]
            n = forget * n + take * k[t, h]
            m = m_new
            out[t, h] = (S.T @ q[t, h]) / (torch.maximum((n @ q[t, h]).abs(), torch.exp(-m)) + 1e-6)
    return out


def mlstm_mixer(h, w: Mapping[str, torch.Tensor], m: Mapping, eps: float, store=keep) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = store(h @ w["q"].T).view(T, H, d) * d ** -0.5
    k = store(h @ w["k"].T).view(T, H, d)
    v = store(h @ w["v"].T).view(T, H, dv)
    log_i, log_f = mlstm_gates(store(h @ w["i"].T) + w["i.b"], store(h @ w["f"].T) + w["f.b"], m["gate_cap"])
    o = unit(mlstm_scan(q, k, v, log_i, log_f), eps).reshape(T, H * dv)
    return store(o * w["norm"] * sigmoid(store(h @ w["g"].T))) @ w["o"].T


def channel_decay(z: torch.Tensor, tau: float) -> torch.Tensor:
    """``sigmoid(z)^(1/tau)``."""

    return torch.exp(log_sigmoid(z) / tau)


def gla_scan(q, k, v, alpha) -> torch.Tensor:
    """q, k, alpha ``[T, H, d]``, v ``[T, H, dv]`` -> ``[T, H, dv]``: ``S <- diag(alpha) S + k v^T``, ``o = S^T q``."""

    T, H, d = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(d, v.shape[2], dtype=q.dtype)
        for t in range(T):
            S = alpha[t, h][:, None] * S + k[t, h][:, None] * v[t, h][None, :]
            out[t, h] = S.T @ q[t, h]
    return out


def gla_mixer(h, w: Mapping[str, torch.Tensor], m: Mapping, eps: float, store=keep) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = store(h @ w["q"].T).view(T, H, d) * d ** -0.5
    k = store(h @ w["k"].T).view(T, H, d)
    v = store(h @ w["v"].T).view(T, H, dv)
    alpha = channel_decay(store(h @ w["a1"].T) @ w["a2"].T + w["a2.b"], m["tau"]).view(T, H, d)
    o = rms_norm(gla_scan(q, k, v, alpha), w["norm"], eps).reshape(T, H * dv)
    return store(o * silu(store(h @ w["g"].T))) @ w["o"].T


# ---------------------------------------------------------------- feed-forward
def gated_mlp(h, w: Mapping[str, torch.Tensor], store=keep) -> torch.Tensor:
    return store(gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


# ----------------------------------------------------------------------- model
MIXERS = {"latent_attention": latent_attention_mixer, "mlstm": mlstm_mixer, "gla": gla_mixer}


def sub(weights: Mapping[str, torch.Tensor], prefix: str, dtype) -> dict:
    return {k[len(prefix):]: v.to(dtype) for k, v in weights.items() if k.startswith(prefix)}


def forward(config: Mapping, weights: Mapping[str, torch.Tensor], tokens, dtype=torch.float64, store=keep, layers_out=None):
    """Logits ``[T, vocab]`` of one sequence.  ``layers_out`` (a list) receives the residual rows after every layer."""

    eps, mult = config["norm"]["eps"], config["residual_mult"]
    x = embedding([int(t) for t in tokens], weights, config, dtype)
    for i, layer in enumerate(config["layers"]):
        out = MIXERS[layer["type"]](store(x), sub(weights, f"l{i}.mix.", dtype), layer["mixer"], eps, store)
        x = x + mult * rms_norm(out, weights[f"l{i}.norm1"].to(dtype), eps)
        if layer.get("mlp"):
            out = gated_mlp(store(x), sub(weights, f"l{i}.mlp.", dtype), store)
            x = x + mult * rms_norm(out, weights[f"l{i}.norm2"].to(dtype), eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    x = store(rms_norm(x, weights["final.norm"].to(dtype), eps))
    logits = x @ weights["head"].to(dtype).T
    cap = config.get("logit_softcap")
    return soft_cap(logits, cap) if cap else logits
