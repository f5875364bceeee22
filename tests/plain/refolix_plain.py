"""Plain, slow Refolix forward pass: whole sequences, no cache, CPU.

One function per mechanism, elementary torch operations only, nothing shared with the engine.  It takes a
``config.json`` dict and ``{tensor name: tensor}`` with the checkpoint's own names.  ``dtype`` is the arithmetic
type (float64 separates rounding from faults).

``store`` (optional) is applied wherever a serving engine with 16-bit activations keeps a tensor in memory
between two operations: the rows a sublayer reads, the results of projections, q, k and v as they enter the softmax
attention, the gated read-outs, the hidden rows of a feed-forward.  The residual stream, the statistics, everything that enters
a recurrence behind its projections, the states, the router and the logits stay in ``dtype`` either way.

Notation: ``T`` tokens at positions ``0..T-1``; ``unit(x) = x / sqrt(mean(x^2) + eps)`` over the last axis;
every linear map is ``x @ W.T`` with ``W`` stored ``[out, in]``.
"""

from __future__ import annotations

import math
from typing import Mapping

import torch

UNIT_EPS = 1e-6


# ----------------------------------------------------------------- elementary
def keep(x: torch.Tensor) -> torch.Tensor:
    return x


def round_bfloat16(x: torch.Tensor) -> torch.Tensor:
    return x.to(torch.bfloat16).to(x.dtype)


def unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * w


def sigmoid(x: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * sigmoid(x)


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


def soft_cap(z: torch.Tensor, cap: float | None) -> torch.Tensor:
    return z if cap is None else cap * torch.tanh(z / cap)


# ------------------------------------------------------------------- rotation
def frequencies(dims: int, base: float, scaling: Mapping | None = None) -> tuple[list[float], float]:
    """One frequency per pair of the ``dims`` rotated columns, and the factor on cosine and sine.

    With ``scaling`` (YaRN) the pairs between the one whose wavelength fits ``fast`` times into ``original`` positions and the one
    whose wavelength fits ``slow`` times go over from their frequency to that frequency divided by ``factor``."""

    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0

    def pair_with(turns: float) -> float:
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    first = max(math.floor(pair_with(scaling["fast"])), 0)
    last = min(math.ceil(pair_with(scaling["slow"])), dims - 1)
    out = []
    for i in range(dims // 2):
        share = (i - first) / max(last - first, 0.001)
        share = 0.0 if share < 0.0 else 1.0 if share > 1.0 else share
        out.append((1.0 - share) * f[i] + share * f[i] / scaling["factor"])
    return out, 1.0 + 0.1 * math.log(scaling["factor"])


def rotate(x: torch.Tensor, freq: list[float], factor: float = 1.0, *, interleaved: bool) -> torch.Tensor:
    """``x`` ``[T, heads, d]``: pair i of the leading ``2 len(freq)`` columns is ``(2i, 2i + 1)`` or, not interleaved, ``(i, i +
    len(freq))``; row p's pair turns by ``p * freq[i]``, cosine and sine times ``factor``.  Further columns pass unchanged."""

    out = x.clone()
    p = torch.arange(x.shape[0], dtype=torch.float64)
    for i, f in enumerate(freq):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + len(freq))
        c = (factor * torch.cos(p * f)).to(x.dtype)[:, None]
        s = (factor * torch.sin(p * f)).to(x.dtype)[:, None]
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


# ----------------------------------------------------------- softmax attention
def window_mask(T: int, size: int | None) -> torch.Tensor:
    """[i, j]: whether i sees j: ``0 <= i - j < size``."""

    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) if size is None else (back >= 0) & (back < size)


def window_attention(q, k, v, *, scale: float, cap: float | None, size: int | None) -> torch.Tensor:
    """q ``[T, H, d]``, k ``[T, G, d]``, v ``[T, G, dv]`` -> ``[T, H, dv]``."""

    T, H, _ = q.shape
    seen = window_mask(T, size)
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // k.shape[1])
        s = soft_cap((q[:, h] @ k[:, g].T) * scale, cap).masked_fill(~seen, -math.inf)
        e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
        out[:, h] = (e / e.sum(dim=-1, keepdim=True)) @ v[:, g]
    return out


def attention_branch(h, w: Mapping[str, torch.Tensor], m: Mapping, eps: float, store=keep) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit(store(h @ w["q"].T).view(T, H, d), eps) * w["q.norm"]
    k = unit(store(h @ w["k"].T).view(T, G, d), eps) * w["k.norm"]
    v = store(h @ w["v"].T).view(T, G, dv)
    freq, factor = frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q, k = (store(rotate(t, freq, factor, interleaved=True)) for t in (q, k))
    o = window_attention(q, k, v, scale=m["scale"], cap=m["softcap"], size=m["mask"]["size"])
    return store(o).reshape(T, H * dv) @ w["o"].T


# ------------------------------------------------------------------ recurrences
def short_convolution(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """``x`` ``[T, C]``, ``taps`` ``[C, K]``: ``y_t = sum_j taps[:, j] x_(t - (K-1) + j)``, zeros before the start."""

    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y


def unit_vectors(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + UNIT_EPS)


def head_decay(z: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor) -> torch.Tensor:
    return torch.exp(-torch.exp(a_log) * softplus(z + dt_bias))


def delta_scan(q, k, v, g, beta) -> torch.Tensor:
    """q, k ``[T, G, d]``, v ``[T, H, dv]``, g and beta ``[T, H]`` -> ``[T, H, dv]``: decay, correct, write, read."""

    T, H, dv = v.shape
    out = torch.zeros(T, H, dv, dtype=v.dtype)
    for h in range(H):
        j = h // (H // q.shape[1])
        S = torch.zeros(q.shape[2], dv, dtype=v.dtype)
        for t in range(T):
            S = g[t, h] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, j])
            S = S + k[t, j][:, None] * u[None, :]
            out[t, h] = S.T @ q[t, j]
    return out


def delta_branch(h, w: Mapping[str, torch.Tensor], m: Mapping, eps: float, store=keep) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_convolution(store(h @ w[n].T), w[f"{n}.conv"])) for n in ("q", "k", "v"))
    q = unit_vectors(q.view(T, G, d)) * d ** -0.5
    k = unit_vectors(k.view(T, G, d))
    beta = sigmoid(store(h @ w["b"].T))
    g = head_decay(store(h @ w["a"].T), w["A_log"], w["dt_bias"])
    o = unit(delta_scan(q, k, v.view(T, H, dv), g, beta), eps) * w["norm"]
    return store(o.reshape(T, H * dv) * silu(store(h @ w["g"].T))) @ w["o"].T


def retention_scan(q, k, v, decay) -> torch.Tensor:
    """q, k ``[T, H, d]``, v ``[T, H, dv]``, one decay per head -> ``[T, H, dv]``: ``S <- decay S + k v^T``, ``o = S^T q``."""

    T, H, d = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(d, v.shape[2], dtype=q.dtype)
        for t in range(T):
            S = decay[h] * S + k[t, h][:, None] * v[t, h][None, :]
            out[t, h] = S.T @ q[t, h]
    return out


def retention_mixer(h, w: Mapping[str, torch.Tensor], m: Mapping, eps: float, store=keep) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, k = (store(h @ w[n].T).view(T, H, d) for n in ("q", "k"))
    v = store(h @ w["v"].T).view(T, H, dv)
    freq, _ = frequencies(m["rot"]["dims"], m["rot"]["base"])
    q, k = rotate(q, freq, interleaved=False), rotate(k, freq, interleaved=False) * d ** -0.5
    o = unit(retention_scan(q, k, v, m["decay"]), eps).reshape(T, H * dv)
    return store(o * silu(store(h @ w["g"].T))) @ w["o"].T


def parallel_mixer(h, w: Mapping[str, torch.Tensor], m: Mapping, eps: float, store=keep) -> torch.Tensor:
    left = attention_branch(h, sub(w, "left."), m["left"], eps, store)
    right = delta_branch(h, sub(w, "right."), m["right"], eps, store)
    return 0.5 * (unit(left, eps) * w["left.out"] + unit(right, eps) * w["right.out"])


# ---------------------------------------------------------------- feed-forward
def route(z: torch.Tensor, correction: torch.Tensor, *, top: int, groups: int, keep_groups: int,
          margins: list | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """Logits ``[T, E]`` -> (chosen ``[T, top]``, weights).  ``margins`` receives, per token, by how much the choices (of
    groups, of experts) were decided."""

    s = sigmoid(z)
    c = s + correction
    T, E = z.shape
    per = E // groups
    chosen = torch.zeros(T, top, dtype=torch.long)
    for t in range(T):
        rank = [sum(sorted(c[t, g * per:(g + 1) * per].tolist(), reverse=True)[:2]) for g in range(groups)]
        order = sorted(range(groups), key=lambda g: (-rank[g], g))
        open_ = [e for g in order[:keep_groups] for e in range(g * per, (g + 1) * per)]
        picks = sorted(open_, key=lambda e: (-float(c[t, e]), e))
        chosen[t] = torch.tensor(picks[:top])
        if margins is not None:
            gap = [rank[order[keep_groups - 1]] - rank[order[keep_groups]]] if keep_groups < groups else []
            gap += [float(c[t, picks[top - 1]] - c[t, picks[top]])] if top < len(picks) else []
            margins.append(min(gap) if gap else math.inf)
    w = torch.gather(s, 1, chosen)
    return chosen, w / (w.sum(dim=1, keepdim=True) + 1e-20)


def gated_unit(h, gate, up, down, store=keep, between=None) -> torch.Tensor:
    """``W_down (silu(W_gate h) * (W_up h))``; ``between``: the rounding of the two products (default: ``store``)."""

    between = between or store
    return store(silu(between(h @ gate.T)) * between(h @ up.T)) @ down.T


def moe(h, w: Mapping[str, torch.Tensor], mlp: Mapping, store=keep, margins: list | None = None) -> torch.Tensor:
    r = mlp["router"]
    chosen, weights = route(h @ w["router"].T, w["correction"], top=r["top"], groups=r["groups"]["count"],
                            keep_groups=r["groups"]["keep"], margins=margins)
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        at, place = (chosen == e).nonzero(as_tuple=True)
        if at.numel():
            out[at] += weights[at, place][:, None] * gated_unit(h[at], *(w[f"e{e}.{n}"] for n in ("gate", "up", "down")), store)
    if mlp.get("shared"):
        out = out + sigmoid(h @ w["shared.sg"].T) * gated_unit(h, *(w[f"shared.{n}"] for n in ("gate", "up", "down")), store, keep)
    return out


# ----------------------------------------------------------------------- model
MIXERS = {"parallel": parallel_mixer, "retention": retention_mixer}


def sub(weights: Mapping[str, torch.Tensor], prefix: str, dtype=None) -> dict:
    return {k[len(prefix):]: v if dtype is None else v.to(dtype) for k, v in weights.items() if k.startswith(prefix)}


def forward(config: Mapping, weights: Mapping[str, torch.Tensor], tokens, dtype=torch.float64, store=keep, layers_out=None,
            margins: list | None = None):
    """Logits ``[T, vocab]`` of one sequence.  ``layers_out`` (a list) receives the residual rows after every layer; ``margins``
    (a list) one list per routed layer, see ``route``."""

    eps, alpha = config["norm"]["eps"], config["postln_alpha"]
    x = weights["embed"].to(dtype)[torch.tensor([int(t) for t in tokens])] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        w = sub(weights, f"l{i}.", dtype)
        y = MIXERS[layer["type"]](store(x), sub(w, "mix."), layer["mixer"], eps, store)
        x = layer_norm(alpha * x + w["ls1"] * y, w["norm1"], eps)
        if layer.get("mlp"):
            mine = None
            if margins is not None:
                margins.append(mine := [])
            y = moe(store(x), sub(w, "mlp."), layer["mlp"], store, mine)
            x = layer_norm(alpha * x + w["ls2"] * y, w["norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    x = store(layer_norm(x, weights["final.norm"].to(dtype), eps))
    return soft_cap((x @ weights["head"].to(dtype).T) * config["logit_scale"], config["logit_softcap"])
