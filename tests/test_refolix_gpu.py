"""Refolix through the framework against the plain implementation: every mechanism's kernels alone (with inputs made so that
a window's edge, a page's border, a cap or a lost state shows), then whole models under every way of cutting the work (whole
prompts, decoding token by token, portions down to two tokens, mixed batches whose pages and slots are used again), in 32-bit
and in bfloat16, and greedy generation through the engine's own entry point."""

import random
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from tests import helpers
from tests.plain import refolix_plain as plain

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
# a row of logits against the plain model in 64-bit, as fractions of the row's root mean square: (rms, largest).
# float32 is the sharp comparison.  bfloat16: the plain model rounds its activations where the engine stores them; a rounding
# that falls the other way moves single rows, so a request passes when at most a tenth of its rows (or one) is beyond
# BF16_USUAL and none beyond BF16_WORST.  A token whose choice of experts was a close call is not counted, nor are those right
# behind one that was as good as undecided: rounding may decide it.  A wrong state, slot or page moves every row after it.
TOL = {"float32": (3e-5, 2e-4)}
BF16_USUAL, BF16_WORST = 6e-2, 3e-1
TYPES = [torch.float32, torch.bfloat16]


def dev(t):
    return t.to(DEV)


def tolerance(dtype):
    return 2e-5 if dtype == torch.float32 else 2e-2


def close(got, want, tol):
    err = float((got.cpu().double() - want).abs().max())
    assert err <= tol * max(1.0, float(want.abs().max())), err


def ints(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def _pages(seed, page, lengths, spare=3):
    """Block tables that scatter each sequence over pages in a shuffled order; returns (table, pages in use)."""

    rng = random.Random(seed)
    need = [-(-n // page) for n in lengths]
    ids = list(range(sum(need) + spare))
    rng.shuffle(ids)
    table = torch.full((len(lengths), max(need)), -1, dtype=torch.int32)
    at = 0
    for r, n in enumerate(need):
        table[r, :n] = torch.tensor(ids[at:at + n], dtype=torch.int32)
        at += n
    return table, len(ids)


def _ctx(lengths, q_lens):
    """What the kernel chooser reads of a step's context: every sequence of ``lengths`` brings its last ``q_lens`` tokens."""

    positions = torch.cat([torch.arange(m - k, m) for m, k in zip(lengths, q_lens)]).int()
    entry = torch.cat([torch.full((k,), i) for i, k in enumerate(q_lens)]).int()
    return SimpleNamespace(positions=dev(positions), token_entry=dev(entry), all_decode=max(q_lens) == 1, num_entries=len(lengths),
                           q_lens=list(q_lens), kv_lens=list(lengths), max_kv_len=max(lengths), max_q_len=max(q_lens), kv_len=ints(lengths))


def _pools(rows_k, rows_v, table, pages, page, dtype):
    """Keys and values ``[T, heads, d]`` of every sequence laid into pages."""

    k_pool = torch.zeros(pages, rows_k[0].shape[1], page, rows_k[0].shape[2], dtype=dtype)
    v_pool = torch.zeros(pages, rows_v[0].shape[1], page, rows_v[0].shape[2], dtype=dtype)
    for e, (k, v) in enumerate(zip(rows_k, rows_v)):
        for t in range(k.shape[0]):
            k_pool[table[e, t // page], :, t % page] = k[t]
            v_pool[table[e, t // page], :, t % page] = v[t]
    return dev(k_pool), dev(v_pool)


# ------------------------------------------------------------------------------------- norm behind the sum
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("hidden", [256, 50, 7, 1100, 4096])
@pytest.mark.parametrize("centred,scaled,alpha", [(True, True, 2.5), (False, False, 1.0)])
def test_the_norm_behind_the_sum_in_its_three_forms(dtype, hidden, centred, scaled, alpha):
    from llm_runtime_study_b200.ops import block_steps as B
    from llm_runtime_study_b200.ops.mixer_steps import NormedBranches, PairedRows

    torch.manual_seed(hidden)
    n, top, eps = 9, 3, 1e-5
    x, w, s = 0.7 + torch.randn(n, hidden), torch.randn(hidden), torch.randn(hidden) if scaled else None
    rows, extra, extra_scale = torch.randn(n * top + 5, hidden), torch.randn(n, hidden), torch.rand(n)
    pair_row, weights = torch.randperm(n * top + 5)[: n * top].int(), torch.rand(n, top)
    left, right, lw, rw = 3 * torch.randn(n, hidden), 0.1 * torch.randn(n, hidden), torch.randn(hidden), torch.randn(hidden)
    summed = torch.einsum("nt,nth->nh", weights.double(), rows[pair_row.long()].view(n, top, hidden).double())
    forms = [
        (dev(left), left.double()),
        (PairedRows(dev(rows), dev(pair_row), dev(weights)), summed),
        (PairedRows(dev(rows), dev(pair_row), dev(weights), dev(extra), dev(extra_scale)), summed + extra_scale.double()[:, None] * extra.double()),
        (NormedBranches([dev(left)], [dev(lw)], 1e-4, 1.0), plain.unit(left.double(), 1e-4) * lw.double()),
        (NormedBranches([dev(left), dev(right)], [dev(lw), dev(rw)], eps, 0.5),
         0.5 * (plain.unit(left.double(), eps) * lw.double() + plain.unit(right.double(), eps) * rw.double())),
    ]
    for y, want_y in forms:
        total = alpha * x.double() + (s.double() if scaled else 1.0) * want_y
        want = plain.layer_norm(total, w.double(), eps) if centred else plain.unit(total, eps) * w.double()
        on_dev = dev(x.clone())
        rounded = B.sum_norm(on_dev, y, dev(w), eps, alpha=alpha, scale=dev(s) if scaled else None, centred=centred,
                             rounded_dtype=dtype if dtype != torch.float32 else None)
        close(on_dev, want, 3e-6)
        assert (rounded is None) if dtype == torch.float32 else torch.equal(rounded, on_dev.to(dtype))


def test_scaled_embedding_and_scaled_capped_logits():
    from llm_runtime_study_b200.ops import functional as F

    torch.manual_seed(1)
    table = torch.randn(30, 50)
    close(F.embedding(ints([3, 29, 0]), dev(table), 2.5), 2.5 * table[[3, 29, 0]].double(), 1e-6)
    x = 40 * torch.randn(7, 333)
    close(F.soft_cap(dev(x.clone()), 12.0, 0.3), plain.soft_cap(0.3 * x.double(), 12.0), 1e-6)
    close(F.soft_cap(dev(x.clone()), None, 0.3), 0.3 * x.double(), 1e-6)


# -------------------------------------------------------------------------------------- softmax attention
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("nq,nkv,d,dv,rot,interleaved,factor,normed", [
    (3, 1, 24, 20, 12, True, 1.3, True), (4, 2, 32, 48, 32, True, 1.0, True), (2, 2, 10, 16, 10, False, 0.7, True), (5, 1, 128, 64, 64, False, 1.1, False),
    (1, 1, 9, 8, 2, True, 1.2, True),
])
def test_head_norm_rotation_and_page_write(dtype, nq, nkv, d, dv, rot, interleaved, factor, normed):
    """Norm with a weight, then rotation of the leading columns, from positions far into a sequence; values go as they are."""

    from llm_runtime_study_b200.ops import mixer_steps as M

    torch.manual_seed(d)
    page, eps, ends, news = 8, 1e-5, [600, 9], [19, 6]
    n = sum(news)
    ld = nq * d + nkv * (d + dv) + 3
    rows = torch.randn(n, ld).to(dtype)
    qw, kw = 1 + 0.3 * torch.randn(d), 1 + 0.3 * torch.randn(d)
    freq, _ = plain.frequencies(rot, 1000.0)
    inv_freq = torch.tensor(freq, dtype=torch.float64).float()
    ctx = _ctx(ends, news)
    table, pages = _pages(n, page, ends)
    k_pool, v_pool = (torch.zeros(pages, nkv, page, c, dtype=dtype, device=DEV) for c in (d, dv))
    got_q = M.head_norm_write(dev(rows), num_q_heads=nq, num_kv_heads=nkv, head_dim=d, value_dim=dv, eps=eps, q_weight=dev(qw) if normed else None,
                              k_weight=dev(kw) if normed else None, normalise=normed, positions=ctx.positions, token_entry=ctx.token_entry,
                              block_table=dev(table), page_size=page, k_pool=k_pool, v_pool=v_pool, rotary=(dev(inv_freq), rot, interleaved, factor))
    x = rows.double()
    q, k = x[:, : nq * d].view(n, nq, d), x[:, nq * d : (nq + nkv) * d].view(n, nkv, d)
    v = x[:, (nq + nkv) * d : (nq + nkv) * d + nkv * dv].view(n, nkv, dv)
    if normed:
        q, k = plain.unit(q, eps) * qw.double(), plain.unit(k, eps) * kw.double()
    at = 0
    for e, (end, new) in enumerate(zip(ends, news)):
        for t in range(new):
            p = end - new + t

            def turned(heads):       # the plain rotation reads positions off the row number
                far = torch.zeros(p + 1, *heads.shape[1:], dtype=torch.float64)
                far[p] = heads[at]
                return plain.rotate(far, [f.item() for f in inv_freq.double()], factor, interleaved=interleaved)[p]

            tol = 1e-4 if dtype == torch.float32 else 2e-2      # float32 angles of hundreds of radians
            close(got_q[at], turned(q), tol)
            page_id = int(table[e, p // page])
            close(k_pool[page_id, :, p % page], turned(k), tol)
            assert torch.equal(v_pool[page_id, :, p % page].cpu(), rows[at, (nq + nkv) * d : (nq + nkv) * d + nkv * dv].view(nkv, dv))
            at += 1
    assert at == n and v[0].shape == (nkv, dv)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("nq,nkv,d,dv,page,window,cap", [
    (3, 1, 24, 20, 4, 5, 2.0), (4, 2, 32, 48, 16, 16, 6.0), (6, 3, 48, 32, 16, 1, 4.0), (6, 1, 96, 64, 16, 64, 15.0), (2, 1, 64, 96, 8, None, 3.0),
    (20, 1, 32, 32, 16, 33, 5.0), (2, 2, 128, 64, 16, 100, None), (2, 2, 16, 16, 16, 65, 0.5),
])
@pytest.mark.parametrize("q_lens", [[150, 41], [1, 1], [2, 37], [70, 1]])
def test_capped_window_attention(dtype, nq, nkv, d, dv, page, window, cap, q_lens):
    """Portions behind cached rows and single tokens, through the tensor-core kernels where they take the sizes and the
    CUDA-core kernel elsewhere.  Scores are drawn wide enough for the cap to bite."""

    from llm_runtime_study_b200.ops import attention_rules

    torch.manual_seed(d + dv + nq)
    lengths = [150, 41]
    ks, vs = [torch.randn(m, nkv, d).to(dtype) for m in lengths], [torch.randn(m, nkv, dv).to(dtype) for m in lengths]
    table, pages = _pages(d, page, lengths)
    k_pool, v_pool = _pools(ks, vs, table, pages, page, dtype)
    cache = SimpleNamespace(keys=k_pool, values=v_pool, page_size=page)
    q = torch.randn(sum(q_lens), nq, d).to(dtype)
    got = attention_rules.paged_attention_rules(dev(q), cache, _ctx(lengths, q_lens), dev(table), scale=0.4, window=window or 0, softcap=cap or 0.0)
    assert tuple(got.shape) == (sum(q_lens), nq, dv)
    at = 0
    for e, (m, k) in enumerate(zip(lengths, q_lens)):
        full_q = torch.zeros(m, nq, d, dtype=torch.float64)
        full_q[m - k:] = q[at:at + k].double()
        want = plain.window_attention(full_q, ks[e].double(), vs[e].double(), scale=0.4, cap=cap, size=window)[m - k:]
        close(got[at:at + k], want, tolerance(dtype))
        at += k


@pytest.mark.parametrize("kernel", ["float32", "odd-bfloat16", "bfloat16"])
@pytest.mark.parametrize("page,window,marked", [(16, 40, 15), (16, 40, 16), (16, 64, 63), (8, 9, 64), (4, 5, 100), (16, 1024, 3), (16, 600, 0), (16, 2, 511)])
def test_a_key_just_inside_and_just_outside_the_window(kernel, page, window, marked):
    """One key stands out (its score reaches the cap, all others lie near zero).  The queries that see it give nearly its value:
    itself, the window's last position; the position before it and the first one past the window do not.  Whole prompts,
    portions that start at the edge and single tokens; a window longer than the sequence finds a key hundreds of positions
    back."""

    from llm_runtime_study_b200.ops import attention_rules

    dtype = torch.float32 if kernel == "float32" else torch.bfloat16
    heads, d, dv, length, cap = 2, (20 if kernel == "odd-bfloat16" else 32), (12 if kernel == "odd-bfloat16" else 48), 700, 18.0
    torch.manual_seed(marked)
    q, k, v = 0.1 * torch.randn(length, heads, d), 0.1 * torch.randn(length, 1, d), 0.2 * torch.randn(length, 1, dv)
    k[marked] = 0.0
    k[marked, 0, 1] = 30.0
    v[marked, 0, :] = 3.0
    q[:, :, 1] = 30.0
    k[:, 0, 1] *= 0.01
    k[marked, 0, 1] = 30.0
    q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
    table, pages = _pages(marked, page, [length])
    cache = SimpleNamespace(page_size=page)
    cache.keys, cache.values = _pools([k], [v], table, pages, page, dtype)
    want = plain.window_attention(q.double(), k.double(), v.double(), scale=1.0, cap=cap, size=window)
    last = min(marked + window - 1, length - 1)

    def run(end, new):
        return attention_rules.paged_attention_rules(dev(q[end - new:end].contiguous()), cache, _ctx([end], [new]), dev(table), scale=1.0,
                                                     window=window, softcap=cap).cpu().double()

    tol = 3e-5 if dtype == torch.float32 else 4e-2
    whole = run(length, length)
    close(whole, want, tol)
    probes = sorted({p for p in (marked - 1, marked, marked + 1, last - 1, last, last + 1, last + 2) if 0 <= p < length})
    for p in probes:
        alone = run(p + 1, 1)[0]
        start = run(min(p + 2, length), 2)[0 if p + 2 <= length else 1]
        for row in (whole[p], alone, start):
            close(row, want[p], tol)
            if marked <= p <= last:
                assert (row - 3.0).abs().max() < 0.1, (p, row[0, :3])
            else:
                assert (row - 3.0).abs().min() > 1.5, (p, row[0, :3])


def test_single_tokens_whose_keys_are_cut_into_parts():
    """Long sequences of single tokens: the parts are sized for the window, and every part starts behind its edge."""

    from llm_runtime_study_b200.ops import attention_bf16, attention_rules

    torch.manual_seed(8)
    nq, nkv, d, dv, page, cap = 4, 2, 64, 96, 16, 8.0
    lengths = [1500, 3, 700, 901]
    ks, vs = [torch.randn(m, nkv, d).bfloat16() for m in lengths], [torch.randn(m, nkv, dv).bfloat16() for m in lengths]
    table, pages = _pages(3, page, lengths)
    cache = SimpleNamespace(page_size=page)
    cache.keys, cache.values = _pools(ks, vs, table, pages, page, torch.bfloat16)
    q = torch.randn(4, nq, d).bfloat16()
    for window in (None, 900, 130):
        assert window == 130 or attention_bf16.decode_splits(4, nkv, 1, window or 1500, head_dim=80) > 1
        got = attention_rules.paged_attention_rules(dev(q), cache, _ctx(lengths, [1] * 4), dev(table), scale=0.3, window=window or 0, softcap=cap)
        for e, m in enumerate(lengths):
            full_q = torch.zeros(m, nq, d, dtype=torch.float64)
            full_q[m - 1] = q[e].double()
            close(got[e], plain.window_attention(full_q, ks[e].double(), vs[e].double(), scale=0.3, cap=cap, size=window)[m - 1], 2e-2)


# -------------------------------------------------------------------------------------------- recurrences
CUTS = [[1, 2, 1, 9, 3, 40, 33, 64], [153], [2, 151], [32, 32, 32, 57]]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("cuts", CUTS)
@pytest.mark.parametrize("heads,dim,vdim,rot", [(1, 14, 40, 14), (3, 20, 12, 8), (2, 200, 33, 64), (4, 64, 64, 64), (5, 9, 7, 2), (2, 32, 16, 0)])
def test_retention_across_cuts(dtype, cuts, heads, dim, vdim, rot):
    """Rotation, the scaled key, the recurrence, the norm without a weight and the gate, one request cut in several ways."""

    from llm_runtime_study_b200.ops import mixer_steps as M
    from llm_runtime_study_b200.ops import sequence_state as S

    torch.manual_seed(dim + len(cuts))
    qk, vw, n, eps = heads * dim, heads * vdim, sum(cuts), 1e-5
    proj = torch.randn(n, 2 * (qk + vw) + 3).to(dtype)
    decay = torch.tensor([[1.0, 0.5, 0.97, 0.999, 0.9][h] for h in range(heads)])
    freq, _ = plain.frequencies(rot, 300.0) if rot else ([], 1.0)
    inv_freq = torch.tensor(freq, dtype=torch.float64).float()
    state = torch.zeros(3, heads, dim, vdim, device=DEV)
    outs, at = [], 0
    for m in cuts:
        part = dev(proj[at:at + m].contiguous())
        q, k = M.rotate_qk(part, heads=heads, head_dim=dim, positions=ints(range(at, at + m)), k_scale=dim ** -0.5,
                           rotary=(dev(inv_freq), rot, False, 1.0) if rot else None)
        out = S.linear_scan(q, k, part[:, 2 * qk : 2 * qk + vw], heads=heads, qk_heads=heads, dim=dim, vdim=vdim, state=state,
                            q_start=ints([0, m]), slots=ints([1]), decay=dev(decay), fixed_order=dtype == torch.float32)
        outs.append(S.group_norm_gate(out, None, eps, part, gate_offset=2 * qk + vw, group=vdim, act="silu", out_dtype=dtype).cpu())
        at += m
    x = proj.double()
    q, k = x[:, :qk].view(n, heads, dim), x[:, qk : 2 * qk].view(n, heads, dim)
    turned = [f.item() for f in inv_freq.double()]
    q, k = plain.rotate(q, turned, interleaved=False), plain.rotate(k, turned, interleaved=False) * dim ** -0.5
    o = plain.retention_scan(q, k, x[:, 2 * qk : 2 * qk + vw].view(n, heads, vdim), decay.double())
    want = plain.unit(o, eps).reshape(n, vw) * plain.silu(x[:, 2 * qk + vw : 2 * (qk + vw)])
    sure = (o.pow(2).mean(dim=-1).sqrt() > 1e-2).repeat_interleave(vdim, dim=1)      # a read-out near zero is normed up with its rounding
    assert sure.double().mean() > 0.9
    got = torch.cat(outs).double()
    close(torch.where(sure, got, torch.zeros_like(got)), torch.where(sure, want, torch.zeros_like(want)), 1e-4 if dtype == torch.float32 else 1e-2)
    assert state[1].abs().max() > 0 and state[0].abs().max() == 0 and state[2].abs().max() == 0


@pytest.mark.parametrize("dtype", TYPES)
def test_rotated_keys_are_not_rounded_to_the_storage_type(dtype):
    from llm_runtime_study_b200.ops import mixer_steps as M

    torch.manual_seed(0)
    heads, dim, rot = 2, 24, 16
    rows = torch.randn(40, 2 * heads * dim + 8).to(dtype)
    freq, _ = plain.frequencies(rot, 50.0)
    for interleaved, factor in ((False, 1.0), (True, 1.4)):
        q, k = M.rotate_qk(dev(rows), heads=heads, head_dim=dim, positions=ints(range(40)), k_scale=0.2,
                           rotary=(dev(torch.tensor(freq)), rot, interleaved, factor))
        for got, offset, scale in ((q, 0, 1.0), (k, heads * dim, 0.2)):
            want = plain.rotate(rows.double()[:, offset : offset + heads * dim].view(40, heads, dim), freq, factor, interleaved=interleaved) * scale
            close(got.view(40, heads, dim), want, 3e-5 / 10)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("cuts", CUTS)
@pytest.mark.parametrize("heads,groups,dim,vdim,taps", [(6, 2, 12, 10, 4), (2, 1, 24, 36, 2), (1, 1, 40, 5, 1), (4, 4, 64, 64, 3), (3, 1, 144, 16, 5)])
def test_delta_rule_with_one_decay_per_head_across_cuts(dtype, cuts, heads, groups, dim, vdim, taps):
    from llm_runtime_study_b200.ops import sequence_state as S

    torch.manual_seed(dim + len(cuts))
    qk, vw, n, eps = groups * dim, heads * vdim, sum(cuts), 1e-5
    channels = 2 * qk + vw
    proj = torch.randn(n, channels + 2 * heads + vw + 1).to(dtype)
    conv = 0.6 * torch.randn(channels, taps)
    conv[:, -1] += 1.5
    a_log, dt_bias, w = 0.5 * torch.randn(heads), 0.5 * torch.randn(heads) - 3, 1 + 0.3 * torch.randn(vdim)
    state = torch.zeros(3, heads, dim, vdim, device=DEV)
    kept = torch.zeros(3, taps - 1, channels, device=DEV)
    outs, decays, at = [], [], 0
    for m in cuts:
        part, q_start, slot = dev(proj[at:at + m].contiguous()), ints([0, m]), ints([1])
        q, k, v, g, beta = S.delta_prepare(
            part, heads=heads, qk_heads=groups, dim=dim, vdim=vdim, beta_offset=channels, low_offset=channels + heads, rank=0, taps=dev(conv),
            conv_state=kept, a_log=dev(a_log), dt_bias=dev(dt_bias), a_up=None, q_start=q_start, slots=slot, token_entry=ints([0] * m),
            unit_eps=1e-6, q_scale=dim ** -0.5)
        if taps > 1:
            S.conv_state_update(part, kept, q_start, slot)
        out = S.linear_scan(q, k, v, heads=heads, qk_heads=groups, dim=dim, vdim=vdim, state=state, q_start=q_start, slots=slot, row_decay=g,
                            beta=beta, fixed_order=dtype == torch.float32)
        outs.append(S.group_norm_gate(out, dev(w), eps, part, gate_offset=channels + 2 * heads, act="silu", out_dtype=dtype).cpu())
        decays.append(g.cpu())
        at += m
    x = proj.double()
    mixed = plain.silu(plain.short_convolution(x[:, :channels], conv.double()))
    q = plain.unit_vectors(mixed[:, :qk].view(n, groups, dim)) * dim ** -0.5
    k = plain.unit_vectors(mixed[:, qk : 2 * qk].view(n, groups, dim))
    v = mixed[:, 2 * qk :].view(n, heads, vdim)
    beta = plain.sigmoid(x[:, channels : channels + heads])
    g = plain.head_decay(x[:, channels + heads : channels + 2 * heads], a_log.double(), dt_bias.double())
    close(torch.cat(decays), g, 3e-6)
    o = plain.delta_scan(q, k, v, g, beta)
    want = (plain.unit(o, eps) * w.double()).reshape(n, vw) * plain.silu(x[:, channels + 2 * heads : channels + 2 * heads + vw])
    sure = (o.pow(2).mean(dim=-1).sqrt() > 5e-3).repeat_interleave(vdim, dim=1)
    assert sure.double().mean() > 0.6
    got = torch.cat(outs).double()
    close(torch.where(sure, got, torch.zeros_like(got)), torch.where(sure, want, torch.zeros_like(want)), 2e-4 if dtype == torch.float32 else 1.5e-2)
    assert state[1].abs().max() > 0 and state[0].abs().max() == 0 and state[2].abs().max() == 0


@pytest.mark.parametrize("dtype", TYPES)
def test_batches_of_unequal_requests_equal_each_alone_and_a_cut_changes_no_bit(dtype):
    """Both recurrences, three requests of 1, 70 and 33 tokens in slots out of order.  In the 32-bit form the bits are the same
    alone, together and cut in three; otherwise the values are."""

    from llm_runtime_study_b200.ops import mixer_steps as M
    from llm_runtime_study_b200.ops import sequence_state as S

    torch.manual_seed(4)
    heads, dim, vdim, taps = 3, 20, 36, 3
    qk, vw = heads * dim, heads * vdim
    channels = 2 * qk + vw
    lengths, slots, starts = [1, 70, 33], [4, 0, 2], [0, 1, 71]
    n = sum(lengths)
    proj = dev(torch.randn(n, channels + 2 * heads).to(dtype))
    conv, zero, decay = dev(torch.randn(channels, taps)), torch.zeros(heads, device=DEV), dev(torch.tensor([0.9, 0.99, 1.0]))
    inv_freq = dev(torch.tensor(plain.frequencies(12, 40.0)[0]))
    fixed = dtype == torch.float32

    def run(pieces, kind):
        """pieces: a list of steps, each a list of (request, first token, tokens)."""

        state, kept = torch.zeros(5, heads, dim, vdim, device=DEV), torch.zeros(5, taps - 1, channels, device=DEV)
        out = torch.zeros(n, vw, device=DEV)
        for step in pieces:
            index = torch.cat([torch.arange(starts[r] + a, starts[r] + a + m) for r, a, m in step]).to(DEV)
            part = proj[index].contiguous()
            q_start, slot = ints(np.cumsum([0] + [m for _, _, m in step]).tolist()), ints([slots[r] for r, _, _ in step])
            sizes = dict(heads=heads, qk_heads=heads, dim=dim, vdim=vdim, state=state, q_start=q_start, slots=slot, fixed_order=fixed)
            if kind == "delta":
                q, k, v, g, beta = S.delta_prepare(
                    part, heads=heads, qk_heads=heads, dim=dim, vdim=vdim, beta_offset=channels, low_offset=channels + heads, rank=0, taps=conv,
                    conv_state=kept, a_log=zero, dt_bias=zero, a_up=None, q_start=q_start, slots=slot,
                    token_entry=ints([i for i, (_, _, m) in enumerate(step) for _ in range(m)]), unit_eps=1e-6, q_scale=1.0)
                S.conv_state_update(part, kept, q_start, slot)
                got = S.linear_scan(q, k, v, row_decay=g, beta=beta, **sizes)
            else:
                q, k = M.rotate_qk(part, heads=heads, head_dim=dim, positions=ints([p for _, a, m in step for p in range(a, a + m)]),
                                   rotary=(inv_freq, 12, False, 1.0))
                got = S.linear_scan(q, k, part[:, 2 * qk : channels], decay=decay, **sizes)
            out[index] = got
        return out

    for kind in ("delta", "retention"):
        together = run([[(0, 0, 1), (1, 0, 70), (2, 0, 33)]], kind)
        alone = run([[(r, 0, lengths[r])] for r in range(3)], kind)
        cut = run([[(2, 0, 2), (1, 0, 65)], [(1, 65, 5), (0, 0, 1), (2, 2, 30)], [(2, 32, 1)]], kind)
        for other in (alone, cut):
            if fixed:
                assert torch.equal(together, other)
            else:
                close(other, together.cpu().double(), 1e-5)


@pytest.mark.parametrize("dtype", TYPES)
def test_a_token_kept_over_two_thousand_others(dtype):
    """Decay 1, one key and value at position 2 and keys orthogonal to it behind: 2,000 tokens later the read-out with that key
    is its value.  With a decay it has shrunk by that power."""

    from llm_runtime_study_b200.ops import sequence_state as S

    n, dim, vdim = 2003, 16, 8
    q, k, v = torch.zeros(n, 2 * dim), torch.zeros(n, 2 * dim), torch.zeros(n, 2 * vdim)
    for h in range(2):
        k[:, h * dim + 1] = 1.0
        k[2, h * dim + 1] = 0.0
        k[2, h * dim] = 1.0
        q[:, h * dim] = 1.0
        v[:, h * vdim :(h + 1) * vdim] = 100.0
        v[2, h * vdim :(h + 1) * vdim] = torch.arange(1.0, vdim + 1)
    decay = dev(torch.tensor([1.0, 0.99853515625]))
    state = torch.zeros(1, 2, dim, vdim, device=DEV)
    out = []
    for a, b in ((0, 1000), (1000, 2001), (2001, 2002), (2002, 2003)):
        out.append(S.linear_scan(dev(q[a:b]), dev(k[a:b]), dev(v[a:b].to(dtype)), heads=2, qk_heads=2, dim=dim, vdim=vdim, state=state,
                                 q_start=ints([0, b - a]), slots=ints([0]), decay=decay, fixed_order=dtype == torch.float32).cpu().double())
    out = torch.cat(out)
    value = torch.arange(1.0, vdim + 1, dtype=torch.float64)
    for p in (2, 3, 999, 1000, 2000, 2001, 2002):
        close(out[p, :vdim], value, 1e-6)
        close(out[p, vdim:], value * 0.99853515625 ** (p - 2), 1e-4)


# ----------------------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("n", [97, 600])
@pytest.mark.parametrize("experts,top,groups,keep,width", [(8, 4, 2, 1, 64), (9, 3, 3, 2, 40), (5, 1, 5, 2, 50), (4, 2, 1, 1, 48), (40, 6, 8, 3, 128), (8, 8, 4, 4, 36)])
def test_the_router_with_sigmoid_scores_and_groups_scored_by_two(dtype, n, experts, top, groups, keep, width):
    """Choice and weights against the plain router for every token whose choice is clear; most choice scores are negative."""

    from llm_runtime_study_b200.ops import grouped as G

    torch.manual_seed(experts + width)
    h = torch.randn(n, width).to(dtype)
    router = torch.randn(experts + 1, width) * 0.3
    correction = torch.randn(experts) * 0.4 - 0.8
    margins = []
    ids, w = plain.route(h.double() @ router[:experts].double().T, correction.double(), top=top, groups=groups, keep_groups=keep, margins=margins)
    routing = G.route(dev(h), dev(router), None, top=top, score="sigmoid_all", correction=dev(correction), groups=groups, keep=keep, extra=1,
                      group_best=2, renormalise=True)
    close(routing.extra[:, 0], plain.sigmoid(h.double() @ router[experts].double()), 1e-5)
    got_ids, got_w = routing.ids.cpu(), routing.weights.cpu().double()
    clear = torch.tensor(margins) > 1e-4
    assert int(clear.sum()) > n // 2
    for t in range(n):
        if clear[t]:
            order = {int(e): j for j, e in enumerate(ids[t])}
            assert sorted(order) == sorted(got_ids[t].tolist()), t
            for j, e in enumerate(got_ids[t].tolist()):
                assert abs(float(got_w[t, j]) - float(w[t, order[e]])) < 1e-5
    if keep < groups:        # the group's two best decide, not its single best: the rules differ somewhere in these draws
        single = G.route(dev(h), dev(router), None, top=top, score="sigmoid_all", correction=dev(correction), groups=groups, keep=keep, extra=1,
                         renormalise=True)
        assert groups == experts or not torch.equal(single.ids, routing.ids)


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("width,ff,experts,top,groups,shared,n", [(64, 24, 9, 3, (3, 2), 40, 33), (128, 64, 8, 4, (4, 2), 32, 300), (50, 17, 4, 2, (1, 1), None, 12),
                                                                  (128, 64, 8, 2, (2, 1), 64, 1)])
def test_experts_with_a_gated_shared_one(dtype, width, ff, experts, top, groups, shared, n):
    """The whole feed-forward, summed and in pieces."""

    from llm_runtime_study_b200.ops import block_steps as B
    from llm_runtime_study_b200.parts import FEED_FORWARDS, Runtime

    torch.manual_seed(width + n)
    part = FEED_FORWARDS.build({"kind": "routed_experts", "hidden_size": width, "intermediate_size": ff, "experts": experts, "top": top, "act": "silu_glu",
                                "router_bias": False, "score": "sigmoid_all", "correction": True, "groups": groups[0], "keep": groups[1], "group_best": 2,
                                "renormalise": True, "shared_size": shared, "shared_gate": shared is not None})
    weights = {name: (torch.randn(spec.shape) * (0.3 if len(spec.shape) == 2 else 1.0)).to(dtype) for name, spec in part.tensor_specs().items()}
    part.load(weights, Runtime(torch.device(DEV), dtype))
    x = torch.randn(n, width).to(dtype)
    margins = []
    store = plain.round_bfloat16 if dtype == torch.bfloat16 else plain.keep
    mlp = {"router": {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]}}, "shared": {"ff": shared} if shared else None}
    want = plain.moe(x.double(), {k: v.double() for k, v in weights.items()}, mlp, store, margins)
    clear = torch.tensor(margins) > 1e-4
    got = part.forward(dev(x), None)
    assert part.returns_gated_pieces == (shared is not None)
    pieces = part.forward(dev(x), None, pieces=True)
    summed = torch.zeros(n, width, device=DEV)
    B.sum_norm(summed, pieces, torch.ones(width, device=DEV), 1e-6, alpha=0.0, centred=False)
    tol = 1e-5 if dtype == torch.float32 else 2e-2
    close(got.cpu()[clear], want[clear], tol)
    close(summed.cpu()[clear], plain.unit(want, 1e-6)[clear], 3 * tol)


# ------------------------------------------------------------------------------------------- whole models
LENGTHS = {"A": [1, 2, 5, 23, 64, 65, 131], "B": [3, 17, 48, 70, 1, 129], "C": [140, 2, 37, 66, 300]}


@pytest.fixture(scope="module", params=[(n, d) for n in ("A", "B", "C") for d in ("float32", "bfloat16")], ids=lambda p: f"{p[0]}-{p[1]}")
def setup(request, tmp_path_factory):
    from llm_runtime_study_b200.engine.runtime import load

    name, dtype = request.param
    config, seed, page = helpers.REFOLIX[name]
    path, weights = helpers.make_refolix_dir(tmp_path_factory.mktemp(f"refolix{name}{dtype}"), config, seed, torch_dtype=dtype)
    rng = random.Random(seed + 1)
    requests = {f"r{i}": helpers.random_tokens(rng, config["vocab"], n) for i, n in enumerate(LENGTHS[name])}
    store = plain.round_bfloat16 if dtype == "bfloat16" else plain.keep
    expected, clear = {}, {}
    for rid, tokens in requests.items():
        margins = []
        expected[rid] = plain.forward(config, weights, tokens, store=store, margins=margins)
        clear[rid] = helpers.rows_without_a_close_call(margins, len(tokens))
        assert len(tokens) < 20 or clear[rid].double().mean() > 0.4
    loaded = load(path, device=DEV, dtype=dtype, strict_dtype=False)
    return dict(name=name, dtype=dtype, config=config, page=page, path=path, requests=requests, plain=expected, clear=clear, loaded=loaded, weights=weights)


def _replay(setup, steps, *, max_requests=4):
    from llm_runtime_study_b200.engine.replay import TraceReplayer

    replayer = TraceReplayer(setup["loaded"], max_tokens=helpers.pool_tokens(steps), page_size=setup["page"], max_requests=max_requests)
    outputs = {}
    for record in steps:
        rows = replayer.run_step(record)
        if rows is not None:
            outputs[record["step"]] = torch.from_numpy(np.array(rows))
    manager = replayer.runner.manager
    manager.check()
    assert manager.active_sequences == 0 and manager.all_free and manager.free_slots == max_requests
    return helpers.collect_logits(steps, outputs)


def _compare(setup, got, requests=None):
    for rid, tokens in (requests or setup["requests"]).items():
        assert sorted(got[rid]) == list(range(len(tokens))), rid
        rows = torch.stack([got[rid][p] for p in range(len(tokens))]).double()
        if setup["dtype"] == "bfloat16":
            want = setup["plain"][rid]
            err = (rows - want).pow(2).mean(dim=1).sqrt() / want.pow(2).mean(dim=1).sqrt()
            assert torch.isfinite(err).all()
            err = torch.where(setup["clear"][rid], err, torch.zeros_like(err))
            assert float(err.max()) <= BF16_WORST, (rid, int(err.argmax()), float(err.max()))
            over = int((err > BF16_USUAL).sum())
            assert over <= max(1, len(tokens) // 10), f"request {rid}: {over} of {len(tokens)} rows beyond {BF16_USUAL}: {err}"
            continue
        bad, err, top = helpers.first_wrong_row(rows, setup["plain"][rid], TOL[setup["dtype"]])
        assert bad is None, f"request {rid}: first wrong position {bad} of {len(tokens)}, rms and largest |diff| / rms {err:.3e}, {top:.3e}"


def test_whole_prompts(setup):
    _compare(setup, _replay(setup, helpers.trace_whole(setup["requests"])))


def test_prefill_then_token_by_token(setup):
    _compare(setup, _replay(setup, helpers.trace_decode_tail(setup["requests"], tail=40)))


def test_portions_down_to_two_tokens(setup):
    rng = random.Random(5)
    _compare(setup, _replay(setup, helpers.trace_chunked(setup["requests"], rng, sizes=(2, 3, 2, 7, 13, 16, 17, 31))))


def test_mixed_batches_with_slots_and_pages_used_again(setup):
    """Three slots for up to seven requests, portions beside single tokens, and a pool sized for what is live."""

    steps = helpers.trace_mixed(setup["requests"], random.Random(9), live_max=3, tail=6)
    _compare(setup, _replay(setup, steps, max_requests=3))


def test_every_token_decoded_alone(setup):
    """A sequence fed one token a step from its first token: the first tokens, long decoding."""

    requests = {rid: tokens for rid, tokens in setup["requests"].items() if len(tokens) in (23, 131, 70, 66)}
    _compare(setup, _replay(setup, helpers.trace_decode_tail(requests, tail=10_000)), requests)


def test_a_cut_changes_no_bit_in_float32(setup):
    if setup["dtype"] != "float32":
        pytest.skip("the 32-bit path is the one whose sums have an order fixed by the position")
    whole = _replay(setup, helpers.trace_whole(setup["requests"]))
    cut = _replay(setup, helpers.trace_chunked(setup["requests"], random.Random(1), sizes=(2, 5, 9)))
    for rid, rows in whole.items():
        for p, row in rows.items():
            assert torch.equal(row, cut[rid][p]), (rid, p)


def test_a_reused_slot_starts_from_zero(setup):
    """One slot: the second request takes the first one's states and pages."""

    requests = {rid: tokens for rid, tokens in setup["requests"].items() if len(tokens) in (23, 17, 48, 65, 37, 66)}
    _compare(setup, _replay(setup, helpers.trace_chunked(requests, random.Random(3), sizes=(7, 16)), max_requests=1), requests)


def test_greedy_generation_through_the_engine(setup):
    """``Engine.generate`` with its scheduler (prompt portions, batching, graph decode) gives the plain model's greedy tokens."""

    from llm_runtime_study_b200.engine.engine import Engine
    from llm_runtime_study_b200.sampling import SamplingConfig

    if setup["dtype"] != "float32":
        pytest.skip("greedy ties are decided by rounding in bfloat16")
    config, weights = setup["config"], setup["weights"]
    prompts = [setup["requests"]["r3"][:19], setup["requests"]["r2"][:30], setup["requests"]["r1"][:20] + [3, 1, 4]]
    new = 12
    want = []
    for prompt in prompts:
        tokens = list(prompt)
        for _ in range(new):
            tokens.append(int(plain.forward(config, weights, tokens)[-1].argmax()))
        want.append(tokens[len(prompt):])
    engine = Engine.from_model_dir(setup["path"], device=DEV, dtype="float32", max_seq_len=64, max_batch_size=2, page_size=setup["page"],
                                   max_tokens_per_step=16, strict_dtype=False)
    got = [[] for _ in prompts]
    for index, event in engine.generate(prompts, max_new_tokens=new, sampling=SamplingConfig(temperature=0.0)):
        if event.token_id is not None:
            got[index].append(event.token_id)
    assert got == want


def test_command_line_and_trace_runner(tmp_path):
    """The command line writes a folder of random weights for the design and generates from it; the trace runner,
    started as a program with four request slots, replays a mixed trace on that folder."""

    import io
    import json
    import subprocess
    import sys
    from pathlib import Path

    from llm_runtime_study_b200.cli import main
    from llm_runtime_study_b200.weights import Checkpoint

    config = helpers.REFOLIX_A
    config_path = tmp_path / "config.json"
    config_path.write_text(json.dumps(config))
    out, err = io.StringIO(), io.StringIO()
    code = main(["--model", str(tmp_path / "m"), "--random-weights", str(config_path), "--weights-seed", "4",
                 "--prompt-ids", "5 17 3 90", "--max-new-tokens", "5", "--max-seq-len", "64", "--dtype", "float32", "--no-stream"],
                output=out, error=err)
    assert code == 0, err.getvalue()
    generated = [int(t) for t in out.getvalue().splitlines()[0].split()]
    weights = Checkpoint.from_model_dir(tmp_path / "m").get_tensors()
    tokens = [5, 17, 3, 90]
    for got in generated:
        logits = plain.forward(config, weights, tokens)[-1]
        top = torch.topk(logits, 2).values
        if float(top[0] - top[1]) < 1e-4:        # a tie: either token is right, and what follows differs
            break
        assert got == int(logits.argmax())
        tokens.append(got)
    rng = random.Random(2)
    requests = {f"q{i}": helpers.random_tokens(rng, config["vocab"], n) for i, n in enumerate([9, 30, 2, 17, 40])}
    steps = helpers.trace_mixed(requests, rng, live_max=4, tail=5)
    root = Path(__file__).resolve().parent.parent
    run = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32",
                          "--out", str(tmp_path / "out"), "--max-tokens", str(helpers.pool_tokens(steps))],
                         input=helpers.dump_trace(steps), capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [line for line in run.stdout.splitlines() if line.startswith("done ")] == [f"done {s['step']}" for s in steps]
    outputs = {s["step"]: torch.from_numpy(np.fromfile(tmp_path / "out" / f"{s['step']}.f32", dtype="<f4").reshape(-1, config["vocab"]))
               for s in steps if any(e["want"] for e in s["entries"])}
    got = helpers.collect_logits(steps, outputs)
    for rid, toks in requests.items():
        want = plain.forward(config, weights, toks)
        rows = torch.stack([got[rid][p] for p in range(len(toks))]).double()
        bad, rms_err, top_err = helpers.first_wrong_row(rows, want, TOL["float32"])
        assert bad is None, (rid, bad, rms_err, top_err)
