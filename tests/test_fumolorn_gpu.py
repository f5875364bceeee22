"""Fumolorn through the framework against the plain implementation: every mechanism's kernels alone (with inputs made so that
a sink, a far key, a page's border or a lost state shows), then whole models under every way of cutting the work (whole
prompts, decoding token by token, portions down to two tokens, mixed batches whose pages and slots are used again), in 32-bit
and in bfloat16, and greedy generation through the engine's own entry point."""

import random
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from tests import helpers
from tests.plain import fumolorn_plain as plain

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
# a row of logits against the plain model in 64-bit, as fractions of the row's root mean square: (rms, largest).
# float32 is the sharp comparison.  bfloat16: the plain model rounds its activations where the engine stores them; a rounding
# that falls the other way moves single rows, so a request passes when at most a tenth of its rows (or one) is beyond
# BF16_USUAL and none beyond BF16_WORST.  A wrong state, slot or page moves every row after it.
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
                           q_lens=list(q_lens), kv_lens=list(lengths), max_kv_len=max(lengths))


# ------------------------------------------------------------------------------------------ embedding
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("hidden,bigram", [(50, True), (64, False), (129, True)])
def test_normed_embedding_across_cuts(dtype, hidden, bigram):
    """Two requests cut into portions, their entries in changing order: token before the portion, first token, norm, rounding."""

    from llm_runtime_study_b200.ops import functional as F

    torch.manual_seed(hidden)
    vocab, buckets, prev, cur, scale, eps = 40, 11, 3_000_000_019, 7, 2.5, 1e-5
    table, rows, w = torch.randn(vocab, hidden).to(dtype), torch.randn(buckets + 1, hidden).to(dtype), 1 + 0.3 * torch.randn(hidden)
    config = {"embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": prev, "mul_cur": cur} if bigram else None}, "norm": {"eps": eps}}
    weights = {"embed": table, "bigram": rows, "embed.norm": w}
    rng = random.Random(1)
    tokens = [helpers.random_tokens(rng, vocab, n) for n in (13, 9)]
    want = [plain.embedding(t, weights, config, torch.float64) for t in tokens]
    kept = torch.zeros(4, 1, dtype=torch.int32, device=DEV)
    at = [0, 0]
    for step in ([(0, 2), (1, 1)], [(1, 3), (0, 1)], [(0, 1)], [(1, 5), (0, 9)]):
        ids = [t for r, n in step for t in tokens[r][at[r]:at[r] + n]]
        pos = [p for r, n in step for p in range(at[r], at[r] + n)]
        entry = [i for i, (_, n) in enumerate(step) for _ in range(n)]
        start = np.cumsum([0] + [n for _, n in step]).tolist()
        out = F.embedding_sum(ints(ids), dev(table), dev(rows) if bigram else None, positions=ints(pos), token_entry=ints(entry),
                              q_start=ints(start), slots=ints([r + 1 for r, _ in step]), previous=kept if bigram else None, freq=None,
                              buckets=buckets, mul_prev=prev, mul_cur=cur, scale=scale, norm=(dev(w), eps),
                              rounded_dtype=dtype if dtype != torch.float32 else None)
        if dtype != torch.float32:
            out, rounded = out
            assert torch.equal(rounded, out.to(dtype))
        for i, (r, n) in enumerate(step):
            close(out[start[i]:start[i + 1]], want[r][at[r]:at[r] + n], 2e-6)
            at[r] += n
    assert at == [13, 9]


# ------------------------------------------------------------------------------------------- rotation
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rot,rot_dims,interleaved,factor", [(12, 12, True, 1.3), (16, 8, True, 1.0), (8, 8, False, 0.7), (2, 2, True, 1.1)])
def test_rotation_of_the_shared_key_part_and_of_the_queries(dtype, rot, rot_dims, interleaved, factor):
    from llm_runtime_study_b200.ops import mixer_steps as M

    torch.manual_seed(rot)
    q_rank, kv_rank, page, eps = 20, 24, 8, 1e-5
    lengths, starts = [19, 6], [1000, 3]
    n = sum(lengths)
    rows = torch.randn(n, q_rank + kv_rank + rot + 3).to(dtype)
    qw, kw = 1 + 0.1 * torch.randn(q_rank), 1 + 0.1 * torch.randn(kv_rank)
    freq = [1000.0 ** (-2.0 * i / rot_dims) for i in range(rot_dims // 2)]
    inv_freq = torch.tensor(freq, dtype=torch.float64).float()
    ctx = _ctx([s + m for s, m in zip(starts, lengths)], lengths)
    table, pages = _pages(n, page, [s + m for s, m in zip(starts, lengths)])
    pool = torch.zeros(pages, page, kv_rank + rot, dtype=dtype, device=DEV)
    M.latent_prepare(dev(rows), q_offset=0, q_rank=q_rank, q_weight=dev(qw), eps=eps, positions=ctx.positions, token_entry=ctx.token_entry,
                     kv_offset=q_rank, kv_rank=kv_rank, kv_weight=dev(kw), rot=rot, rot_dims=rot_dims, inv_freq=dev(inv_freq),
                     block_table=dev(table), page_size=page, pool=pool, interleaved=interleaved, rot_factor=factor)

    def rotated(x, positions):
        if not interleaved:       # the same pairs in the other layout
            half = rot_dims // 2
            order = [c for i in range(half) for c in (i, i + half)] + list(range(rot_dims, rot))
            back = [order.index(c) for c in range(rot)]
            return plain.rotate_pairs(x[..., order], positions, [f.item() for f in inv_freq.double()], factor)[..., back]
        return plain.rotate_pairs(x, positions, [f.item() for f in inv_freq.double()], factor)

    positions = ctx.positions.cpu()
    tol = 2e-4 if dtype == torch.float32 else 3e-2      # float32 angles of a thousand turns' worth of radians
    want = rotated(rows.double()[:, q_rank + kv_rank : q_rank + kv_rank + rot], positions)
    entry = ctx.token_entry.cpu()
    got = torch.stack([pool[table[int(entry[t]), int(positions[t]) // page], int(positions[t]) % page] for t in range(n)])
    close(got[:, kv_rank:], want, tol)
    heads, head, off = 3, 10 + rot, 10
    src = torch.randn(n, heads * head).to(dtype)
    dst = torch.zeros(n, heads * (5 + rot), dtype=dtype, device=DEV)
    M.rope_slice(dev(src), dst, heads=heads, src_head=head, src_offset=off, dst_head=5 + rot, dst_offset=5, rot=rot, rot_dims=rot_dims,
                 inv_freq=dev(inv_freq), positions=ctx.positions, interleaved=interleaved, rot_factor=factor)
    close(dst.view(n, heads, 5 + rot)[..., 5:], rotated(src.double().view(n, heads, head)[..., off:], positions), tol)
    assert dst.view(n, heads, 5 + rot)[..., :5].abs().max() == 0


# ------------------------------------------------------------------------------------------ attention
SINKS = [-30.0, 3.0, 0.0, 40.0, 1.0, -2.0, 6.0]      # none to speak of, some, and one that swallows nearly everything


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("heads,rank,rot,page", [(3, 40, 12, 4), (6, 64, 16, 16), (4, 32, 16, 8), (70, 48, 0, 16), (5, 512, 64, 16), (1, 24, 4, 16)])
@pytest.mark.parametrize("q_lens", [[130, 41], [1, 1], [2, 37]])
def test_latent_attention_with_sinks(dtype, heads, rank, rot, page, q_lens):
    """Portions behind cached rows and single tokens, through the tensor-core kernel where it takes the sizes and the CUDA-core
    kernel elsewhere."""

    from llm_runtime_study_b200.ops import attention_latent

    torch.manual_seed(rank + heads)
    lengths, d = [130, 41], rank + rot
    table, pages = _pages(rank, page, lengths)
    rows = [0.5 * torch.randn(m, d).to(dtype) for m in lengths]
    pool = torch.zeros(pages, page, d, dtype=dtype)
    for e, m in enumerate(lengths):
        for t in range(m):
            pool[table[e, t // page], t % page] = rows[e][t]
    sink = torch.tensor([SINKS[h % len(SINKS)] for h in range(heads)])
    q = (0.5 * torch.randn(sum(q_lens), heads, d)).to(dtype)
    got = attention_latent.latent_attention(dev(q), dev(pool), _ctx(lengths, q_lens), dev(table), value_dim=rank, scale=0.3, sink=dev(sink))
    at = 0
    for e, (m, k) in enumerate(zip(lengths, q_lens)):
        full_q = torch.zeros(m, heads, d, dtype=torch.float64)
        full_q[m - k:] = q[at:at + k].double()
        keys = rows[e].double()[:, None, :]
        want = plain.sink_attention(full_q, keys, keys[:, :, :rank], scale=0.3, sink=sink.double())[m - k:]
        close(got[at:at + k], want, tolerance(dtype))
        at += k


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("page,marked", [(16, 15), (16, 16), (8, 63), (4, 0), (16, 3), (16, 1499)])
def test_a_far_key_and_a_sink_that_matches_it(dtype, page, marked):
    """One key of 1,500 stands out by as much as the sink of the second head does: the first head's result is its value, the
    second's half of it, the third's (whose sink is larger) nearly zero; for a single token, whose keys are cut into parts, and
    for a portion."""

    from llm_runtime_study_b200.ops import attention_latent

    torch.manual_seed(marked)
    heads, rank, rot, length, new = 3, 32, 16, 1500, 3
    d = rank + rot
    rows = 0.1 * torch.randn(length, d)
    rows[marked] = 0.0
    rows[marked, 1] = 8.0
    q = torch.zeros(length, heads, d)
    q[:, :, 1] = 5.0
    rows, q = rows.to(dtype), q.to(dtype)
    sink = torch.tensor([-60.0, 40.0, 60.0])
    table, pages = _pages(marked, page, [length])
    pool = torch.zeros(pages, page, d, dtype=dtype)
    for t in range(length):
        pool[table[0, t // page], t % page] = rows[t]
    for k in (1, new):
        got = attention_latent.latent_attention(dev(q[length - k:].contiguous()), dev(pool), _ctx([length], [k]), dev(table), value_dim=rank, scale=1.0,
                                                sink=dev(sink)).cpu().double()
        for row in got:
            if int(marked) == length - 1 and row is not got[-1]:
                continue
            value = rows[marked, :rank].double()
            assert (row[0] - value).abs().max() < 0.05 and (row[1] - value / 2).abs().max() < 0.05 and row[2].abs().max() < 0.05
    keys = rows.double()[:, None, :]
    close(got, plain.sink_attention(q.double(), keys, keys[:, :, :rank], scale=1.0, sink=sink.double())[length - new:], tolerance(dtype))


def test_single_tokens_whose_keys_are_cut_into_parts_count_the_sink_once():
    from llm_runtime_study_b200.ops import attention_latent

    torch.manual_seed(8)
    heads, rank, rot, page = 6, 64, 16, 16
    lengths, d = [1500, 3, 700], rank + rot
    assert attention_latent.decode_splits(len(lengths), heads, max(lengths)) > 1
    sink = torch.tensor(SINKS[:heads])
    table, pages = _pages(0, page, lengths)
    rows = [0.5 * torch.randn(m, d).bfloat16() for m in lengths]
    pool = torch.zeros(pages, page, d, dtype=torch.bfloat16)
    for e, m in enumerate(lengths):
        for t in range(m):
            pool[table[e, t // page], t % page] = rows[e][t]
    q = (0.5 * torch.randn(3, heads, d)).bfloat16()
    got = attention_latent.latent_attention(dev(q), dev(pool), _ctx(lengths, [1, 1, 1]), dev(table), value_dim=rank, scale=0.3, sink=dev(sink))
    for e, m in enumerate(lengths):
        full_q = torch.zeros(m, heads, d, dtype=torch.float64)
        full_q[m - 1] = q[e].double()
        keys = rows[e].double()[:, None, :]
        close(got[e], plain.sink_attention(full_q, keys, keys[:, :, :rank], scale=0.3, sink=sink.double())[m - 1], 2e-2)


# ---------------------------------------------------------------------------------------- recurrences
CUTS = [[1, 2, 1, 9, 3, 40, 33, 64], [153], [2, 151], [32, 32, 32, 57]]


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("cuts", CUTS)
@pytest.mark.parametrize("heads,dim,vdim,cap", [(1, 24, 40, 5.0), (5, 9, 33, 15.0), (2, 130, 64, 1.5), (3, 64, 31, 10.0)])
def test_matrix_memory_across_cuts(dtype, cuts, heads, dim, vdim, cap):
    """Gates, scan and read-out of a sequence fed in portions, in a slot between two others: the rows equal the plain
    whole-sequence values, the three states carry over, and the neighbours' slots stay untouched."""

    from llm_runtime_study_b200.ops import sequence_state as S

    torch.manual_seed(dim + len(cuts))
    qk, vw, n, eps = heads * dim, heads * vdim, sum(cuts), 1e-5
    proj = torch.randn(n, 2 * (qk + vw) + 2 * heads + 3)
    proj[:, 2 * (qk + vw) :] *= 4.0
    proj = proj.to(dtype)
    ib, fb, w = torch.randn(heads), 3 + torch.randn(heads), 1 + 0.3 * torch.randn(vw)
    state, norm_state = torch.zeros(3, heads, dim, vdim, device=DEV), torch.zeros(3, heads, dim, device=DEV)
    m_state = torch.zeros(3, heads, device=DEV)
    slot, outs, raws, divisors, at = ints([1]), [], [], [], 0
    for m in cuts:
        part, q_start = dev(proj[at:at + m].contiguous()), ints([0, m])
        decay, gain, floor = S.memory_gates(part, heads=heads, i_offset=2 * (qk + vw), f_offset=2 * (qk + vw) + heads, i_bias=dev(ib),
                                            f_bias=dev(fb), cap=cap, m_state=m_state, q_start=q_start, slots=slot)
        out, den = S.linear_scan_row_gates(part[:, :qk], part[:, qk : 2 * qk], part[:, 2 * qk : 2 * qk + vw], heads=heads, dim=dim, vdim=vdim,
                                           decay=decay, gain=gain, state=state, norm_state=norm_state, q_start=q_start, slots=slot,
                                           q_scale=dim ** -0.5, fixed_order=dtype == torch.float32)
        divisors.append((torch.maximum(den.abs(), floor) + 1e-6).repeat_interleave(vdim, dim=1).cpu())
        raws.append((out.cpu() / divisors[-1]))
        outs.append(S.group_norm_gate(out, dev(w), eps, part, gate_offset=2 * qk + vw, group=vdim, divisor=(den, floor, 1e-6), out_dtype=dtype).cpu())
        at += m
    x = proj.double()
    q, k = x[:, :qk].view(n, heads, dim) * dim ** -0.5, x[:, qk : 2 * qk].view(n, heads, dim)
    v = x[:, 2 * qk : 2 * qk + vw].view(n, heads, vdim)
    zi, zf = x[:, 2 * (qk + vw) : 2 * (qk + vw) + heads], x[:, 2 * (qk + vw) + heads : 2 * (qk + vw) + 2 * heads]
    li, lf = plain.mlstm_gates(zi + ib.double(), zf + fb.double(), cap)
    o = plain.mlstm_scan(q, k, v, li, lf)
    # where n . q nearly cancels the quotient magnifies its rounding: compared times the divisor
    divisor = torch.cat(divisors).double()
    close(torch.cat(raws).double() * divisor, o.reshape(n, vw) * divisor, 2e-5)
    want = plain.unit(o, eps).reshape(n, vw) * w.double() * plain.sigmoid(x[:, 2 * qk + vw : 2 * (qk + vw)])
    # likewise where a head's read-out nearly cancels and is divided by its root mean square
    sure = ((o.reshape(n, vw) * divisor).view(n, heads, vdim).pow(2).mean(dim=-1).sqrt() > 1e-2).repeat_interleave(vdim, dim=1)
    assert sure.double().mean() > 0.5
    got = torch.cat(outs).double()
    close(torch.where(sure, got, torch.zeros_like(got)), torch.where(sure, want, torch.zeros_like(want)), 3e-4 if dtype == torch.float32 else 1e-2)
    for s in (state, norm_state, m_state):
        assert s[1].abs().max() > 0 and s[0].abs().max() == 0 and s[2].abs().max() == 0


@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("cuts", CUTS)
@pytest.mark.parametrize("heads,dim,vdim,rank,tau", [(1, 40, 7, 16, 1.0), (3, 12, 20, 5, 8.0), (2, 200, 33, 16, 16.0), (4, 64, 64, 3, 2.0)])
def test_gated_linear_attention_across_cuts(dtype, cuts, heads, dim, vdim, rank, tau):
    from llm_runtime_study_b200.ops import sequence_state as S

    torch.manual_seed(dim + len(cuts))
    qk, vw, n, eps = heads * dim, heads * vdim, sum(cuts), 1e-5
    proj = torch.randn(n, 2 * (qk + vw) + rank + 1).to(dtype)
    a2, a2b, w = torch.randn(qk, rank).to(dtype), torch.randn(qk), 1 + 0.3 * torch.randn(vdim)
    state = torch.zeros(3, heads, dim, vdim, device=DEV)
    slot, outs, at = ints([1]), [], 0
    for m in cuts:
        part, q_start = dev(proj[at:at + m].contiguous()), ints([0, m])
        alpha = S.channel_decay(part, dev(a2.t().contiguous()), dev(a2b), offset=2 * (qk + vw), tau=tau)
        out = S.linear_scan(part[:, :qk], part[:, qk : 2 * qk], part[:, 2 * qk : 2 * qk + vw], heads=heads, qk_heads=heads, dim=dim, vdim=vdim,
                            state=state, q_start=q_start, slots=slot, gate=alpha, q_scale=dim ** -0.5, fixed_order=dtype == torch.float32)
        outs.append(S.group_norm_gate(out, dev(w), eps, part, gate_offset=2 * qk + vw, act="silu", out_dtype=dtype).cpu())
        at += m
    x = proj.double()
    q, k = x[:, :qk].view(n, heads, dim) * dim ** -0.5, x[:, qk : 2 * qk].view(n, heads, dim)
    v = x[:, 2 * qk : 2 * qk + vw].view(n, heads, vdim)
    want_alpha = plain.channel_decay(x[:, 2 * (qk + vw) : 2 * (qk + vw) + rank] @ a2.double().T + a2b.double(), tau)
    close(alpha, want_alpha[n - cuts[-1]:], 3e-6)
    o = plain.gla_scan(q, k, v, want_alpha.view(n, heads, dim))
    want = plain.rms_norm(o, w.double(), eps).reshape(n, vw) * plain.silu(x[:, 2 * qk + vw : 2 * (qk + vw)])
    sure = (o.pow(2).mean(dim=-1).sqrt() > 1e-2).repeat_interleave(vdim, dim=1)
    got = torch.cat(outs).double()
    close(torch.where(sure, got, torch.zeros_like(got)), torch.where(sure, want, torch.zeros_like(want)), 1e-4 if dtype == torch.float32 else 1e-2)
    assert state[1].abs().max() > 0 and state[0].abs().max() == 0 and state[2].abs().max() == 0


@pytest.mark.parametrize("dtype", TYPES)
def test_batches_of_unequal_requests_equal_each_alone_and_a_cut_changes_no_bit(dtype):
    """Both recurrences, three requests of 1, 70 and 33 tokens in slots out of order.  In the 32-bit form the bits are the same
    alone, together and cut in two; otherwise the values are."""

    from llm_runtime_study_b200.ops import sequence_state as S

    torch.manual_seed(4)
    heads, dim, vdim, rank = 3, 20, 36, 8
    qk, vw = heads * dim, heads * vdim
    lengths, slots = [1, 70, 33], [4, 0, 2]
    n = sum(lengths)
    starts = [0, 1, 71, 104]
    proj = dev(torch.randn(n, 2 * qk + vw + 2 * heads + rank).to(dtype))
    zero, three = torch.zeros(heads, device=DEV), torch.full((heads,), 3.0, device=DEV)
    up, bias = dev(torch.randn(rank, qk).to(dtype)), dev(torch.randn(qk))
    fixed = dtype == torch.float32

    def run(pieces, kind):
        """pieces: a list of steps, each a list of (request, first token, tokens)."""

        shape = (5, heads, dim, vdim)
        state, norm_state, m_state = torch.zeros(shape, device=DEV), torch.zeros(shape[:3], device=DEV), torch.zeros(shape[:2], device=DEV)
        out = torch.zeros(n, vw, device=DEV)
        for step in pieces:
            index = torch.cat([torch.arange(starts[r] + a, starts[r] + a + m) for r, a, m in step]).to(DEV)
            part = proj[index].contiguous()
            q_start, slot = ints(np.cumsum([0] + [m for _, _, m in step]).tolist()), ints([slots[r] for r, _, _ in step])
            args = (part[:, :qk], part[:, qk : 2 * qk], part[:, 2 * qk : 2 * qk + vw])
            if kind == "memory":
                decay, gain, floor = S.memory_gates(part, heads=heads, i_offset=2 * qk + vw, f_offset=2 * qk + vw + heads, i_bias=zero, f_bias=three,
                                                    cap=9.0, m_state=m_state, q_start=q_start, slots=slot)
                got, den = S.linear_scan_row_gates(*args, heads=heads, dim=dim, vdim=vdim, decay=decay, gain=gain, state=state,
                                                   norm_state=norm_state, q_start=q_start, slots=slot, fixed_order=fixed)
                got = got / (torch.maximum(den.abs(), floor) + 1e-6).repeat_interleave(vdim, dim=1)
            else:
                alpha = S.channel_decay(part, up, bias, offset=2 * qk + vw + 2 * heads, tau=4.0)
                got = S.linear_scan(*args, heads=heads, qk_heads=heads, dim=dim, vdim=vdim, gate=alpha, state=state, q_start=q_start, slots=slot,
                                    fixed_order=fixed)
            out[index] = got
        return out

    for kind in ("memory", "linear"):
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
    """Both recurrences hold what one early token stored (a key of its own, gates that keep it) until a query asks for it 2,000
    tokens later; the tokens in between use other keys."""

    from llm_runtime_study_b200.ops import sequence_state as S

    n, dim, vdim = 2050, 16, 8
    torch.manual_seed(0)
    k, v, q = torch.zeros(n, dim), torch.randn(n, vdim), torch.zeros(n, dim)
    k[:, 1:] = 0.3 * torch.randn(n, dim - 1)
    k[5] = 0.0
    k[5, 0], v[5] = 4.0, torch.arange(1.0, vdim + 1)
    q[:, 0] = 1.0
    q, k, v = (dev(t.to(dtype)) for t in (q, k, v))
    want = 4.0 * torch.arange(1.0, vdim + 1, dtype=torch.float64)
    q_start, slot = ints([0, n]), ints([0])
    state = torch.zeros(1, 1, dim, vdim, device=DEV)
    proj = torch.zeros(n, 2, dtype=dtype, device=DEV)          # logits: the input gate stays at e^0, the forget gate nearly at 1
    decay, gain, floor = S.memory_gates(proj, heads=1, i_offset=0, f_offset=1, i_bias=torch.zeros(1, device=DEV),
                                        f_bias=torch.full((1,), 60.0, device=DEV), cap=14.0, m_state=torch.zeros(1, 1, device=DEV), q_start=q_start, slots=slot)
    out, den = S.linear_scan_row_gates(q, k, v, heads=1, dim=dim, vdim=vdim, decay=decay, gain=gain, state=state,
                                       norm_state=torch.zeros(1, 1, dim, device=DEV), q_start=q_start, slots=slot, fixed_order=dtype == torch.float32)
    got = (out / (torch.maximum(den.abs(), floor) + 1e-6)).cpu().double()
    assert got[4].abs().max() == 0
    assert (got[[5, 6, 1000, n - 1]] - want / 4.0).abs().max() < 1e-2
    state.zero_()
    alpha = S.channel_decay(torch.zeros(n, 1, dtype=dtype, device=DEV), torch.zeros(1, dim, dtype=dtype, device=DEV),
                            torch.full((dim,), 15.0, device=DEV), offset=0, tau=16.0)
    got = S.linear_scan(q, k, v, heads=1, qk_heads=1, dim=dim, vdim=vdim, state=state, q_start=q_start, slots=slot, gate=alpha,
                        fixed_order=dtype == torch.float32).cpu().double()
    assert got[4].abs().max() == 0 and (got[[5, 6, 1000, n - 1]] - want).abs().max() < 1e-2


# --------------------------------------------------------------- feed-forward, norm on the output, soft cap
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("width,ff", [(64, 72), (128, 256), (50, 33), (512, 1024)])
@pytest.mark.parametrize("n", [1, 13, 40, 300])
def test_gated_feed_forward(dtype, width, ff, n):
    """Every kernel a row count reaches: weight-streaming, library, tcgen05, and the activation as a kernel of its own."""

    from llm_runtime_study_b200.parts import Runtime
    from llm_runtime_study_b200.parts.mlp import GatedMLP

    torch.manual_seed(n + ff)
    w = {"gate": (3 * torch.randn(ff, width) / width ** 0.5).to(dtype), "up": (torch.randn(ff, width) / width ** 0.5).to(dtype),
         "down": (torch.randn(width, ff) / ff ** 0.5).to(dtype)}
    part = GatedMLP(hidden_size=width, intermediate_size=ff, act="gelu_tanh", names=("gate", "up", "down"))
    part.load(w, Runtime(torch.device(DEV), dtype))
    x = torch.randn(n, width).to(dtype)
    store = plain.keep if dtype == torch.float32 else plain.round_bfloat16
    close(part.forward(dev(x), None), plain.gated_mlp(x.double(), {k: t.double() for k, t in w.items()}, store), tolerance(dtype))


def test_the_activation_far_from_zero():
    from llm_runtime_study_b200.ops import functional as F

    g = torch.tensor([-1e20, -200.0, -9.0, -3.0, -1e-3, 0.0, 1e-3, 0.7, 5.0, 200.0, 1e15, 1e3], dtype=torch.float32)
    row = torch.cat([g, torch.ones_like(g)])[None]
    want = plain.gelu_tanh(g.double())
    got = F.silu_mul(dev(row), "gelu_tanh").cpu().double()[0]
    assert torch.isfinite(got).all() and ((got - want).abs() <= 1e-6 * want.abs() + 1e-7).all()


def test_the_factor_on_a_sublayers_output_and_the_soft_cap():
    from llm_runtime_study_b200.ops import functional as F
    from llm_runtime_study_b200.ops import mixer_steps as M

    torch.manual_seed(1)
    for hidden in (56, 49):
        out, w, resid = 3 * torch.randn(5, hidden), torch.randn(hidden), torch.randn(5, hidden)
        on_dev = dev(resid.clone())
        rounded = M.norm_accumulate_round(dev(out), dev(w), 1e-5, on_dev, torch.bfloat16, 0.3)
        close(on_dev, resid.double() + 0.3 * plain.rms_norm(out.double(), w.double(), 1e-5), 2e-6)
        assert torch.equal(rounded, on_dev.to(torch.bfloat16))
    x = 40 * torch.randn(7, 333)
    close(F.soft_cap(dev(x.clone()), 12.0), plain.soft_cap(x.double(), 12.0), 1e-6)


# ------------------------------------------------------------------------------------------- whole models
LENGTHS = {"A": [1, 2, 5, 23, 64, 65, 131], "B": [3, 17, 48, 70, 1, 129], "C": [140, 2, 37, 66, 300]}


@pytest.fixture(scope="module", params=[(n, d) for n in ("A", "B", "C") for d in ("float32", "bfloat16")], ids=lambda p: f"{p[0]}-{p[1]}")
def setup(request, tmp_path_factory):
    from llm_runtime_study_b200.engine.runtime import load

    name, dtype = request.param
    config, seed, page = helpers.FUMOLORN[name]
    path, weights = helpers.make_fumolorn_dir(tmp_path_factory.mktemp(f"fumolorn{name}{dtype}"), config, seed, torch_dtype=dtype,
                                              ranks={0: 10, 2: 5} if name != "C" else None)
    rng = random.Random(seed + 1)
    requests = {f"r{i}": helpers.random_tokens(rng, config["vocab"], n) for i, n in enumerate(LENGTHS[name])}
    store = plain.round_bfloat16 if dtype == "bfloat16" else plain.keep
    expected = {rid: plain.forward(config, weights, tokens, store=store) for rid, tokens in requests.items()}
    loaded = load(path, device=DEV, dtype=dtype, strict_dtype=False)
    return dict(name=name, dtype=dtype, config=config, page=page, path=path, requests=requests, plain=expected, loaded=loaded, weights=weights)


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
    """One slot: the second request takes the first one's states, previous token and pages."""

    requests = {rid: tokens for rid, tokens in setup["requests"].items() if len(tokens) in (23, 17, 48, 65, 37, 66)}
    _compare(setup, _replay(setup, helpers.trace_chunked(requests, random.Random(3), sizes=(7, 16)), max_requests=1), requests)


def test_greedy_generation_through_the_engine(setup):
    """``Engine.generate`` with its scheduler (prompt portions, batching, graph decode) gives the plain model's greedy tokens."""

    from llm_runtime_study_b200.engine.engine import Engine
    from llm_runtime_study_b200.sampling import SamplingConfig

    if setup["dtype"] != "float32":
        pytest.skip("greedy ties are decided by rounding in bfloat16")
    config, weights = setup["config"], setup["weights"]
    prompts = [setup["requests"]["r3"][:19], setup["requests"]["r2"], setup["requests"]["r1"] + [3, 1, 4]]
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

    config = helpers.FUMOLORN_A
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
