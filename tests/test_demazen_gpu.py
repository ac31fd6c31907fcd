"""Demazen on the GPU against the plain implementation (tests/plain_demazen.py): the new kernels and options alone (position
vectors, capped logits, the router's bias, the join of two normed results, decays, exponential gates, the recurrence whole and in
chunks, the one-token kernel, attention with values of another size), one-layer models of both mixers and feed-forwards, keys made
to stand out at a window's and a page's edges and writes far back in a state, then whole models from small configurations with
random weights: prompts, token-by-token decoding, portions, batches of unequal requests, slots used again, long decoding, greedy
generation, trace replay."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from conftest import ROOT, close_enough, has_gpu
from demazen_configs import CONFIGS, _dense, _layer, _mem, _model, _moe, _par

pytestmark = [pytest.mark.gpu, pytest.mark.skipif(not has_gpu(), reason="needs a CUDA device")]
DEV = "cuda:0"


def _ops():
    from ultima_b200.kernels import ops
    return ops


def rel_err(got, ref):
    got, ref = got.double().cpu(), ref.double().cpu()
    return float((got - ref).abs().max() / max(1e-30, float(ref.abs().max())))


def _ids(seed, n, vocab, avoid=()):
    ids = np.random.default_rng(seed).integers(0, vocab, size=n).tolist()
    if avoid:
        free = [t for t in range(vocab) if t not in avoid]
        ids = [free[t % len(free)] for t in ids]
    return ids


def _all(n):
    return list(range(n))


def agree(got, ref, dtype, layers, what):
    """float32: every position within rounding.  bfloat16: the same bound for all but a few positions, since a router
    whose two candidates lie within rounding of each other may choose the other one there."""
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    if dtype == "float32":
        err, bound = close_enough(got, ref, dtype, layers)
        assert err <= bound, (what, err, bound)
        return
    assert got.shape == ref.shape and np.isfinite(got).all(), what
    _, bound = close_enough(got, ref, dtype, layers)
    rows = np.abs(got - ref).max(axis=-1)
    over = int((rows > bound).sum())
    assert over <= max(1, len(rows) // 25) and float(np.median(rows)) <= bound / 2, (what, over, len(rows), float(rows.max()), bound)


class _Step:
    """The fields of a step's batch that the kernels read."""

    def __init__(self, befores, news, slots=None):
        start = np.concatenate([[0], np.cumsum(news)]).astype(np.int32)
        self.seq_start = torch.tensor(start, device=DEV)
        self.seq_before = torch.tensor(befores, dtype=torch.int32, device=DEV)
        self.seq_slot = torch.tensor(slots if slots is not None else list(range(len(news))), dtype=torch.int32, device=DEV)
        self.n_seqs, self.max_new, self.max_after = len(news), max(news), max(b + n for b, n in zip(befores, news))
        self.start = start


# ---------------------------------------------------------------------------------------
# embedding, head, router, join
# ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [64, 37])
def test_the_position_vector_is_added_and_not_scaled(width, dtype):
    ops = _ops()
    g = torch.Generator().manual_seed(width)
    table, pos = torch.randn(11, width, generator=g).to(dtype), torch.randn(9, width, generator=g).to(dtype)
    ids, at = torch.tensor([3, 10, 0, 3], dtype=torch.int32), torch.tensor([0, 8, 4, 7], dtype=torch.int32)
    status, out = torch.zeros(1, dtype=torch.int32, device=DEV), torch.empty(4, width, device=DEV)
    ops.embed(table.to(DEV), ids.to(DEV), out, status, 2.5, pos_table=pos.to(DEV), positions=at.to(DEV))
    assert rel_err(out, table[ids.long()].double() * 2.5 + pos[at.long()].double()) < 1e-6 and int(status[0]) == 0
    ops.embed(table.to(DEV), ids.to(DEV), out, status, 1.0, pos_table=pos[:8].contiguous().to(DEV), positions=at.to(DEV))
    assert int(status[0]) == 1                                      # a position outside the table is flagged, its row zero
    assert float(out[1].abs().max()) == 0.0 and float(out[3].abs().max()) > 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,N,K", [(1, 300, 64), (5, 97, 50), (70, 512, 128), (600, 4096, 256)])
def test_capped_results_of_a_product(T, N, K, dtype):
    """Every token tile, the two-CTA product and the CUDA-core path; results far beyond the cap."""
    from ultima_b200.engine import Runtime
    import plain_demazen as P
    rt = Runtime(DEV, dtype)
    g = torch.Generator().manual_seed(T)
    a, w = torch.randn(T, K, generator=g).to(dtype), torch.randn(N, K, generator=g).to(dtype)
    for cap in (3.0, 40.0):
        out = torch.full((T, N), 7.0, device=DEV)
        rt.matmul(a.to(DEV), w.to(DEV), out, unary=_ops().UNARY_SOFTCAP, unary_arg=cap)
        assert rel_err(out, P.capped(a.double() @ w.double().T, cap)) < 2e-5
    rt.check_status()


@pytest.mark.parametrize("ne,top", [(6, 2), (33, 5), (4, 4), (7, 1)])
def test_the_routers_bias_counts_for_the_choice_and_the_weights(ne, top):
    import plain_demazen as P
    ops = _ops()
    T = 50
    g = torch.Generator().manual_seed(ne)
    z, bias = torch.randn(T, ne, generator=g) * 2, torch.randn(ne, generator=g) * 2
    ref_idx, ref_w = P.route(z.double() + bias.double(), top)
    assert top == ne or not torch.equal(P.route(z, top)[0], ref_idx)
    mode = ops.ROUTE_LOGITS | ops.ROUTE_LOGIT_BIAS
    coarse = (z * 4).round() / 4
    for zs in (z, torch.stack([coarse, z - coarse, torch.zeros_like(z)])):
        for small in (False, True):
            n = min(T, ops.ROUTE_SMALL_TOKENS) if small else T
            zd = (zs[:n] if zs.dim() == 2 else zs[:, :n]).contiguous().to(DEV)
            idx, wts = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV)
            if small:
                ws = [torch.zeros(k, dtype=torch.int32, device=DEV) for k in (4 * (n * top + ne), 1, n * top, n * top)]
                ops.route_small(zd, bias.to(DEV), ne, top, 1, 1, idx, wts, ws[0].view(-1, 4), ws[1], ws[2].view(n, top), ws[3], 16, mode=mode)
            else:
                counts = torch.zeros(ne, dtype=torch.int32, device=DEV)
                ops.route(zd, bias.to(DEV), ne, top, 1, 1, idx, wts, counts, mode=mode)
                assert counts.cpu().tolist() == torch.bincount(ref_idx.flatten(), minlength=ne).tolist()
            assert torch.equal(idx.cpu().long(), ref_idx[:n]) and float((wts.cpu().double() - ref_w[:n]).abs().max()) < 3e-6


@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,width", [(1, 48), (37, 101), (5, 258), (3, 1024), (9, 2048), (2, 4100), (2, 8200)])
def test_the_join_of_two_normed_results(T, width, out_dtype):
    """Widths on the kernel with rows in registers and on the other; with and without the norm of the sum."""
    import plain_demazen as P
    ops = _ops()
    g = torch.Generator().manual_seed(T * 7 + width)
    x, y, y2 = torch.randn(T, width, generator=g) * 3, torch.randn(T, width, generator=g) * 0.02, torch.randn(T, width, generator=g) * 50
    w, w2, aw = (1 + 0.3 * torch.randn(width, generator=g) for _ in range(3))
    for scales in ((0.5, 0.5), (1.3, -0.4)):
        z = scales[0] * P.rms_norm(y.double(), w.double(), 1e-3) + scales[1] * P.rms_norm(y2.double(), w2.double(), 1e-3)
        for after, new in (((aw.to(DEV), 1e-2), x.double() + P.rms_norm(z, aw.double(), 1e-2)), (None, x.double() + z)):
            for with_out in (True, False):
                xd, yd, y2d = x.to(DEV), y.to(DEV), y2.to(DEV)
                o = torch.empty(T, width, dtype=out_dtype, device=DEV) if with_out else None
                ops.norm_join_two(yd, y2d, xd, (w.to(DEV), w2.to(DEV)), scales, 1e-3, after=after, out=o)
                assert rel_err(xd, new) < 1e-6 and float(yd.abs().max()) == 0.0 and float(y2d.abs().max()) == 0.0
                assert o is None or rel_err(o, new) < (1e-6 if out_dtype == torch.float32 else 2 ** -7)


# ---------------------------------------------------------------------------------------
# the recurrences
# ---------------------------------------------------------------------------------------
def _projection(T, H, D, E, extra, seed, parts=1, pad=0):
    """Rows [q | k | v | gate | extra ... | pad] and where they start; with ``parts`` the rows in slices that add up to them.
    Queries share a part of the keys (see ``_sharpen``)."""
    g = torch.Generator().manual_seed(seed)
    offs, at = [], 0
    for n in (H * D, H * D, H * E, H * E) + tuple(extra):
        offs.append(at)
        at += n
    p = torch.randn(T, at + pad, generator=g)
    p[:, :H * D] = 0.6 * p[:, :H * D] + p[:, offs[1]:offs[1] + H * D]
    if parts == 1:
        return p, p.to(DEV), offs
    slices = [torch.randn(T, at + pad, generator=g) for _ in range(parts - 1)]
    rest = p - sum(slices)
    return sum(slices) + rest, torch.stack(slices + [rest]).to(DEV), offs


def _cols(p, offs, which, H, n):
    return p[:, offs[which]:offs[which] + H * n].view(p.shape[0], H, n).double()


@pytest.mark.parametrize("T,H,D,rank,tau", [(1, 1, 8, 1, 16.0), (19, 3, 24, 5, 4.0), (130, 5, 40, 64, 1.0), (9, 2, 200, 300, 0.5)])
def test_decays_of_every_channel(T, H, D, rank, tau):
    import plain_demazen as P
    ops = _ops()
    E = 4
    for parts in (1, 3):
        p, pd, offs = _projection(T, H, D, E, (rank,), T + rank, parts)
        g = torch.Generator().manual_seed(rank)
        up, bias = torch.randn(rank, H * D, generator=g) / rank ** 0.5, torch.randn(H * D, generator=g) * 6
        form = ops.LinForm(H, D, E, offs + [0], rank=rank)
        dec = torch.empty(T, H * D, device=DEV)
        ops.lin_decay(pd, form, up.to(DEV), bias.to(DEV), dec, tau)
        z = p[:, offs[4]:offs[4] + rank].double() @ up.double() + bias.double()
        assert float((dec.cpu().double() - torch.exp(P.log_sigmoid(z) / tau)).abs().max()) < 2e-6 / min(tau, 1.0)


def test_exponential_gates_with_their_running_maximum():
    """Sequences of one token, of several rounds of the scan's block and of lengths that end inside a warp, in several calls that
    go on from the state; gates of all kinds: large input gates far apart, input gates so small that the maximum stays near its
    start at 0, forget gates that hold and that forget at once."""
    import plain_demazen as P
    ops = _ops()
    H, D, E, cap = 3, 4, 4, 8.0
    lens = [1, 31, 33, 1100, 512]
    shift_i, shift_f = torch.tensor([-7.0, 0.0, 4.0]), torch.tensor([30.0, 2.0, -6.0])
    g = torch.Generator().manual_seed(3)
    rows = [torch.randn(n, 2 * H, generator=g) * 5 for n in lens]
    m_ref = []
    for r in rows:
        eye = torch.eye(H, dtype=torch.float64)
        i, f = P.mlstm_gates(r.double(), {"i": torch.cat([eye, 0 * eye], 1), "f": torch.cat([0 * eye, eye], 1), "i.b": shift_i.double(),
                                          "f.b": shift_f.double()}, cap, "")
        m, out = torch.zeros(H, dtype=torch.float64), []
        for t in range(len(r)):
            new = torch.maximum(f[t] + m, i[t])
            out.append(torch.stack([torch.exp(f[t] + m - new), torch.exp(i[t] - new), torch.exp(-new)]))
            m = new
        m_ref.append((torch.stack(out), m))
    form = ops.LinForm(H, D, E, (0, 0, 0, 0, 0, H), head_form=True)
    state = torch.zeros(9, H, device=DEV)
    slots = [4, 0, 7, 2, 8]
    got = [[] for _ in lens]
    done = [0] * len(lens)
    for share in (0.3, 0.6, 1.0):
        news = [max(0, int(n * share) - d) if share < 1 else n - d for n, d in zip(lens, done)]
        live = [s for s in range(len(lens)) if news[s] > 0]
        x = torch.cat([rows[s][done[s]:done[s] + news[s]] for s in live])
        x = torch.cat([x, torch.zeros(len(x), 12 - 2 * H)], dim=1).contiguous().to(DEV)      # (rows as wide as the form's columns)
        form.cols = 12
        b = _Step([done[s] for s in live], [news[s] for s in live], [slots[s] for s in live])
        keep, put, floor = (torch.empty(len(x), H, device=DEV) for _ in range(3))
        ops.lin_gates(x, form, shift_i.to(DEV), shift_f.to(DEV), cap, state, b, keep, put, floor)
        for j, s in enumerate(live):
            lo, hi = int(b.start[j]), int(b.start[j + 1])
            got[s].append(torch.stack([keep[lo:hi], put[lo:hi], floor[lo:hi]], dim=1).cpu().double())
            done[s] += news[s]
    assert done == lens
    for s, n in enumerate(lens):
        out = torch.cat(got[s])
        # a gate is exp of differences of numbers below the cap: absolute errors of a few 1e-6, times the gate's own size
        assert float(((out - m_ref[s][0]).abs() / (1e-3 + m_ref[s][0].abs())).max()) < 2e-4, s
        assert float((state[slots[s]].cpu().double() - m_ref[s][1]).abs().max()) < 2e-5
    untouched = [i for i in range(9) if i not in slots]
    assert float(state[untouched].abs().max()) == 0.0


SCAN_SIZES = [(2, 8, 12), (3, 24, 40), (1, 64, 64), (2, 64, 128), (2, 128, 60), (1, 200, 33), (1, 256, 72), (3, 7, 5), (2, 30, 65), (2, 48, 256)]


def _scan_case(head_form, H, D, E, news, chunks, seed, slow=False):
    """Outputs and states of the scan kernels against the plain recurrence, from states that are not zero."""
    import plain_demazen as P
    ops = _ops()
    T = sum(news)
    extra = (H, H) if head_form else (6,)
    p, pd, offs = _projection(T, H, D, E, extra, seed, pad=(-(2 * H * D + 2 * H * E + sum(extra))) % 4)
    form = ops.LinForm(H, D, E, (offs + [0])[:6], rank=0 if head_form else 6, head_form=head_form)
    g = torch.Generator().manual_seed(seed + 1)
    n_slots = len(news) + 2
    slots = torch.randperm(n_slots, generator=g)[:len(news)].tolist()
    S0 = torch.randn(n_slots, H, D, E, generator=g)
    n0 = torch.randn(n_slots, H, D, generator=g)
    S, n = S0.to(DEV), n0.to(DEV)
    rate = 0.002 if slow else 0.4
    if head_form:
        dec, put = torch.exp(-torch.rand(T, H, generator=g) * rate), torch.rand(T, H, generator=g)
    else:
        dec, put = torch.exp(-torch.rand(T, H, D, generator=g) * rate), None
    ew = E + 1 if head_form else E
    b = _Step([0] * len(news), news, slots)
    out = torch.full((T, H, ew), float("nan"), device=DEV)
    work = torch.full((chunks[0], len(news), H, D, ew), float("nan"), device=DEV) if chunks[0] > 1 else None
    decay = torch.full((chunks[0], len(news), H, 1 if head_form else D), float("nan"), device=DEV) if chunks[0] > 1 else None
    ops.lin_scan(pd, form, dec.to(DEV).contiguous(), put.to(DEV) if head_form else None, out, S, n if head_form else None, b, work, decay,
                 chunks)
    torch.cuda.synchronize()
    q, k, v = (_cols(p, offs, i, H, m) for i, m in ((0, D), (1, D), (2, E)))
    for s, (lo, hi) in enumerate(zip(b.start[:-1], b.start[1:])):
        Sr, nr = S0[slots[s]].double(), n0[slots[s]].double()
        ref, refn = [], []
        for t in range(lo, hi):
            a = dec[t].double()[:, None] if head_form else dec[t].double()
            w = put[t].double()[:, None] * k[t] if head_form else k[t]
            Sr = a[:, :, None] * Sr + w[:, :, None] * v[t][:, None, :]
            nr = a * nr + w
            ref.append(torch.einsum("hde,hd->he", Sr, q[t]))
            refn.append((nr * q[t]).sum(-1))
        if hi > lo:
            assert rel_err(out[lo:hi, :, :E], torch.stack(ref)) < 5e-6, (H, D, E, chunks, s)
            if head_form:
                assert rel_err(out[lo:hi, :, E], torch.stack(refn)) < 5e-6
        assert rel_err(S[slots[s]], Sr) < 5e-6, (H, D, E, chunks, s, "state")
        if head_form:
            assert rel_err(n[slots[s]], nr) < 5e-6
    idle = [i for i in range(n_slots) if i not in slots]
    assert torch.equal(S[idle].cpu(), S0[idle])
    # the plain functions from a zero state agree with the loop above
    if not head_form:
        assert torch.allclose(P.decayed_memory(q[:3], k[:3], v[:3], dec[:3].double())[0], torch.einsum("hd,hd,he->he", q[0], k[0], v[0]))


@pytest.mark.parametrize("head_form", [False, True])
@pytest.mark.parametrize("H,D,E", SCAN_SIZES)
def test_the_recurrence_whole_and_in_chunks(H, D, E, head_form):
    """Every number of channels a lane holds, one and several blocks of columns, sizes in fours and odd ones; unequal sequences
    whose last chunk is full, short, of one token, and sequences shorter than a chunk; states that hold on and that fade."""
    news = [37, 2, 80, 17]
    for chunks in ((1, 80), (5, 16), (2, 40), (10, 8), (80, 1)):
        _scan_case(head_form, H, D, E, news, chunks, seed=D + E + chunks[0], slow=chunks[0] % 2 == 0)


def test_the_recurrence_over_a_long_sequence_keeps_far_writes():
    for head_form in (False, True):
        _scan_case(head_form, 2, 32, 48, [1500], (23, 66), seed=9, slow=True)
        _scan_case(head_form, 1, 64, 16, [700, 1], (1, 700), seed=10, slow=True)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,E", SCAN_SIZES + [(1, 16, 520), (2, 4, 1024)])
def test_one_token_a_sequence_in_one_kernel(H, D, E, dtype):
    """Both forms, the projection whole and in slices, a norm weight a head and one for all, both output gates, several tokens in
    a row from the states the kernel left."""
    import plain_demazen as P
    ops = _ops()
    B, tol = 5, 2e-5 if dtype == torch.float32 else 2 ** -7
    g = torch.Generator().manual_seed(D * E)
    slots = [3, 0, 6, 1, 5]
    step = _Step([0] * B, [1] * B, slots)
    scale, eps = D ** -0.5, 1e-4
    # exponential gates
    S, n, m = torch.zeros(7, H, D, E, device=DEV), torch.zeros(7, H, D, device=DEV), torch.zeros(7, H, device=DEV)
    bi, bf = torch.randn(H, generator=g), torch.randn(H, generator=g) * 2
    w = 1 + 0.3 * torch.randn(H * E, generator=g)
    seen = []
    for t in range(4):
        p, pd, offs = _projection(B, H, D, E, (H, H), 10 * t + D, parts=1 + t % 3, pad=3)
        form = ops.LinForm(H, D, E, offs, head_form=True)
        out = torch.full((B, H * E), float("nan"), dtype=dtype, device=DEV)
        ops.lin_step(pd, form, (S, n, m), step, w.to(DEV), out, scale, eps, out_scale=1.5, gates=(bi.to(DEV), bf.to(DEV), 5.0))
        seen.append(p.double())
        q, k, v = (torch.stack([_cols(x, offs, i, H, sz) for x in seen]) for i, sz in ((0, D), (1, D), (2, E)))
        for b in range(B):
            x = torch.stack([r[b] for r in seen])
            eye = torch.eye(H, dtype=torch.float64)
            i, f = P.mlstm_gates(x[:, offs[4]:offs[4] + 2 * H], {"i": torch.cat([eye, 0 * eye], 1), "f": torch.cat([0 * eye, eye], 1),
                                                                  "i.b": bi.double(), "f.b": bf.double()}, 5.0, "")
            o = P.mlstm_memory(q[:, b] * scale, k[:, b], v[:, b], i, f)[-1]
            o = P.over_rms(o, eps).reshape(-1) * w.double() * torch.sigmoid(x[-1, offs[3]:offs[3] + H * E]) * 1.5
            assert rel_err(out[b], o) < tol, (H, D, E, t, b)
    assert float(S[[2, 4]].abs().max()) == 0.0
    # decays a channel
    rank, tau = 5, 3.0
    S = torch.zeros(7, H, D, E, device=DEV)
    up, bias = torch.randn(rank, H * D, generator=g) * 0.5, torch.randn(H * D, generator=g)
    w = 1 + 0.3 * torch.randn(E, generator=g)
    seen = []
    for t in range(4):
        p, pd, offs = _projection(B, H, D, E, (rank,), 10 * t + E, parts=1 + t % 3, pad=1)
        form = ops.LinForm(H, D, E, offs + [0], rank=rank)
        out = torch.full((B, H * E), float("nan"), dtype=dtype, device=DEV)
        ops.lin_step(pd, form, (S,), step, w.to(DEV), out, scale, eps, silu_gate=True, decay=(up.to(DEV), bias.to(DEV), tau))
        seen.append(p.double())
        q, k, v = (torch.stack([_cols(x, offs, i, H, sz) for x in seen]) for i, sz in ((0, D), (1, D), (2, E)))
        for b in range(B):
            x = torch.stack([r[b] for r in seen])
            a = torch.exp(P.log_sigmoid(x[:, offs[4]:offs[4] + rank] @ up.double() + bias.double()) / tau).view(-1, H, D)
            o = P.rms_norm(P.decayed_memory(q[:, b] * scale, k[:, b], v[:, b], a)[-1], w.double(), eps).reshape(-1)
            o = o * P.silu(x[-1, offs[3]:offs[3] + H * E])
            assert rel_err(out[b], o) < tol, (H, D, E, t, b, "channel")


# ---------------------------------------------------------------------------------------
# attention with values of another size
# ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,hd,hdv", [(4, 2, 32, 48), (3, 1, 20, 28), (2, 2, 64, 128), (16, 4, 64, 128), (32, 8, 128, 128), (3, 3, 10, 14), (5, 5, 9, 4)])
def test_placement_with_a_norm_over_all_heads(nh, nkv, hd, hdv, dtype):
    """Sizes in fours (rows in registers, of every length the kernel is built for) and others; the projection whole, in slices, and
    as columns of wider rows; two sequences on a ring that wraps."""
    import plain_demazen as P
    ops = _ops()
    qn, kn, vn, T, eps = nh * hd, nkv * hd, nkv * hdv, 70, 1e-3
    g = torch.Generator().manual_seed(qn)
    qw, kw = 1 + 0.2 * torch.randn(qn, generator=g), 1 + 0.2 * torch.randn(kn, generator=g)
    pos = torch.cat([torch.arange(40) + 100, torch.arange(30)]).to(torch.int32)
    seq = torch.tensor([0] * 40 + [1] * 30, dtype=torch.int32)
    table = torch.tensor([[4, 1], [0, 3]], dtype=torch.int32)
    for parts, pad in ((1, 0), (3, 0), (1, 8), (2, 4)):
        xs = torch.randn(parts, T, qn + kn + vn + pad, generator=g)
        x = xs.sum(0).double()
        dev = xs.to(DEV)[..., :qn + kn + vn]
        q = torch.full((T, qn), float("nan"), dtype=dtype, device=DEV)
        kc = torch.full((5, nkv, 64, hd), 9.0, dtype=dtype, device=DEV)
        vc = torch.full((5, nkv, 64, hdv), 9.0, dtype=dtype, device=DEV)
        ops.qkv_place_rows(dev if parts > 1 else dev[0], 0, qn, qn + kn, q, qw.to(DEV), kw.to(DEV), True, None, None, 0, False, pos.to(DEV),
                           seq.to(DEV), kc, vc, table.to(DEV), 128, 64, nh, nkv, hd, hdv, eps)
        tol = 3e-6 if dtype == torch.float32 else 2 ** -7
        assert rel_err(q, P.rms_norm(x[:, :qn], qw.double(), eps)) < tol
        k = P.rms_norm(x[:, qn:qn + kn], kw.double(), eps).view(T, nkv, hd)
        v = x[:, qn + kn:qn + kn + vn].reshape(T, nkv, hdv)
        page = table[seq.long(), (pos.long() % 128) // 64].long()
        assert rel_err(kc.cpu()[page, :, pos.long() % 64], k) < tol and rel_err(vc.cpu()[page, :, pos.long() % 64], v) < tol
        used = torch.zeros(5, 64, dtype=torch.bool)
        used[page, pos.long() % 64] = True
        assert bool((kc.cpu().permute(0, 2, 1, 3)[~used] == 9.0).all()) and bool((vc.cpu().permute(0, 2, 1, 3)[~used] == 9.0).all())


class _KV:
    def __init__(self, k, v, table, ring, window):
        self.k, self.v, self.table, self.ring, self.page, self.window, self.owner = k, v, table, ring, 64, window, True


def _attention_case(nh, nkv, hd, hdv, befores, news, window, seed, slices=None, ring_pages=None, kernel=None):
    from ultima_b200.engine import Runtime
    from ultima_b200.kernels import attn_tc
    rt = Runtime(DEV, torch.bfloat16)
    g = torch.Generator().manual_seed(seed)
    lens = [b + n for b, n in zip(befores, news)]
    pages = ring_pages or max(-(-n // 64) for n in lens)
    n_pages = len(lens) * pages + 3
    perm = torch.randperm(n_pages, generator=g)[:len(lens) * pages].view(len(lens), pages).to(torch.int32)
    kc = torch.full((n_pages, nkv, 64, hd), float("nan"), dtype=torch.bfloat16)      # unwritten rows must reach no result
    vc = torch.full((n_pages, nkv, 64, hdv), float("nan"), dtype=torch.bfloat16)
    dense = []
    for s, n in enumerate(lens):
        k, v = torch.randn(n, nkv, hd, generator=g).to(torch.bfloat16), torch.randn(n, nkv, hdv, generator=g).to(torch.bfloat16)
        for p in range(max(0, n - pages * 64), n):
            kc[perm[s, (p // 64) % pages], :, p % 64] = k[p]
            vc[perm[s, (p // 64) % pages], :, p % 64] = v[p]
        dense.append((k.double(), v.double()))
    T = sum(news)
    q = torch.randn(T, nh * hd, generator=g).to(torch.bfloat16).to(DEV)
    b = _Step(befores, news)
    out = torch.full((T, nh * hdv), float("nan"), dtype=torch.bfloat16, device=DEV)
    scale = hd ** -0.5
    attn_tc.attention(q, _KV(kc.to(DEV), vc.to(DEV), perm.to(DEV), pages * 64, window), out, b, nh, nkv, hd, scale, rt, slices=slices,
                      kernel=kernel)
    torch.cuda.synchronize()
    rt.check_status()
    assert torch.isfinite(out).all()
    worst, qd, od = 0.0, q.double().cpu().view(T, nh, hd), out.double().cpu().view(T, nh, hdv)
    for s, (bf, n) in enumerate(zip(befores, news)):
        for t in range(n):
            pos = bf + t
            lo = max(0, pos - window + 1) if window else 0
            k, v = (x[lo:pos + 1].repeat_interleave(nh // nkv, dim=1) for x in dense[s])
            p = torch.softmax(torch.einsum("hd,jhd->hj", qd[b.start[s] + t], k) * scale, dim=-1)
            worst = max(worst, rel_err(od[b.start[s] + t], torch.einsum("hj,jhe->he", p, v)))
    return worst


TWO_SIZES = [(4, 2, 64, 128), (6, 3, 32, 48), (3, 3, 96, 16), (2, 1, 128, 256), (8, 2, 16, 32), (16, 2, 48, 112), (4, 4, 256, 64), (5, 1, 128, 64),
             (6, 2, 96, 192), (2, 2, 112, 96), (3, 1, 208, 224)]


@pytest.mark.parametrize("kernel", [None, "mma", "wide"])
@pytest.mark.parametrize("nh,nkv,hd,hdv", TWO_SIZES)
def test_attention_of_prompts_with_values_of_another_size(nh, nkv, hd, hdv, kernel):
    """On tcgen05 where the sizes fit (128 rows a CTA, and 256 where the values do), and on mma.sync; rows that end inside a block
    of 64 columns, heads that do and do not divide 128, continued prompts, a ring that has wrapped."""
    from ultima_b200.kernels import attn_tc
    if kernel == "wide" and (not attn_tc.tc_sizes_fit(hd, hdv) or hdv > 128):
        pytest.skip("not a size of that kernel")
    held = attn_tc.WIDE
    attn_tc.set_wide(2 if kernel == "wide" else 0)
    try:
        k = None if kernel == "wide" else kernel
        for window in (None, 40, 1, 100):
            err = _attention_case(nh, nkv, hd, hdv, [0, 0, 0, 70], [1, 17, 130, 65], window, seed=hd + hdv, kernel=k)
            assert err <= 2 ** -6, (window, err)
        err = _attention_case(nh, nkv, hd, hdv, [0, 200], [300, 70], 150, seed=hd, ring_pages=6, kernel=k)
        assert err <= 2 ** -6, err
    finally:
        attn_tc.set_wide(held)


@pytest.mark.parametrize("nh,nkv,hd,hdv", TWO_SIZES)
@pytest.mark.parametrize("slices", [None, 1, 3])
def test_attention_of_single_tokens_with_values_of_another_size(nh, nkv, hd, hdv, slices):
    for window in (None, 40, 64, 1, 129):
        err = _attention_case(nh, nkv, hd, hdv, [0, 63, 64, 300, 127], [1] * 5, window, seed=hd + 3, slices=slices)
        assert err <= 2 ** -6, (window, err)
    err = _attention_case(nh, nkv, hd, hdv, [500, 129], [1, 1], 100, seed=hd, ring_pages=3, slices=slices)
    assert err <= 2 ** -6, err


# ---------------------------------------------------------------------------------------
# models of one layer
# ---------------------------------------------------------------------------------------
_SMALL = _mem(2, 16, 8, 6.0)
ONE_LAYER = {
    "memory": _model([_layer(_mem(3, 24, 40, 5.0))], width=56, cap=9.0),
    "memory_one_head_wide": _model([_layer(_mem(1, 128, 200, 12.0))], cap=30.0),
    "memory_no_fours": _model([_layer(_mem(5, 9, 7, 3.0))], width=50, eps=1e-3),
    "parallel": _model([_layer(_par((4, 2, 32, 64, 0.2, 50), (2, 48, 32, 8.0, 16)))], width=72),
    "parallel_equal_sizes": _model([_layer(_par((4, 4, 64, 64, 0.12, 64), (4, 32, 32, 16.0, 32)))], width=64),
    "parallel_window_of_one": _model([_layer(_par((2, 1, 48, 32, 0.3, 1), (1, 64, 96, 2.0, 7)))], eps=1e-3),
    "parallel_no_fours": _model([_layer(_par((3, 1, 10, 14, 0.3, 30), (3, 11, 13, 1.0, 5)))], width=50),
    "parallel_large_heads": _model([_layer(_par((2, 1, 160, 320, 0.08, 45), (1, 128, 288, 4.0, 24)))], width=72),
    "routed": _model([_layer(_SMALL, _moe(10, 3, 24))], width=72),
    "routed_all_chosen": _model([_layer(_SMALL, _moe(3, 3, 128))], width=48),
    "routed_no_eights": _model([_layer(_SMALL, _moe(6, 1, 21))], width=50),
    "dense": _model([_layer(_SMALL, _dense(80))], width=64),
}


def _sharpen(W, amp=1.7):
    """Random weights scaled so that scores, gates and decays are far from uniform, the positions count, the router's bias moves
    choices and the logits meet their cap.  The recurrent mixers' queries share a part of their keys' matrix: what is read is
    normed, and a read-out near zero (a query across every key) would turn rounding into errors of any size."""
    out = {}
    for n, t in W.items():
        if n.endswith(".mix.q") or n.endswith(".mix.right.q"):
            t = 0.35 * t + W[n[:-1] + "k"]
        leaf = n.split(".")[-1]
        if ".mix." in n and t.dim() == 2 and leaf in ("q", "k", "g"):
            t = t * amp
        if leaf in ("i", "f"):                                  # (one token that outweighs all others is such a case too)
            t = t * 0.5
        if ".mix." in n and leaf in ("q", "k", "v", "o", "g") and t.dim() == 2:
            t = t * 6                                           # (drawn with a deviation of 0.02; widths here are small)
        if leaf == "a1":
            t = t * 20
        if ".mlp." in n and leaf in ("gate", "up", "down"):
            t = t * 6
        if n in ("embed", "pos"):
            t = t * (40 if n == "embed" else 15)
        out[n] = t.to(torch.bfloat16)
    return out


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    import plain_demazen as P
    import ultima_b200 as u
    from ultima_b200.weights.safetensors_io import write_safetensors
    base = tmp_path_factory.mktemp("demazen")
    made = {}

    def get(name, raw=None, change=None):
        if name not in made:
            d = str(base / name.replace("/", "_"))
            plain_name = name.split("/")[0]
            raw = copy.deepcopy(raw or CONFIGS.get(plain_name) or ONE_LAYER[plain_name])
            if name.endswith("/all_chosen"):
                for L in raw["layers"]:
                    if L.get("mlp") and L["mlp"]["kind"] == "moe":
                        L["mlp"]["router"]["top"] = L["mlp"]["router"]["experts"]
            u.write_random_model(d, u.config_from_dict(raw), seed=len(plain_name), dtype="bfloat16")
            cfg, W = P.read_folder(d)
            W = _sharpen(W)
            if change is not None:
                W = {n: t.to(torch.bfloat16) for n, t in change(cfg, {n: t.double() for n, t in W.items()}).items()}
            write_safetensors(os.path.join(d, "model.safetensors"), W)
            made[name] = (d,) + P.read_folder(d)
        return made[name]
    return get


_engines = {}


def _engine(folder, dtype, **kw):
    from ultima_b200.engine import Engine
    key = (folder, dtype, tuple(sorted(kw.items())))
    if key not in _engines:
        _engines[key] = Engine.from_dir(folder, dtype=dtype, with_sampler=False, **{"max_tokens": 2048, "max_seqs": 6, **kw})
    return _engines[key]


def _for(name, dtype):
    """The model's folder for a run in ``dtype``.  In bfloat16 a router's near tie between two outputs may go either way, and
    one other choice reaches every later position through keys and states; so the bfloat16 runs of whole models use the same
    models with routers that choose every output (the weights still differ from token to token).  The choice itself is held to
    the plain implementation by the 32-bit runs of the same models, by the one-layer models in both types and by the router's
    own test."""
    return name + "/all_chosen" if dtype == "bfloat16" else name


def _whole(eng, ids, want=None):
    s = eng.open(1)
    got = eng.step(s, [ids], [want if want is not None else _all(len(ids))]).cpu().numpy()
    eng.close(s)
    eng.check_errors()
    return got


def _prompt_then_single_tokens(eng, ids, cut, want_from=0):
    s = eng.open(1)
    rows = [eng.step(s, [ids[:cut]], [list(range(want_from, cut))]).cpu().numpy()]
    for t in range(cut, len(ids)):
        rows.append(eng.step(s, [[ids[t]]]).cpu().numpy())
    eng.close(s)
    eng.check_errors()
    return np.concatenate(rows)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ONE_LAYER))
def test_one_layer_alone_in_a_prompt_and_token_by_token(folders, name, dtype):
    import plain_demazen as P
    d, cfg, W = folders(name)
    eng = _engine(d, dtype, poison_cache=True)
    ids = _ids(len(name), 140, cfg["vocab"])
    layers, taps = [], []
    with torch.no_grad():
        ref = P.forward(cfg, W, ids, torch.float64, layers).numpy()
    eng.model.tap = lambda i, x: taps.append(x.detach().double().cpu())
    got = _whole(eng, ids)
    eng.model.tap = None
    assert len(taps) == len(layers) == 1
    if dtype == "float32":
        assert rel_err(taps[0], layers[0]) < 2e-5, name
    agree(got, ref, dtype, 2, (name, "prompt"))
    agree(_prompt_then_single_tokens(eng, ids, 3), ref, dtype, 2, (name, "single tokens"))


def test_every_mechanism_shows_in_these_models(folders):
    """A test that could not fail would prove little: leaving a mechanism out of the plain implementation moves the logits of
    the one-layer models by far more than the bounds above."""
    import plain_demazen as P

    def moved(name, change):
        _, cfg, W = folders(name)
        ids = _ids(1, 60, cfg["vocab"])
        cfg2, W2 = copy.deepcopy(cfg), dict(W)
        change(cfg2, W2)
        a, b = P.logits(cfg, W, ids), P.logits(cfg2, W2, ids)
        return float(np.abs(a - b).max() / np.abs(a).max())

    def setw(name, f):
        return lambda c, W: W.__setitem__(name, f(W[name]))

    def mixer(*path, **new):
        def change(c, W):
            m = c["layers"][0]["mixer"]
            for k in path:
                m = m[k]
            m.update(new)
        return change
    zero, one = torch.zeros_like, torch.ones_like
    cases = [("memory", setw("pos", zero)), ("memory", lambda c, W: c.update(logit_softcap=30.0)), ("memory", mixer(gate_cap=1.0)),
             ("memory", setw("l0.mix.i.b", lambda t: t + 20)), ("memory", setw("l0.mix.f.b", lambda t: t - 4)), ("memory", setw("l0.mix.i", zero)),
             ("memory", setw("l0.mix.g", zero)), ("memory", setw("l0.mix.norm", one)), ("memory", setw("l0.norm1", one)),
             ("parallel", mixer("left", "mask", size=20)), ("parallel", mixer("left", scale=0.1)),
             ("parallel", setw("l0.mix.left.q.norm", one)), ("parallel", setw("l0.mix.right.a2.b", lambda t: t - 4)),
             ("parallel", setw("l0.mix.right.a2", zero)), ("parallel", mixer("right", tau=1.0)), ("parallel", setw("l0.mix.right.g", zero)),
             ("parallel", setw("l0.mix.right.norm", one)), ("parallel", setw("l0.mix.left.out", zero)),
             ("parallel", setw("l0.mix.right.out", zero)), ("routed", setw("l0.mlp.router.b", lambda t: t * 0)),
             ("routed", setw("l0.mlp.router", zero)), ("routed", setw("l0.norm2", one)), ("dense", setw("l0.mlp.gate", zero))]
    for i, (name, change) in enumerate(cases):
        m = moved(name, change)
        assert m > 0.01, (i, name, m)


# ---------------------------------------------------------------------------------------
# one key made to stand out: at a window's and a page's edges, and far back in a state
# ---------------------------------------------------------------------------------------
ASKER, MARKED = 5, 11


def _turn(W, pre, heads, kv_heads):
    """The queries of token ASKER are turned towards the keys of token MARKED (a rank-one change of W_q), and MARKED's values are
    made large."""
    a, e = W["embed"][ASKER], W["embed"][MARKED]
    k = (W[pre + "k"] @ e).view(kv_heads, -1).repeat_interleave(heads // kv_heads, dim=0).reshape(-1)
    W[pre + "q"] = 0.25 * W[pre + "q"] + torch.outer(k * 3.5, a / (a @ a))
    v = W[pre + "v"]
    W[pre + "v"] = v + torch.outer(torch.ones(v.shape[0], dtype=torch.float64) * 3.5, e / (e @ e))


def _marked_window(cfg, W):
    """Only the windowed side counts: the other side's result is multiplied by a weight of zeros."""
    m = cfg["layers"][0]["mixer"]["left"]
    W["pos"] = W["pos"] * 0.02
    _turn(W, "l0.mix.left.", m["heads"], m["kv_heads"])
    W["l0.mix.right.out"] = W["l0.mix.right.out"] * 0
    return W


MARKED_WINDOWS = {
    "marked_window_37": _model([_layer(_par((4, 2, 32, 48, 0.6, 37), (1, 16, 16, 4.0, 4)))]),
    "marked_window_64": _model([_layer(_par((2, 1, 64, 128, 0.4, 64), (1, 16, 16, 4.0, 4)))]),
    "marked_window_100_equal": _model([_layer(_par((4, 2, 64, 64, 0.4, 100), (2, 16, 16, 4.0, 4)))]),
    "marked_window_129_no_sixteens": _model([_layer(_par((3, 3, 20, 28, 0.7, 129), (1, 16, 16, 4.0, 4)))], width=52),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MARKED_WINDOWS))
def test_a_key_just_inside_and_just_outside_the_window(folders, name, dtype):
    import plain_demazen as P
    d, cfg, W = folders(name, MARKED_WINDOWS[name], _marked_window)
    size = cfg["layers"][0]["mixer"]["left"]["mask"]["size"]
    eng = _engine(d, dtype, poison_cache=True)
    wider, narrower = copy.deepcopy(cfg), copy.deepcopy(cfg)
    wider["layers"][0]["mixer"]["left"]["mask"]["size"] = size + 1
    narrower["layers"][0]["mixer"]["left"]["mask"]["size"] = size - 1
    for m in (0, 1, 27, 63, 64, 127, 128, 200):
        for inside in (True, False):
            p = m + size - 1 + (0 if inside else 1)
            ids = _ids(m * 100 + p, p + 1, cfg["vocab"], avoid=(ASKER, MARKED))
            ids[m], ids[p] = MARKED, ASKER
            ref = P.logits(cfg, W, ids)[p]
            bound = close_enough(ref[None], ref[None], dtype, 2)[1]
            # a window that is one off would show
            moved = float(np.abs(P.logits(narrower if inside else wider, W, ids)[p] - ref).max())
            assert moved > 3 * bound, (name, m, p, inside, moved, bound)
            err = float(np.abs(_whole(eng, ids, [p])[0] - ref).max())
            assert err <= bound, (name, dtype, m, p, "prompt", err, bound)
            cut = max(1, p - 3)                                     # and decoded alone, three tokens behind the prompt
            got = _prompt_then_single_tokens(eng, ids, cut, want_from=cut - 1)[-1]
            err = float(np.abs(got - ref).max())
            assert err <= bound, (name, dtype, m, p, "decoded", err, bound)


def _marked_state(cfg, W):
    """States that hold on for hundreds of tokens, with a write of token MARKED that outweighs the others."""
    L = cfg["layers"][0]
    W["pos"] = W["pos"] * 0.02
    e = W["embed"][MARKED] / W["embed"][MARKED].norm() ** 2
    others = [t for t in range(cfg["vocab"]) if t != MARKED]        # no other token shares in what MARKED's row is turned to
    W["embed"][others] -= torch.outer(W["embed"][others] @ W["embed"][MARKED], e)
    if L["type"] == "mlstm":
        m = L["mixer"]
        _turn(W, "l0.mix.", m["heads"], m["heads"])
        W["l0.mix.f"], W["l0.mix.f.b"] = W["l0.mix.f"] * 0.1, torch.full_like(W["l0.mix.f.b"], 30.0)
        W["l0.mix.i"] = W["l0.mix.i"] * 0.1 + torch.outer(torch.ones(m["heads"], dtype=torch.float64) * 7.0, e)
        W["l0.mix.i.b"] = torch.full_like(W["l0.mix.i.b"], -3.0)
    else:
        m = L["mixer"]["right"]
        _turn(W, "l0.mix.right.", m["heads"], m["heads"])
        W["l0.mix.right.a2"], W["l0.mix.right.a2.b"] = W["l0.mix.right.a2"] * 0.1, torch.full_like(W["l0.mix.right.a2.b"], 7.0)
        W["l0.mix.right.k"] = 0.1 * W["l0.mix.right.k"] + torch.outer((W["l0.mix.right.k"] @ W["embed"][MARKED]) * 2.0, e)
        W["l0.mix.left.out"] = W["l0.mix.left.out"] * 0
    return W


MARKED_STATES = {
    "marked_memory": _model([_layer(_mem(2, 32, 48, 12.0))]),
    "marked_memory_no_fours": _model([_layer(_mem(3, 21, 15, 9.0))], width=52),
    "marked_linear": _model([_layer(_par((2, 1, 32, 32, 0.2, 10), (2, 64, 48, 16.0, 16)))]),
    "marked_linear_no_fours": _model([_layer(_par((2, 1, 32, 32, 0.2, 10), (3, 17, 22, 4.0, 5)))], width=60),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MARKED_STATES))
def test_a_write_far_back_in_the_state(folders, name, dtype):
    """At the chunks' edges of a prompt of its length, at the edges of portions, in the first tokens, and carried through decoding."""
    import plain_demazen as P
    from ultima_b200.kernels import ops
    d, cfg, W = folders(name, MARKED_STATES[name], _marked_state)
    eng = _engine(d, dtype, poison_cache=True)
    m = cfg["layers"][0]["mixer"]
    m = m.get("right", m)
    form = ops.LinForm(m["heads"], m["dim"], m["vdim"], (0,) * 6, rank=1, head_form="gate_cap" in m)
    n, size = ops.lin_chunks(form, 1, 450)
    assert n > 3
    for mk, p in ((0, 1), (0, 449), (1, 2), (3, 420), (size - 1, size), (size, 449), (size + 1, 2 * size), (63, 64), (2 * size - 1, 449)):
        ids = _ids(mk * 1000 + p, p + 1, cfg["vocab"], avoid=(ASKER, MARKED))
        ids[mk], ids[p] = MARKED, ASKER
        ref = P.logits(cfg, W, ids)[p]
        without = list(ids)
        without[mk] = ids[mk + 1] if mk + 1 < p else (ids[mk] + 1) % cfg["vocab"]
        bound = close_enough(ref[None], ref[None], dtype, 2)[1]
        moved = float(np.abs(P.logits(cfg, W, without)[p] - ref).max())
        assert moved > 3 * bound, (name, mk, p, moved, bound)        # the test's weights do show the write
        err = float(np.abs(_whole(eng, ids, [p])[0] - ref).max())
        assert err <= bound, (name, dtype, mk, p, "prompt", err, bound)
        got = _prompt_then_single_tokens(eng, ids, max(1, p - 3), want_from=max(1, p - 3) - 1)[-1]
        err = float(np.abs(got - ref).max())
        assert err <= bound, (name, dtype, mk, p, "decoded", err, bound)
        s = eng.open(1)                                             # the prompt in two portions that meet at the write
        eng.step(s, [ids[:mk + 1]], [[]])
        got = eng.step(s, [ids[mk + 1:]], [[p - mk - 1]]).cpu().numpy()[0]
        eng.close(s)
        assert float(np.abs(got - ref).max()) <= bound, (name, dtype, mk, p, "portions")


def test_the_running_maximum_starts_at_zero_and_the_denominators_floor_holds(folders):
    """Input gates far below zero from the first token on: the maximum is then the forget gate's sum, not the input gate, and the
    denominator is its floor; input gates far above: the other branch."""
    import plain_demazen as P

    def low(cfg, W):
        W["l0.mix.i.b"] = torch.tensor([-40.0, -6.0, 40.0], dtype=torch.float64)
        W["l0.mix.f.b"] = torch.tensor([3.0, 30.0, 1.0], dtype=torch.float64)
        return W
    d, cfg, W = folders("low_gates", _model([_layer(_mem(3, 16, 24, 5.0))], eps=1e-3), low)
    ids = _ids(2, 300, cfg["vocab"])
    ref = P.logits(cfg, W, ids)
    for dtype in ("float32", "bfloat16"):
        eng = _engine(d, dtype)
        agree(_whole(eng, ids), ref, dtype, 2, ("low gates", dtype))
        agree(_prompt_then_single_tokens(eng, ids, 1), ref, dtype, 2, ("low gates", dtype, "decoded"))


# ---------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_a_prompt_in_one_step_every_position_and_every_layer(folders, name, dtype):
    import plain_demazen as P
    d, cfg, W = folders(_for(name, dtype))
    eng = _engine(d, dtype, poison_cache=True)
    L = len(cfg["layers"])
    for seed, n in ((1, 1), (2, 2), (3, 277)):
        ids = _ids(seed, n, cfg["vocab"])
        taps, layers = [], []
        eng.model.tap = lambda i, x: taps.append(x.detach().double().cpu())
        got = _whole(eng, ids)
        eng.model.tap = None
        with torch.no_grad():
            ref = P.forward(cfg, W, ids, torch.float64, layers).numpy()
        assert len(taps) == len(layers) == L
        if dtype == "float32":
            for i, (a, b) in enumerate(zip(taps, layers)):
                assert rel_err(a, b) < 2e-5, (name, n, i)
        agree(got, ref, dtype, 3 * L, (name, dtype, n))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_against_token_by_token_and_portions(folders, name, dtype):
    import plain_demazen as P
    d, cfg, W = folders(_for(name, dtype))
    eng = _engine(d, dtype, poison_cache=True)
    n, layers = 150, 4 if dtype == "float32" else 3 * len(cfg["layers"])
    ids = _ids(11, n, cfg["vocab"])
    ref = P.logits(cfg, W, ids)
    for sizes in ([1] * n, [2] * 75, [3, 2, 64, 1, 65, 2, 13], [149, 1], [5] + [1] * 145):
        assert sum(sizes) == n
        s = eng.open(1)
        rows, at = [], 0
        for m in sizes:
            rows.append(eng.step(s, [ids[at:at + m]], [_all(m)]).cpu().numpy())
            at += m
        eng.close(s)
        eng.check_errors()
        agree(np.concatenate(rows), ref, dtype, layers, (name, sizes[:4]))
    small = _engine(d, dtype, max_step_tokens=16)                  # passes inside one step
    agree(_whole(small, ids), ref, dtype, layers, (name, "passes"))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_unequal_requests_together_then_decoded_with_slots_used_again(folders, name, dtype):
    import plain_demazen as P
    d, cfg, W = folders(_for(name, dtype))
    eng = _engine(d, dtype, poison_cache=True)
    L = len(cfg["layers"])
    for turn in range(2):                                          # the second time on slots and pages just given back
        lens, tail = [1, 130, 66, 23], [3, 20, 9, 20]
        seqs = [_ids(20 + 10 * turn + i, a + b, cfg["vocab"]) for i, (a, b) in enumerate(zip(lens, tail))]
        refs = [P.logits(cfg, W, s) for s in seqs]
        slots = eng.open(4)
        got = [dict() for _ in seqs]
        out = eng.step(slots, [s[:a] for s, a in zip(seqs, lens)], [_all(a) for a in lens]).cpu().numpy()
        o = 0
        for i, a in enumerate(lens):
            for p in range(a):
                got[i][p] = out[o]
                o += 1
        live = list(range(4))
        for t in range(max(tail)):
            live = [i for i in live if t < tail[i]]                # the shorter requests end earlier
            out = eng.step([slots[i] for i in live], [[seqs[i][lens[i] + t]] for i in live]).cpu().numpy()
            for r, i in enumerate(live):
                got[i][lens[i] + t] = out[r]
            for i in list(live):
                if t + 1 == tail[i]:
                    eng.close([slots[i]])
        eng.check_errors()
        for i, s in enumerate(seqs):
            agree(np.stack([got[i][p] for p in range(len(s))]), refs[i], dtype, 3 * L, (name, dtype, turn, i))
        # mixed: a portion of one request beside a single token of another
        slots = eng.open(2)
        a, b = seqs[1], seqs[2]
        rows = [eng.step(slots, [a[:40], b[:70]], [_all(40), _all(70)]).cpu().numpy()]
        rows.append(eng.step(slots, [a[40:41], b[70:75]], [[0], _all(5)]).cpu().numpy())
        rows.append(eng.step(slots, [a[41:100], b[75:]], [_all(59), _all(len(b) - 75)]).cpu().numpy()[:59])
        eng.close(slots)
        eng.check_errors()
        agree(np.concatenate([rows[0][:40], rows[1][:1], rows[2]]), refs[1][:100], dtype, 3 * L, (name, dtype, "mixed a"))
        agree(np.concatenate([rows[0][40:], rows[1][1:]]), refs[2][:75], dtype, 3 * L, (name, dtype, "mixed b"))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_decoding_over_page_borders(folders, name, dtype):
    import plain_demazen as P
    d, cfg, W = folders(_for(name, dtype))
    ids = _ids(5, 210, cfg["vocab"])
    agree(_prompt_then_single_tokens(_engine(d, dtype), ids, 4), P.logits(cfg, W, ids), dtype, 3 * len(cfg["layers"]), (name, dtype))


def test_the_last_position_of_the_table_and_none_beyond(folders):
    import plain_demazen as P
    from ultima_b200.engine.engine import StepError
    d, cfg, W = folders("few_positions", _model([_layer(_mem(2, 16, 24, 5.0))], positions=70))
    eng = _engine(d, "float32")
    ids = _ids(1, 71, cfg["vocab"])
    agree(_whole(eng, ids[:70]), P.logits(cfg, W, ids[:70]), "float32", 2, "all positions")
    s = eng.open(1)
    with pytest.raises(StepError):
        eng.step(s, [ids], [[70]])
    eng.close(s)


def test_greedy_generation_through_the_loop(folders):
    import plain_demazen as P
    import ultima_b200 as u
    d, cfg, W = folders("mixed")
    llm = u.LLM(d, dtype="float32", n_ctx=128, max_batch=2)
    prompts = [_ids(1, 9, cfg["vocab"]), _ids(2, 30, cfg["vocab"])]
    outs = llm.generate(prompts, n_predict=8, temp=0.0)
    for p, g in zip(prompts, outs):
        ids = list(p)
        for _ in range(8):
            ids.append(int(np.argmax(P.logits(cfg, W, ids)[-1])))
        assert g.tokens == ids[len(p):], (g.tokens, ids[len(p):])


def test_trace_replay_and_the_command_line(folders, tmp_path):
    import plain_demazen as P
    d, cfg, W = folders("odd")
    listed = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "ultima"), "archinfo", d], capture_output=True,
                            text=True, timeout=300)
    assert listed.returncode == 0 and "l0.mix.right.a2.b" in listed.stdout and "all " in listed.stdout, listed.stderr[-1500:]
    a, b = _ids(3, 70, cfg["vocab"]), _ids(4, 9, cfg["vocab"])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:5], "want": [4]}], "end": []}]
    for t in range(4):
        steps.append({"step": t + 1, "entries": [{"id": "a", "tokens": [a[66 + t]], "want": [0]},
                                                 {"id": "b", "tokens": [b[5 + t]], "want": [0]}],
                      "end": ["a", "b"] if t == 3 else []})
    steps.append({"step": 5, "entries": [{"id": "c", "tokens": b, "want": [8]}], "end": ["c"]})      # a slot used again
    for dtype in ("float32", "bfloat16"):
        d, cfg, W = folders(_for("mixed", dtype))
        ra, rb = P.logits(cfg, W, a), P.logits(cfg, W, b)
        out_dir = str(tmp_path / ("out_" + dtype))
        p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", dtype,
                            "--out", out_dir, "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps),
                           capture_output=True, text=True, timeout=900)
        assert p.returncode == 0 and "done 5" in p.stdout, p.stderr[-2000:]
        got = [np.fromfile(os.path.join(out_dir, "0.f32"), dtype="<f4").reshape(3, cfg["vocab"])]
        want = [ra[0], ra[65], rb[4]]
        for t in range(4):
            got.append(np.fromfile(os.path.join(out_dir, f"{t + 1}.f32"), dtype="<f4").reshape(2, cfg["vocab"]))
            want += [ra[66 + t], rb[5 + t]]
        got.append(np.fromfile(os.path.join(out_dir, "5.f32"), dtype="<f4").reshape(1, cfg["vocab"]))
        want.append(rb[8])
        agree(np.concatenate(got), np.stack(want), dtype, 18, dtype)
