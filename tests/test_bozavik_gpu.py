"""Bozavik on the GPU against the plain implementation (tests/plain_bozavik.py): the new kernels and options alone (norms
with a bias and the joining kernel, the router that weighs chosen logits, gated and clamped products, the placement's
sections, latent attention on the tensor cores), one-layer models of both mixers and of the feed-forward, keys made to stand
out at page borders and far away, a heavy sink, then whole models from small configurations with random weights: prompts,
token-by-token decoding, portions, batches of unequal requests, slots used again, long decoding, greedy generation, trace
replay."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from bozavik_configs import CONFIGS, _layer, _model, _moe, _plain, _rotated
from conftest import ROOT, close_enough, has_gpu

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


class _Rt:
    def __init__(self):
        self.status = torch.zeros(4, dtype=torch.int32, device=DEV)


# ---------------------------------------------------------------------------------------
# norms and the joining kernel
# ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,width", [(1, 48), (37, 100), (5, 257), (3, 1024), (9, 2048), (2, 4100), (2, 8200)])
def test_layer_norm_with_a_bias_and_the_join_with_a_norm_on_the_result(T, width, out_dtype):
    """Widths on the kernel with rows in registers and on the other; every kind of norm behind and ahead."""
    import plain_bozavik as P
    ops = _ops()
    g = torch.Generator().manual_seed(T * 7 + width)
    x, y = torch.randn(T, width, generator=g) * 3 + 1.5, torch.randn(T, width, generator=g) * 2 - 0.7
    aw, ab, nw, nb = (torch.randn(width, generator=g) for _ in range(4))
    tol = 1e-5 if out_dtype == torch.float32 else 2 ** -7
    out = torch.empty(T, width, dtype=out_dtype, device=DEV)
    ops.layernorm(x.to(DEV), nw.to(DEV), out, 1e-4, bias=nb.to(DEV))
    assert rel_err(out, P.layer_norm(x.double(), nw.double(), nb.double(), 1e-4)) < tol
    mult = 0.37
    for after, norm_y in ((ops.NEXT_LAYER, P.layer_norm(y.double(), aw.double(), ab.double(), 1e-3)),
                          (ops.NEXT_RMS, P.rms_norm(y.double(), aw.double(), 1e-3))):
        new = x.double() + mult * norm_y
        b = ab.to(DEV) if after == ops.NEXT_LAYER else None
        for mode, ref in ((ops.NEXT_NONE, None), (ops.NEXT_PLAIN, new), (ops.NEXT_RMS, P.rms_norm(new, nw.double(), 1e-5)),
                          (ops.NEXT_LAYER, P.layer_norm(new, nw.double(), nb.double(), 1e-5))):
            xd, yd = x.to(DEV), y.to(DEV)
            o = torch.empty(T, width, dtype=out_dtype, device=DEV) if ref is not None else None
            then = (nw.to(DEV), nb.to(DEV) if mode == ops.NEXT_LAYER else None, 1e-5) if mode >= ops.NEXT_RMS else None
            ops.norm_join(yd, xd, mult, (after, aw.to(DEV), b, 1e-3), mode, then, o)
            assert rel_err(xd, new) < 1e-6 and float(yd.abs().max()) == 0.0, (after, mode)
            if ref is not None:
                assert rel_err(o, ref) < tol, (after, mode)


def test_the_embedding_is_scaled_in_float32():
    ops = _ops()
    for width in (64, 37):
        table = torch.randn(11, width).to(torch.bfloat16)
        ids = torch.tensor([3, 10, 0], dtype=torch.int32)
        out = torch.empty(3, width, device=DEV)
        ops.embed(table.to(DEV), ids.to(DEV), out, torch.zeros(1, dtype=torch.int32, device=DEV), 12.7)
        assert rel_err(out, table[ids.long()].double() * 12.7) < 1e-7


# ---------------------------------------------------------------------------------------
# the router
# ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("ne,top,spread", [(6, 2, 2.0), (33, 5, 3.0), (4, 4, 1.0), (7, 1, 2.0), (12, 3, 300.0)])
def test_the_router_weighs_the_chosen_logits_and_hands_the_extra_column_on(ne, top, spread):
    """``spread`` 300: all but the largest logits vanish in a softmax over all outputs; the choice must not depend on that."""
    import plain_bozavik as P
    ops = _ops()
    T = 50
    g = torch.Generator().manual_seed(ne)
    z = torch.randn(T, ne + 1, generator=g) * spread                # one column behind the router's outputs
    ref_idx, ref_w = P.route(z[:, :ne].double(), {"r.router": torch.eye(ne, dtype=torch.float64)}, top, "r.")
    coarse = (z * 4).round() / 4
    for parts, zs in ((1, z), (3, torch.stack([coarse, z - coarse, torch.zeros_like(z)]))):
        for small in (False, True):
            n = min(T, ops.ROUTE_SMALL_TOKENS) if small else T
            zd = (zs[:n] if zs.dim() == 2 else zs[:, :n]).contiguous().to(DEV)
            idx, wts = torch.empty(n, top, dtype=torch.int32, device=DEV), torch.empty(n, top, device=DEV)
            extra = torch.full((n,), 7.0, device=DEV)
            if small:
                ws = [torch.zeros(k, dtype=torch.int32, device=DEV) for k in (4 * (n * top + ne), 1, n * top, n * top)]
                ops.route_small(zd, None, ne, top, 1, 1, idx, wts, ws[0].view(-1, 4), ws[1], ws[2].view(n, top), ws[3], 16,
                                mode=ops.ROUTE_LOGITS, extra=extra)
            else:
                counts = torch.zeros(ne, dtype=torch.int32, device=DEV)
                ops.route(zd, None, ne, top, 1, 1, idx, wts, counts, mode=ops.ROUTE_LOGITS, extra=extra)
                assert counts.cpu().tolist() == torch.bincount(ref_idx.flatten(), minlength=ne).tolist()
            assert torch.equal(idx.cpu().long(), ref_idx[:n]) and float((wts.cpu().double() - ref_w[:n]).abs().max()) < 2e-6
            assert float((extra.cpu() - z[:n, ne]).abs().max()) <= 1e-6 * spread
    # a view that leaves the extra column out gives the same choice
    idx, wts = torch.empty(T, top, dtype=torch.int32, device=DEV), torch.empty(T, top, device=DEV)
    ops.route(z.to(DEV)[:, :ne], None, ne, top, 1, 1, idx, wts, torch.zeros(ne, dtype=torch.int32, device=DEV), mode=ops.ROUTE_LOGITS)
    assert torch.equal(idx.cpu().long(), ref_idx)


# ---------------------------------------------------------------------------------------
# products with a sigmoid gate on the result, and clamped gate products
# ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [1, 37, 300])
def test_head_products_with_a_gate_a_head_or_an_element(T, dtype):
    """Gates in the columns of a wider row, on the tensor cores (bfloat16, sizes in eights) and on the CUDA cores."""
    from ultima_b200.engine import Runtime
    rt = Runtime(DEV, dtype)
    for B, K, N in ((3, 40, 72), (5, 24, 20), (2, 36, 16)):
        g = torch.Generator().manual_seed(T + N)
        a = torch.randn(T, B, K, generator=g).to(dtype).to(DEV)
        w = (torch.randn(B, N, K, generator=g) * 0.3).to(dtype).to(DEV)
        ref = torch.einsum("tbk,bnk->tbn", a.double().cpu(), w.double().cpu())
        wide = torch.randn(T, B * N + 9, generator=g) * 2
        for gate, factor in ((wide[:, 5:5 + B], torch.sigmoid(wide[:, 5:5 + B].double())[:, :, None]),
                             (wide[:, 9:], torch.sigmoid(wide[:, 9:].double()).view(T, B, N)), (None, 1.0)):
            out = torch.full((T, B, N), 3.0, dtype=dtype, device=DEV)
            dev_gate = None if gate is None else wide.to(DEV)[:, gate.storage_offset():gate.storage_offset() + gate.shape[1]]
            rt.matmul_heads(a, w, out, gate=dev_gate)
            assert rel_err(out, ref * factor) < (1e-5 if dtype == torch.float32 else 2 ** -7), (B, K, N)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,inner", [(1, 64), (5, 40), (50, 128), (400, 192), (1500, 256)])
def test_the_clamped_feed_forward_with_a_gate_a_token(T, inner, dtype):
    """Interleaved and separate gate and up rows, one tile and many, the two-CTA product; limits that bite on both sides."""
    import plain_bozavik as P
    from ultima_b200.engine import Runtime
    from ultima_b200.parts.mlp import GatedClamped
    rt = Runtime(DEV, dtype)
    width, limit = 96, 0.8
    g = torch.Generator().manual_seed(inner)
    W = {n: (torch.randn(*s, generator=g) * 0.15).to(torch.bfloat16) for n, s in
         (("gate", (inner, width)), ("up", (inner, width)), ("down", (width, inner)))}
    h = torch.randn(T, width, generator=g).to(torch.bfloat16)
    gates = torch.randn(T, 3, generator=g) * 2
    ff = GatedClamped(width, inner, limit)
    ff.bind({f"{n}_proj.weight": t.to(dtype).to(DEV) for n, t in W.items()}, rt)
    ref = P.clamped_expert(h.double(), {n: t.double() for n, t in W.items()}, limit, "")
    for gate, factor in ((None, 1.0), (gates.to(DEV)[:, 1], torch.sigmoid(gates[:, 1:2].double()))):
        y = torch.zeros(T, width, device=DEV)
        ff.forward(h.to(dtype).to(DEV), y, None, rt, row_gate=gate)
        assert rel_err(y, ref * factor) < (1e-5 if dtype == torch.float32 else 2 ** -6), (T, inner)
    rt.check_status()


@pytest.mark.parametrize("tile", [16, 64, 128])
def test_grouped_product_with_the_clamped_gate_product(tile):
    from ultima_b200.kernels import gemm_tc
    from ultima_b200.parts.routed import RoutePlan
    ops = _ops()
    counts = [0, 3, 130, tile, 17, 1]
    E, N, K, rows = len(counts), 72, 136, sum(counts)
    g = torch.Generator().manual_seed(tile)
    a = torch.randn(rows, K, generator=g).to(torch.bfloat16).to(DEV)
    w = (torch.randn(E, 2 * N, K, generator=g) * 0.2).to(torch.bfloat16).to(DEV)
    max_tiles = -(-rows // tile) + E
    tiles, ws = torch.zeros(max_tiles, 4, dtype=torch.int32, device=DEV), torch.zeros(3 * E + 1, dtype=torch.int32, device=DEV)
    ws[:E] = torch.tensor(counts, dtype=torch.int32)
    ops.route_plan(ws[:E], ws[E:2 * E], ws[2 * E:3 * E], tiles, ws[3 * E:], E, tile)
    plan = RoutePlan(tiles, ws[3 * E:], None, max_tiles, rows, gather=False, tile=tile)
    expert = torch.repeat_interleave(torch.arange(E), torch.tensor(counts))
    gate = torch.einsum("rk,rnk->rn", a.double().cpu(), w.double().cpu()[expert, :N])
    up = torch.einsum("rk,rnk->rn", a.double().cpu(), w.double().cpu()[expert, N:])
    consts = (1.3, 1.702, 1.0)
    gc, uc = torch.clamp(gate, max=1.3), torch.clamp(up, -1.3, 1.3)
    ref = gc * torch.sigmoid(1.702 * gc) * (uc + 1.0)
    out = torch.full((rows, N), 7.0, dtype=torch.bfloat16, device=DEV)
    gemm_tc.grouped(a, w[:, :N], out, plan, ops.EPI_SWIGLU, w[:, N:], _Rt(), gate=consts)
    assert rel_err(out, ref) < 2 ** -7
    if tile <= ops.ROUTE_TILE:
        out32 = torch.empty(rows, N, device=DEV)
        ops.gemm_grouped(a, w[:, :N], out32, tiles, ws[3 * E:], None, max_tiles, ops.EPI_SWIGLU, w[:, N:], gate=consts)
        assert rel_err(out32, ref) < 1e-5


# ---------------------------------------------------------------------------------------
# the placement kernel's sections
# ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("T", [3, 70])
@pytest.mark.parametrize("parts", [1, 3])
@pytest.mark.parametrize("act", [torch.float32, torch.bfloat16])
def test_the_placement_norms_two_latents_and_gathers_gates(T, parts, act):
    import plain_bozavik as P
    ops = _ops()
    q_rank, rank, rot, rd, gw = 40, 24, 12, 8, 11
    g = torch.Generator().manual_seed(T)
    x = torch.randn(T, q_rank + rank + rot + gw, generator=g)
    xs = torch.stack([x - 2.0, torch.full_like(x, 1.5), torch.full_like(x, 0.5)]) if parts == 3 else x
    pos = torch.arange(T, dtype=torch.int32) + 50                  # a sequence that goes on at position 50
    n_pages = -(-(T + 50) // 64)
    cache = torch.full((n_pages + 1, 1, 64, rank + rot), 9.0, dtype=act, device=DEV)
    table = torch.arange(n_pages, 0, -1, dtype=torch.int32, device=DEV).view(1, -1).contiguous()
    angle = pos.double()[:, None] * (100.0 ** (-2.0 * torch.arange(rd // 2, dtype=torch.float64) / rd))[None]
    full = torch.zeros(T + 50, rd // 2, dtype=torch.float64)
    full[50:] = angle
    wq, wc = 1 + 0.2 * torch.randn(q_rank, generator=g), 1 + 0.2 * torch.randn(rank, generator=g)
    dq = torch.empty(T, q_rank, dtype=act, device=DEV)
    gates = torch.empty(T, gw, device=DEV)
    ops.latent_place(xs.contiguous().to(DEV), k_cache=cache, table=table, ring=n_pages * 64, page=64, tok_pos=pos.to(DEV),
                     tok_seq=torch.zeros(T, dtype=torch.int32, device=DEV), c_off=q_rank, c_weight=wc.to(DEV), rank=rank, rot=rot,
                     cos=torch.cos(full).float().to(DEV), sin=torch.sin(full).float().to(DEV), rotary_dim=rd, eps=1e-3,
                     dq_off=0, dq_weight=wq.to(DEV), dq_out=dq, g_off=q_rank + rank + rot, gate_out=gates)
    tol = 3e-6 if act == torch.float32 else 2 ** -7
    xd = x.double()
    assert rel_err(dq, P.rms_norm(xd[:, :q_rank], wq.double(), 1e-3)) < tol
    assert rel_err(gates, xd[:, q_rank + rank + rot:]) < 3e-6
    kr = xd[:, q_rank + rank:q_rank + rank + rot].clone()
    u, v, c, s = kr[:, 0:rd:2].clone(), kr[:, 1:rd:2].clone(), torch.cos(angle), torch.sin(angle)
    kr[:, 0:rd:2], kr[:, 1:rd:2] = u * c - v * s, v * c + u * s
    row = torch.cat([P.rms_norm(xd[:, q_rank:q_rank + rank], wc.double(), 1e-3), kr], dim=1)
    got = cache.cpu()[table.cpu()[0].long()].view(-1, rank + rot)
    assert rel_err(got[50:50 + T], row) < tol and bool((got[:50] == 9.0).all()) and bool((got[50 + T:] == 9.0).all())


# ---------------------------------------------------------------------------------------
# latent attention on the tensor cores
# ---------------------------------------------------------------------------------------
class _KV:
    def __init__(self, k, table, ring, window):
        self.k = self.v = k
        self.table, self.ring, self.page, self.window = table, ring, 64, window


class _B:
    pass


def _latent_case(nh, row, rank, befores, news, seed, window=None, sink=False, slices=None, ring_pages=None, q_gain=1.0, key_row=None):
    from ultima_b200.engine import Runtime
    from ultima_b200.kernels import attn_tc
    rt = Runtime(DEV, torch.bfloat16)
    g = torch.Generator().manual_seed(seed)
    lens = [b + n for b, n in zip(befores, news)]
    pages = ring_pages or max(-(-n // 64) for n in lens)
    n_pages = len(lens) * pages + 3
    perm = torch.randperm(n_pages, generator=g)[:len(lens) * pages].view(len(lens), pages).to(torch.int32)
    cache = torch.full((n_pages, 1, 64, row), float("nan"), dtype=torch.bfloat16)      # unwritten rows must reach no result
    dense = []
    for s, n in enumerate(lens):
        k = torch.randn(n, row, generator=g).to(torch.bfloat16)
        if key_row is not None:
            key_row(k)
        for p in range(max(0, n - pages * 64), n):
            cache[perm[s, (p // 64) % pages], 0, p % 64] = k[p]
        dense.append(k.double())
    T = sum(news)
    q = (torch.randn(T, nh, row, generator=g) * q_gain).to(torch.bfloat16).to(DEV)
    sinks = (torch.randn(nh, generator=g) * 2).float() if sink else None
    b = _B()
    start = np.concatenate([[0], np.cumsum(news)]).astype(np.int32)
    b.seq_start = torch.tensor(start, device=DEV)
    b.seq_before = torch.tensor(befores, dtype=torch.int32, device=DEV)
    b.n_seqs, b.max_new, b.max_after = len(lens), max(news), max(lens)
    kv = _KV(cache.to(DEV), perm.to(DEV), pages * 64, window)
    scale = row ** -0.5
    out = torch.full((T, nh, rank), float("nan"), dtype=torch.bfloat16, device=DEV)
    assert attn_tc.accepts_latent(q, kv, row, rank, nh, scale)
    attn_tc.latent_attention(q, kv, out, b, nh, row, rank, scale, rt, window=window, slices=slices,
                             sink_vals=sinks.to(DEV) if sink else None)
    torch.cuda.synchronize()
    rt.check_status()
    worst, qd = 0.0, q.double().cpu()
    assert torch.isfinite(out).all()
    for s, (bf, n) in enumerate(zip(befores, news)):
        for t in range(n):
            pos = bf + t
            lo = max(0, pos - window + 1) if window else 0
            k = dense[s][lo:pos + 1]
            sc = qd[start[s] + t] @ k.T * scale
            if sink:
                sc = torch.cat([sc, sinks.double()[:, None]], dim=1)
            p = torch.softmax(sc, dim=1)[:, :pos + 1 - lo]
            worst = max(worst, rel_err(out[start[s] + t], p @ k[:, :rank]))
    return worst


LATENT_SHAPES = [(4, 144, 128), (6, 96, 96), (16, 256, 192), (32, 256, 256), (1, 64, 48), (128, 64, 8), (7, 40, 24), (3, 72, 56),
                 (5, 192, 144), (20, 320, 272), (2, 384, 320), (9, 448, 448), (12, 512, 512), (16, 576, 512)]


@pytest.mark.parametrize("nh,row,rank", LATENT_SHAPES)
def test_latent_attention_of_prompts(nh, row, rank):
    """Whole and continued prompts of unequal lengths; heads that do and do not divide 128; every number of row blocks; rows
    that end inside a block of 64 or of 16; values of one and of two parts."""
    for sink, (befores, news) in ((False, ([0, 0, 0, 0], [1, 17, 64, 130])), (True, ([5, 64, 130, 0], [70, 1, 33, 129]))):
        err = _latent_case(nh, row, rank, befores, news, seed=row + nh, sink=sink)
        assert err <= 2 ** -6, (sink, err)


@pytest.mark.parametrize("nh,row,rank", LATENT_SHAPES)
@pytest.mark.parametrize("slices", [None, 1, 3, 16])
def test_latent_attention_of_single_tokens(nh, row, rank, slices):
    for sink in (False, True):
        err = _latent_case(nh, row, rank, [0, 63, 64, 300, 700], [1] * 5, seed=row + 3, sink=sink, slices=slices)
        assert err <= 2 ** -6, (sink, err)


@pytest.mark.parametrize("row,rank", [(96, 64), (256, 192), (576, 512)])
def test_latent_attention_with_a_window_on_a_wrapped_ring(row, rank):
    for befores, news in (([127, 200, 257, 60], [20, 29, 5, 29]), ([100, 120, 128, 500], [1, 1, 1, 1])):
        err = _latent_case(4, row, rank, befores, news, seed=row, window=100, ring_pages=2)
        assert err <= 2 ** -6, (befores, err)


@pytest.mark.parametrize("row,rank", [(128, 128), (576, 512)])
def test_latent_attention_rescales_when_the_maximum_grows(row, rank):
    """Keys that grow along the sequence push the reference maximum up again and again."""
    def grow(k):
        k[:, 0] = torch.linspace(0, 60, k.shape[0]).to(torch.bfloat16)
    err = _latent_case(3, row, rank, [0, 40], [330, 1], seed=5, sink=True, q_gain=6.0, key_row=grow)
    assert err <= 2 ** -5, err


# ---------------------------------------------------------------------------------------
# models of one layer
# ---------------------------------------------------------------------------------------
_SMALL = _plain(2, 16, 8, 16, 24, 0.2)
ONE_LAYER = {
    "plain_latent": _model([_layer(_plain(3, 24, 40, 56, 48, 0.2))], width=56, scale=2.0, mult=0.9),
    "plain_latent_one_head": _model([_layer(_plain(1, 40, 72, 8, 256, 0.1))], mult=1.0),
    "plain_latent_many_heads": _model([_layer(_plain(24, 8, 16, 32, 64, 0.3))], width=40, eps=1e-3),
    "rotated_whole": _model([_layer(_rotated(4, 16, 24, 40, 32, 0.17, 16, 10000.0))], scale=1.0),
    "rotated_in_part": _model([_layer(_rotated(5, 8, 8, 24, 40, 0.3, 24, 77.0, 10))], width=72),
    "rotated_wide_row": _model([_layer(_rotated(2, 32, 16, 24, 320, 0.1, 32, 500.0))]),
    "rotated_row_of_sixteens": _model([_layer(_rotated(5, 12, 20, 16, 20, 0.3, 12, 900.0))]),      # the mma.sync kernel's: rank no multiple of 8
    "rotated_no_eights": _model([_layer(_rotated(3, 10, 14, 19, 21, 0.3, 6, 300.0, 4))], width=50),
    "routed": _model([_layer(_SMALL, _moe(10, 3, 24, 1.0, (40, 0.6)))], mult=0.7),
    "routed_no_shared": _model([_layer(_SMALL, _moe(7, 1, 64, 2.0))], width=80),
    "routed_all_chosen": _model([_layer(_SMALL, _moe(3, 3, 128, 0.5, (64, 1.5)))], width=48),
    "routed_no_eights": _model([_layer(_SMALL, _moe(6, 2, 21, 1.3, (13, 0.9)))], width=50),
}


def _sharpen(W, amp=1.7):
    """Random weights scaled so that attention weights are far from uniform, sinks weigh something, gates are open and shut,
    the experts' limits bite and the router's logits are far from equal."""
    out = {}
    for n, t in W.items():
        leaf = n.split(".")[-1]
        if ".mix." in n and t.dim() == 2 and leaf in ("uq", "uk", "g"):
            t = t * amp
        if leaf == "sink":
            t = t * 2 + 1.5
        if ".mlp." in n and leaf in ("gate", "up"):
            t = t * 3
        if n == "head":
            t = t * amp
        out[n] = t.to(torch.bfloat16)
    return out


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    import plain_bozavik as P
    import ultima_b200 as u
    from ultima_b200.weights.safetensors_io import write_safetensors
    base = tmp_path_factory.mktemp("bozavik")
    made = {}

    def get(name, raw=None, change=None):
        if name not in made:
            d = str(base / name.replace("/", "_"))
            plain_name = name.split("/")[0]
            raw = copy.deepcopy(raw or CONFIGS.get(plain_name) or ONE_LAYER[plain_name])
            if name.endswith("/all_chosen"):
                for L in raw["layers"]:
                    if L.get("mlp"):
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
    one other choice reaches every later position through the keys; so the bfloat16 runs of whole models use the same models
    with routers that choose every output (the weights still differ from token to token).  The choice itself is held to the
    plain implementation by the 32-bit runs of the same models, by the one-layer models in both types and by the router's
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
    import plain_bozavik as P
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
    import plain_bozavik as P

    def moved(name, change):
        _, cfg, W = folders(name)
        ids = _ids(1, 60, cfg["vocab"])
        cfg2, W2 = copy.deepcopy(cfg), dict(W)
        change(cfg2, W2)
        a, b = P.logits(cfg, W, ids), P.logits(cfg2, W2, ids)
        return float(np.abs(a - b).max() / np.abs(a).max())

    def setw(name, f):
        return lambda c, W: W.__setitem__(name, f(W[name]))
    zero = torch.zeros_like
    cases = [("plain_latent", setw("l0.mix.sink", lambda t: t - 60)), ("plain_latent", setw("l0.mix.g", zero)),
             ("plain_latent", setw("l0.norm1.b", zero)), ("plain_latent", setw("l0.norm1b.b", zero)),
             ("plain_latent", setw("l0.mix.dq.norm", torch.ones_like)), ("plain_latent", lambda c, W: c["embedding"].update(scale=1.0)),
             ("plain_latent", lambda c, W: c.update(residual_mult=0.5)), ("rotated_whole", setw("l0.mix.g", zero)),
             ("rotated_in_part", lambda c, W: c["layers"][0]["mixer"]["rot"].update(dims=24)),
             ("rotated_whole", lambda c, W: c["layers"][0]["mixer"]["rot"].update(base=100.0)),
             ("routed", lambda c, W: c["layers"][0]["mlp"]["expert"].update(limit=9.0)),
             ("routed", lambda c, W: c["layers"][0]["mlp"]["shared"].update(limit=1.0)),
             ("routed", setw("l0.mlp.shared.sg", zero)), ("routed", setw("l0.mlp.router", zero)),
             ("routed", setw("l0.norm2b.b", zero))]
    for i, (name, change) in enumerate(cases):
        m = moved(name, change)
        assert m > 0.02, (i, name, m)


# ---------------------------------------------------------------------------------------
# one key made to stand out
# ---------------------------------------------------------------------------------------
ASKER, MARKED = 5, 11


def _stand_out(cfg, W):
    """Layer 0's queries of token ASKER are turned towards the keys of token MARKED (a rank-one change of W_uq a head), so that
    this one score lies far above the others, and MARKED's values are made large."""
    import plain_bozavik as P
    m, eps = cfg["layers"][0]["mixer"], cfg["norm"]["eps"]
    h = {t: P.layer_norm(W["embed"][t] * cfg["embedding"]["scale"], W["l0.norm1"], W["l0.norm1.b"], eps) for t in (ASKER, MARKED)}
    cq = P.rms_norm(W["l0.mix.dq"] @ h[ASKER], W["l0.mix.dq.norm"], eps)
    H, d, r, rank = m["heads"], m["dim"], m.get("rot_dim", 0), m["kv_rank"]
    c = P.rms_norm((W["l0.mix.dkv"] @ h[MARKED])[:rank], W["l0.mix.dkv.norm"], eps)
    k = (W["l0.mix.uk"] @ c).view(H, d)
    uq = W["l0.mix.uq"].clone()
    for a in range(H):
        uq[a * (d + r):a * (d + r) + d] += torch.outer(k[a] / k[a].norm() ** 2 * (12.0 / m["scale"]), cq / (cq @ cq))
    W["l0.mix.uq"] = uq
    W["l0.mix.uv"] = W["l0.mix.uv"] + torch.outer(torch.ones(W["l0.mix.uv"].shape[0], dtype=torch.float64) * 0.7, c / (c @ c))
    W["l0.mix.g"] = W["l0.mix.g"] * 0.2
    if "l0.mix.sink" in W:
        W["l0.mix.sink"] = W["l0.mix.sink"] * 0.3
    return W


MARKED_MODELS = {
    "marked_plain": _model([_layer(_plain(4, 32, 16, 48, 64, 0.2)), _layer(_plain(2, 16, 16, 16, 32, 0.2))]),
    "marked_rotated": _model([_layer(_rotated(4, 32, 24, 40, 48, 0.17, 16, 10000.0)), _layer(_plain(2, 16, 16, 16, 32, 0.2))]),
    "marked_rotated_deep": _model([_layer(_rotated(3, 24, 16, 48, 512, 0.2, 64, 300.0))]),
    "marked_plain_no_eights": _model([_layer(_plain(3, 28, 20, 30, 44, 0.2))], width=52),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MARKED_MODELS))
def test_a_key_at_page_borders_far_away_and_among_the_first_tokens(folders, name, dtype):
    import plain_bozavik as P
    d, cfg, W = folders(name, MARKED_MODELS[name], _stand_out)
    eng = _engine(d, dtype, poison_cache=True)
    for m, p in ((0, 1), (0, 449), (1, 2), (3, 420), (31, 32), (32, 96), (62, 63), (63, 64), (64, 65), (64, 300), (127, 128), (128, 192),
                 (255, 449)):
        ids = _ids(m * 1000 + p, p + 1, cfg["vocab"], avoid=(ASKER, MARKED))
        ids[m], ids[p] = MARKED, ASKER
        ref = P.logits(cfg, W, ids)[p]
        without = list(ids)
        without[m] = ids[m + 1] if m + 1 < p else (ids[m] + 1) % cfg["vocab"]
        bound = close_enough(ref[None], ref[None], dtype, 2)[1]
        moved = float(np.abs(P.logits(cfg, W, without)[p] - ref).max())
        assert moved > 3 * bound, (name, m, p, moved, bound)        # the test's weights do show the key
        err = float(np.abs(_whole(eng, ids, [p])[0] - ref).max())
        assert err <= bound, (name, dtype, m, p, "prompt", err, bound)
        cut = max(1, p - 3)                                         # and decoded alone, three tokens behind the prompt
        got = _prompt_then_single_tokens(eng, ids, cut, want_from=cut - 1)[-1]
        err = float(np.abs(got - ref).max())
        assert err <= bound, (name, dtype, m, p, "decoded", err, bound)


def test_a_heavy_sink(folders):
    """A sink that is left out, counted twice or scaled would hide behind random weights; here it outweighs the keys."""
    import plain_bozavik as P

    def heavy(cfg, W):
        W["l0.mix.sink"] = torch.tensor([6.0, -3.0, 4.0], dtype=torch.float64)
        return W
    d, cfg, W = folders("heavy_sink", _model([_layer(_plain(3, 16, 16, 24, 32, 0.25))]), heavy)
    ids = _ids(1, 300, cfg["vocab"])
    ref = P.logits(cfg, W, ids)
    for other in (-50.0, np.log(2.0)):
        changed = P.logits(cfg, {**W, "l0.mix.sink": W["l0.mix.sink"] + other}, ids)
        assert np.abs(changed - ref).max() > 0.05 * np.abs(ref).max()
    for dtype in ("float32", "bfloat16"):
        eng = _engine(d, dtype)
        agree(_whole(eng, ids), ref, dtype, 2, ("sink", dtype))
        agree(_prompt_then_single_tokens(eng, ids, 200)[-100:], ref[-100:], dtype, 2, ("sink", dtype, "decoded"))


# ---------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_a_prompt_in_one_step_every_position_and_every_layer(folders, name, dtype):
    import plain_bozavik as P
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
        agree(got, ref, dtype, 2 * L, (name, dtype, n))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_against_token_by_token_and_portions(folders, name, dtype):
    import plain_bozavik as P
    d, cfg, W = folders(_for(name, dtype))
    eng = _engine(d, dtype, poison_cache=True)
    n, layers = 150, 4 if dtype == "float32" else 2 * len(cfg["layers"])
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
    import plain_bozavik as P
    d, cfg, W = folders(_for(name, dtype))
    eng = _engine(d, dtype, poison_cache=True)
    L = len(cfg["layers"])
    for round_ in range(2):                                        # the second time on slots and pages just given back
        lens, tail = [1, 130, 66, 23], [3, 20, 9, 20]
        seqs = [_ids(20 + 10 * round_ + i, a + b, cfg["vocab"]) for i, (a, b) in enumerate(zip(lens, tail))]
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
            agree(np.stack([got[i][p] for p in range(len(s))]), refs[i], dtype, 2 * L, (name, dtype, round_, i))
        # mixed: a portion of one request beside a single token of another
        slots = eng.open(2)
        a, b = seqs[1], seqs[2]
        rows = [eng.step(slots, [a[:40], b[:70]], [_all(40), _all(70)]).cpu().numpy()]
        rows.append(eng.step(slots, [a[40:41], b[70:75]], [[0], _all(5)]).cpu().numpy())
        rows.append(eng.step(slots, [a[41:100], b[75:]], [_all(59), _all(len(b) - 75)]).cpu().numpy()[:59])
        eng.close(slots)
        eng.check_errors()
        agree(np.concatenate([rows[0][:40], rows[1][:1], rows[2]]), refs[1][:100], dtype, 2 * L, (name, dtype, "mixed a"))
        agree(np.concatenate([rows[0][40:], rows[1][1:]]), refs[2][:75], dtype, 2 * L, (name, dtype, "mixed b"))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_decoding_over_page_borders(folders, name, dtype):
    import plain_bozavik as P
    d, cfg, W = folders(_for(name, dtype))
    ids = _ids(5, 210, cfg["vocab"])
    agree(_prompt_then_single_tokens(_engine(d, dtype), ids, 4), P.logits(cfg, W, ids), dtype, 2 * len(cfg["layers"]), (name, dtype))


def test_layers_before_and_after_one_with_another_arrangement(folders):
    """The join hands the next layer's input on only to a layer that takes it; a run list that repeats layers or holds other
    arrangements must come out the same.  Here: the same model with every norm handed on, and with none."""
    d, cfg, W = folders("mixed")
    eng = _engine(d, "float32")
    ids = _ids(8, 60, cfg["vocab"])
    a = _whole(eng, ids)
    held = eng.model._following
    eng.model._following = [None] * len(held)
    b = _whole(eng, ids)
    eng.model._following = held
    assert np.abs(a - b).max() <= 1e-4 * np.abs(a).max()


def test_greedy_generation_through_the_loop(folders):
    import plain_bozavik as P
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
    import plain_bozavik as P
    d, cfg, W = folders("odd")
    listed = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "ultima"), "archinfo", d], capture_output=True,
                            text=True, timeout=300)
    assert listed.returncode == 0 and "l0.mix.dkv.norm" in listed.stdout and "all " in listed.stdout, listed.stderr[-1500:]
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
        agree(np.concatenate(got), np.stack(want), dtype, 8, dtype)
