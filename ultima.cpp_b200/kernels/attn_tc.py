"""Entry point of the tensor-core attention kernels (csrc/attn_mma.cu), which are compiled
once for each head size a model uses."""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p

import torch

from . import build
from .ops import KernelError, _check, _ptr, _stream, sm_count

SOURCE = "attn_mma.cu"
import os as _os
SLICE_FACTOR = int(_os.environ.get("ULTIMA_SLICE_FACTOR", "2"))
SLICE_CAP = int(_os.environ.get("ULTIMA_SLICE_CAP", "16"))
_libs: dict = {}


def target(head_dim: int, value_dim: int | None = None):
    extra = tuple(x for x in _os.environ.get("ULTIMA_ATTN_DEFINES", "").split(",") if x)
    if value_dim is not None and value_dim != head_dim:
        extra = (f"HEAD_DIM_V={int(value_dim)}",) + extra
    return (SOURCE, (f"HEAD_DIM={int(head_dim)}",) + extra)


def sizes_fit(head_dim: int, value_dim: int) -> bool:
    """Whether the mma.sync kernels are built for these sizes of queries and keys and of values."""
    return all(d % 16 == 0 and 16 <= d <= 256 for d in (head_dim, value_dim))


def lib(head_dim: int, value_dim: int | None = None):
    value_dim = value_dim or head_dim
    L = _libs.get((head_dim, value_dim))
    if L is None:
        L = build.load(*target(head_dim, value_dim))
        L.ub_attn_mma.argtypes = [c_int, c_void_p, c_longlong, c_void_p, c_longlong, c_void_p, c_void_p, c_void_p,
                                  c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                                  c_float, c_int, c_void_p, c_void_p, c_void_p]
        L.ub_attn_mma.restype = c_int
        L.ub_attn_mma_ext.argtypes = L.ub_attn_mma.argtypes[:-1] + [c_int, c_int, c_void_p, c_float, c_void_p, c_longlong, c_float, c_void_p,
                                                                       c_int, c_void_p, c_void_p]
        L.ub_attn_mma_ext.restype = c_int
        L.ub_attn_head_dim.restype = c_int
        L.ub_attn_value_dim.restype = c_int
        if L.ub_attn_head_dim() != head_dim or L.ub_attn_value_dim() != value_dim:
            raise KernelError(f"attention library was built for head size {L.ub_attn_head_dim()} (values {L.ub_attn_value_dim()}), not "
                              f"{head_dim} ({value_dim})")
        if head_dim % 64 == 0 and value_dim == head_dim:
            L.ub_attn_map_kv.argtypes = [c_void_p, c_void_p, c_longlong, c_int]
            L.ub_attn_map_kv.restype = c_int
            L.ub_attn_decode_tma.argtypes = [c_void_p, c_void_p, c_void_p, c_longlong, c_void_p, c_longlong, c_void_p,
                                             c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int, c_int,
                                             c_float, c_int, c_void_p, c_void_p, c_void_p, c_void_p]
            L.ub_attn_decode_tma.restype = c_int
            L.ub_attn_decode_tma_qkv.argtypes = [c_void_p, c_void_p, c_void_p, c_int, c_longlong, c_void_p, c_void_p,
                                                 c_void_p, c_void_p, c_float, c_void_p, c_void_p, c_void_p, c_longlong,
                                                 c_void_p, c_void_p, c_void_p, c_int, c_int, c_int, c_int, c_int, c_int,
                                                 c_int, c_float, c_int, c_void_p, c_void_p, c_void_p, c_void_p]
            L.ub_attn_decode_tma_qkv.restype = c_int
        _libs[(head_dim, value_dim)] = L
    return L


TC_SOURCE = "attn_tcgen05.cu"
_tc_libs: dict = {}
_tc_maps: dict = {}
USE_TCGEN05 = _os.environ.get("ULTIMA_ATTN_TCGEN05", "1") != "0"
USE_TCGEN05_DECODE = _os.environ.get("ULTIMA_ATTN_TCGEN05_DECODE", "0") != "0"
USE_TMA_DECODE = _os.environ.get("ULTIMA_ATTN_TMA_DECODE", "1") != "0"
# prompts on the tcgen05 kernel: 1 = 256 rows a CTA when that still gives every SM a CTA, 0 = always 128 rows
# a CTA, 2 = always 256
WIDE = int(_os.environ.get("ULTIMA_ATTN_WIDE", "1"))


def tc_target(head_dim: int, value_dim: int | None = None):
    own = (f"HEAD_DIM_V={int(value_dim)}",) if value_dim is not None and value_dim != head_dim else ()
    return (TC_SOURCE, (f"HEAD_DIM={int(head_dim)}",) + own)


def tc_sizes_fit(head_dim: int, value_dim: int) -> bool:
    """The sizes the tcgen05 kernels are built for: 64 and 128, and for prompts values of another size than keys (keys in
    sixteens, values in thirty-twos, up to 256)."""
    if head_dim == value_dim:
        return head_dim in (64, 128)
    return head_dim % 16 == 0 and 16 <= head_dim <= 256 and value_dim % 32 == 0 and 32 <= value_dim <= 256


def tc_lib(head_dim: int, value_dim: int | None = None):
    value_dim = value_dim or head_dim
    L = _tc_libs.get((head_dim, value_dim))
    if L is None:
        L = build.load(*tc_target(head_dim, value_dim))
        L.ub_attn_tc_map_q.argtypes = [c_void_p, c_void_p, c_longlong, c_int, c_longlong, c_int]
        L.ub_attn_tc_map_q.restype = c_int
        L.ub_attn_tc_map_kv.argtypes = [c_void_p, c_void_p, c_longlong, c_int, c_int]
        L.ub_attn_tc_map_kv.restype = c_int
        L.ub_attn_tc.argtypes = [c_int, c_void_p, c_void_p, c_void_p, c_void_p, c_longlong, c_void_p, c_void_p, c_void_p,
                                 c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_int, c_void_p,
                                 c_void_p, c_void_p, c_void_p]
        L.ub_attn_tc.restype = c_int
        L.ub_attn_tc_ext.argtypes = [c_void_p, c_void_p, c_void_p, c_void_p, c_longlong, c_void_p, c_void_p, c_void_p,
                                     c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_void_p,
                                     c_int, c_float, c_void_p, c_longlong, c_void_p]
        L.ub_attn_tc_ext.restype = c_int
        L.ub_attn_tc_set_wide.argtypes = [c_int]
        L.ub_attn_tc_set_wide.restype = None
        L.ub_attn_tc_set_wide(WIDE)
        if L.ub_attn_tc_head_dim() != head_dim or L.ub_attn_tc_value_dim() != value_dim:
            raise KernelError(f"attention library was built for head size {L.ub_attn_tc_head_dim()} (values {L.ub_attn_tc_value_dim()}), "
                              f"not {head_dim} ({value_dim})")
        _tc_libs[(head_dim, value_dim)] = L
    return L


def set_wide(mode: int) -> None:
    """Choose between the two prompt kernels (see ``WIDE``) in every library loaded so far and later."""
    global WIDE
    WIDE = int(mode)
    for L in _tc_libs.values():
        L.ub_attn_tc_set_wide(WIDE)


def tcgen05_fits(head_dim: int, n_heads: int, n_kv_heads: int, value_dim: int | None = None) -> bool:
    """The tcgen05 kernel: sizes it is built for, groups of up to 128 query heads a KV head."""
    return USE_TCGEN05 and tc_sizes_fit(head_dim, value_dim or head_dim) and n_heads // n_kv_heads <= 128


def _tc_map(key, make):
    import ctypes
    hit = _tc_maps.get(key)
    if hit is not None:
        return hit[1]
    raw = ctypes.create_string_buffer(128 + 64)
    addr = (ctypes.addressof(raw) + 63) & ~63
    rc = make(addr)
    if rc != 0:
        raise KernelError(f"tensor map for attention could not be made (code {rc})")
    if len(_tc_maps) > 1024:
        _tc_maps.clear()
    _tc_maps[key] = (raw, addr)
    return addr


def run_tcgen05(q, kv, out, batch, n_heads, n_kv_heads, head_dim, scale, rt, decode: bool, n_slices: int = 1,
                mask: int | None = None):
    value_dim = kv.v.shape[-1]
    L = tc_lib(head_dim, value_dim)
    group = n_heads // n_kv_heads
    T = q.shape[0]
    mq = _tc_map(("q", q.data_ptr(), T, n_heads, q.stride(0), group, head_dim),
                 lambda a: L.ub_attn_tc_map_q(a, q.data_ptr(), T, n_heads, q.stride(0), group))
    mk = _tc_map(("kv", kv.k.data_ptr(), kv.k.shape[0], n_kv_heads, head_dim),
                 lambda a: L.ub_attn_tc_map_kv(a, kv.k.data_ptr(), kv.k.shape[0], n_kv_heads, head_dim))
    mv = _tc_map(("kv", kv.v.data_ptr(), kv.v.shape[0], n_kv_heads, value_dim),
                 lambda a: L.ub_attn_tc_map_kv(a, kv.v.data_ptr(), kv.v.shape[0], n_kv_heads, value_dim))
    part_o = part_ml = None
    if decode and n_slices > 1:
        part_o = rt.arena.alloc((batch.n_seqs, n_heads, n_slices, value_dim), torch.float32)
        part_ml = rt.arena.alloc((batch.n_seqs, n_heads, n_slices, 2), torch.float32)
    rc = L.ub_attn_tc(1 if decode else 0, mq, mk, mv, _ptr(out), out.stride(0), _ptr(batch.seq_start),
                      _ptr(batch.seq_before), _ptr(kv.table), kv.table.shape[1], kv.ring, kv.page, batch.n_seqs,
                      batch.max_new, n_heads, n_kv_heads, int(kv.window or 0) if mask is None else mask, float(scale),
                      n_slices, _ptr(part_o), _ptr(part_ml), _ptr(rt.status[1:2]), _stream())
    _check(rc, "attn_tc")


def accepts(q, kv, head_dim, n_heads, n_kv_heads) -> bool:
    return (q.dtype == torch.bfloat16 and kv.k.dtype == torch.bfloat16 and head_dim % 16 == 0
            and 16 <= head_dim <= 256 and kv.page == 64 and q.stride(1) == 1 and q.stride(0) % 8 == 0
            and q.data_ptr() % 16 == 0)


def decode_slices(n_seqs: int, n_kv_heads: int, longest: int, window, per_sm: int = SLICE_FACTOR,
                  n_sms: int | None = None, cap: int = SLICE_CAP) -> int:
    """Slices of the key range, so that a decode step with few sequences still fills the GPU
    (``per_sm`` CTAs an SM; ``n_sms``: the device's multiprocessors, asked of it when not given)."""
    span = longest if not window else min(longest, window + 64)
    tiles = max(1, -(-span // 64))
    ctas = n_seqs * n_kv_heads
    want = -(-per_sm * (n_sms or sm_count()) // ctas)
    n = max(1, min(want, tiles, cap))
    return 1 << (n.bit_length() - 1)            # a power of two: few distinct captured graphs


# ULTIMA_ATTN_LATENT=0: latent attention stays on the any-shape kernel; 1: not on the tcgen05 kernel
LATENT = int(_os.environ.get("ULTIMA_ATTN_LATENT", "2"))
LATENT_SLICE_CAP = int(_os.environ.get("ULTIMA_LATENT_SLICE_CAP", "64"))
LATENT_SOURCE = "attn_latent.cu"
_latent_libs: dict = {}


def latent_fits(row: int, rank: int, n_heads: int) -> bool:
    """The tcgen05 kernel of latent attention (csrc/attn_latent.cu): rows and values in eights, up to 576 and 512 of them,
    up to 128 heads."""
    return LATENT >= 2 and row % 8 == 0 and rank % 8 == 0 and 8 <= rank <= min(row, 512) and row <= 576 and n_heads <= 128


def latent_target(row: int):
    return (LATENT_SOURCE, (f"ROW_BLOCKS={-(-int(row) // 64)}",))


def latent_needs(row: int, rank: int, n_heads: int) -> list:
    """The libraries latent attention over key rows of ``row`` numbers uses beyond the any-shape kernel."""
    if latent_fits(row, rank, n_heads):
        return [latent_target(row)]
    if LATENT and row % 16 == 0 and 16 <= row <= 256:
        return [target(row)]
    return []


def latent_lib(row: int):
    blocks = -(-int(row) // 64)
    L = _latent_libs.get(blocks)
    if L is None:
        L = build.load(*latent_target(row))
        L.ub_attn_latent_map_q.argtypes = [c_void_p, c_void_p, c_longlong, c_int, c_longlong, c_int]
        L.ub_attn_latent_map_q.restype = c_int
        L.ub_attn_latent_map_k.argtypes = [c_void_p, c_void_p, c_longlong, c_int]
        L.ub_attn_latent_map_k.restype = c_int
        L.ub_attn_latent.argtypes = [c_int, c_void_p, c_void_p, c_void_p, c_longlong, c_void_p, c_void_p, c_void_p, c_int, c_int,
                                     c_int, c_int, c_int, c_int, c_int, c_int, c_int, c_float, c_void_p, c_int, c_void_p, c_void_p,
                                     c_void_p, c_void_p]
        L.ub_attn_latent.restype = c_int
        if L.ub_attn_latent_row_blocks() != blocks:
            raise KernelError(f"latent attention library was built for {L.ub_attn_latent_row_blocks()} row blocks, not {blocks}")
        _latent_libs[blocks] = L
    return L


def accepts_latent(q, kv, row: int, rank: int, n_heads: int, scale: float) -> bool:
    return (latent_fits(row, rank, n_heads) and scale > 0 and q.dtype == torch.bfloat16 and kv.k.dtype == torch.bfloat16
            and kv.page == 64 and kv.k.is_contiguous() and q.is_contiguous() and q.data_ptr() % 16 == 0 and kv.k.data_ptr() % 16 == 0)


def latent_attention(q, kv, out, batch, n_heads, row, rank, scale, rt, window=None, sink_vals=None, slices: int | None = None):
    """q [T, heads, row] over one key head whose rows of ``row`` numbers have the values as their leading ``rank`` columns;
    out [T, heads, rank].  ``sink_vals`` float32 [heads]: one more term exp(sink) in the softmax's sum."""
    L = latent_lib(row)
    T = q.shape[0]
    assert out.dtype == torch.bfloat16 and out.is_contiguous() and out.shape == (T, n_heads, rank)
    assert sink_vals is None or (sink_vals.dtype == torch.float32 and sink_vals.is_contiguous() and sink_vals.numel() == n_heads)
    decode = batch.max_new == 1 and batch.n_seqs == T
    mq = _tc_map(("lq", q.data_ptr(), T, n_heads, row), lambda a: L.ub_attn_latent_map_q(a, q.data_ptr(), T, n_heads, n_heads * row, row))
    mk = _tc_map(("lk", kv.k.data_ptr(), kv.k.shape[0], row), lambda a: L.ub_attn_latent_map_k(a, kv.k.data_ptr(), kv.k.shape[0], row))
    part_o = part_ml = None
    n_slices = 1
    if decode:
        parts = -(-rank // 256)
        n_slices = slices or latent_slices(batch.n_seqs, batch.max_after, window, parts)
        if n_slices > 1:
            part_o = rt.arena.alloc((batch.n_seqs, n_heads, n_slices, rank), torch.float32)
            part_ml = rt.arena.alloc((batch.n_seqs, n_heads, n_slices, 2), torch.float32)
    rc = L.ub_attn_latent(1 if decode else 0, mq, mk, _ptr(out), n_heads * rank, _ptr(batch.seq_start), _ptr(batch.seq_before),
                          _ptr(kv.table), kv.table.shape[1], kv.ring, kv.page, batch.n_seqs, batch.max_new, n_heads, row, rank,
                          int(window or 0), float(scale), _ptr(sink_vals), n_slices, _ptr(part_o), _ptr(part_ml),
                          _ptr(rt.status[1:2]), _stream())
    _check(rc, "attn_latent")


def latent_slices(n_seqs: int, longest: int, window, parts: int = 1, n_sms: int | None = None) -> int:
    """Slices of the key range of a latent decode step: a CTA an SM.  What ``decode_slices`` gives with the same cap and more
    CTAs an SM determines it, so that is what a captured step may be looked up by."""
    return decode_slices(n_seqs * parts, 1, longest, window, per_sm=1, n_sms=n_sms, cap=LATENT_SLICE_CAP)


FUSE_QKV = _os.environ.get("ULTIMA_ATTN_FUSE_QKV", "1") != "0"


def decode_from_qkv(qkv, q_norm, k_norm, cos, sin, eps, kv, out, batch, n_heads, n_kv_heads, head_dim, scale, rt,
                    slices: int | None = None, force: bool = False) -> bool:
    """A step of one token a sequence, straight from the fused projection's float32 partial results
    ``qkv`` [parts, T, (heads + 2 kv heads) * head size]: the attention kernel sums them, norms and
    rotates its own query heads and the new key, and writes the new key and value into the cache
    (when this layer owns it).  False: the case is not this kernel's (the caller prepares q and
    calls ``attention``)."""
    if not (FUSE_QKV or force) or not (USE_TMA_DECODE or force):
        return False
    group = n_heads // n_kv_heads
    if not (batch.max_new == 1 and group <= 16 and head_dim in (64, 128, 256) and qkv.dim() == 3
            and qkv.dtype == torch.float32 and qkv.is_contiguous() and kv.k.dtype == torch.bfloat16
            and kv.k.is_contiguous() and kv.v.is_contiguous() and kv.page == 64
            and out.dtype == torch.bfloat16 and out.stride(1) == 1 and qkv.stride(0) % 4 == 0
            and qkv.shape[2] == (n_heads + 2 * n_kv_heads) * head_dim):
        return False
    if USE_TCGEN05_DECODE and not force:
        return False
    for t in (q_norm, k_norm, cos, sin):
        if t is not None and not (t.dtype == torch.float32 and t.is_contiguous() and t.data_ptr() % 16 == 0):
            return False
    L = lib(head_dim)
    n_slices = slices or decode_slices(batch.n_seqs, n_kv_heads, batch.max_after, kv.window)
    part_o = part_ml = None
    if n_slices > 1:
        part_o = rt.arena.alloc((batch.n_seqs, n_heads, n_slices, head_dim), torch.float32)
        part_ml = rt.arena.alloc((batch.n_seqs, n_heads, n_slices, 2), torch.float32)
    mk = _tc_map(("kvd", kv.k.data_ptr(), kv.k.shape[0], n_kv_heads, head_dim),
                 lambda a: L.ub_attn_map_kv(a, kv.k.data_ptr(), kv.k.shape[0], n_kv_heads))
    mv = _tc_map(("kvd", kv.v.data_ptr(), kv.v.shape[0], n_kv_heads, head_dim),
                 lambda a: L.ub_attn_map_kv(a, kv.v.data_ptr(), kv.v.shape[0], n_kv_heads))
    own = bool(kv.owner)
    rc = L.ub_attn_decode_tma_qkv(mk, mv, _ptr(qkv), qkv.shape[0], qkv.stride(0), _ptr(q_norm), _ptr(k_norm),
                                  _ptr(cos), _ptr(sin), float(eps), _ptr(kv.k) if own else None,
                                  _ptr(kv.v) if own else None, _ptr(out), out.stride(0), _ptr(batch.seq_start),
                                  _ptr(batch.seq_before), _ptr(kv.table), kv.table.shape[1], kv.ring, kv.page,
                                  batch.n_seqs, n_heads, n_kv_heads, int(kv.window or 0), float(scale), n_slices,
                                  _ptr(part_o), _ptr(part_ml), _ptr(rt.status[1:2]), _stream())
    _check(rc, "attn_decode_tma_qkv")
    return True


# The kernels take the mask as one integer: w > 0, the last w positions; w < 0, blocks of -w positions
# counted from the sequence's start (a token sees the earlier tokens of its own block); 0, everything before.
BLOCK_MASK = True
# ULTIMA_ATTN_EXTENDED=0: layers with the further options (see ``attention_ext``) stay on the any-shape kernel
EXTENDED = _os.environ.get("ULTIMA_ATTN_EXTENDED", "1") != "0"


def _mask_arg(kv, block) -> int:
    if block:
        if kv.window:
            raise KernelError("attention: a window and a block mask together are not built into these kernels")
        return -int(block)
    return int(kv.window or 0)


def attention(q, kv, out, batch, n_heads, n_kv_heads, head_dim, scale, rt, slices: int | None = None,
              kernel: str | None = None, block: int | None = None):
    """kernel: None picks (tcgen05 for prompts where it fits, mma.sync otherwise); "mma" forces the latter.
    ``block``: mask by blocks of this many positions instead of by the cache's window.  Values may have another size than
    keys: prompts on tcgen05 where the sizes fit, single tokens on mma.sync."""
    value_dim = kv.v.shape[-1]
    same = value_dim == head_dim
    mask = _mask_arg(kv, block)
    reach = block or kv.window                       # how far back a token looks at most (None: to the start)
    assert out.dtype == torch.bfloat16 and out.stride(1) == 1
    group = n_heads // n_kv_heads
    decode = batch.max_new == 1 and group <= 16
    tc_ok = (kernel != "mma" and tcgen05_fits(head_dim, n_heads, n_kv_heads, value_dim) and scale > 0 and out.stride(0) % 8 == 0
             and out.data_ptr() % 16 == 0 and kv.k.is_contiguous() and kv.v.is_contiguous())
    if tc_ok and not decode:
        return run_tcgen05(q, kv, out, batch, n_heads, n_kv_heads, head_dim, scale, rt, False, mask=mask)
    if tc_ok and same and decode and (USE_TCGEN05_DECODE or kernel == "tc"):
        n = slices or decode_slices(batch.n_seqs, n_kv_heads, batch.max_after, reach, per_sm=1)
        return run_tcgen05(q, kv, out, batch, n_heads, n_kv_heads, head_dim, scale, rt, True, n, mask=mask)
    L = lib(head_dim, value_dim)
    part_o = part_ml = None
    n_slices = 1
    tma = (same and decode and head_dim % 64 == 0 and kernel in (None, "tma") and (USE_TMA_DECODE or kernel == "tma")
           and kv.k.is_contiguous() and kv.v.is_contiguous())
    if decode:
        n_slices = slices or decode_slices(batch.n_seqs, n_kv_heads, batch.max_after, reach)
        if n_slices > 1:
            part_o = rt.arena.alloc((batch.n_seqs, n_heads, n_slices, value_dim), torch.float32)
            part_ml = rt.arena.alloc((batch.n_seqs, n_heads, n_slices, 2), torch.float32)
    if tma:
        mk = _tc_map(("kvd", kv.k.data_ptr(), kv.k.shape[0], n_kv_heads, head_dim),
                     lambda a: L.ub_attn_map_kv(a, kv.k.data_ptr(), kv.k.shape[0], n_kv_heads))
        mv = _tc_map(("kvd", kv.v.data_ptr(), kv.v.shape[0], n_kv_heads, head_dim),
                     lambda a: L.ub_attn_map_kv(a, kv.v.data_ptr(), kv.v.shape[0], n_kv_heads))
        rc = L.ub_attn_decode_tma(mk, mv, _ptr(q), q.stride(0), _ptr(out), out.stride(0), _ptr(batch.seq_start),
                                  _ptr(batch.seq_before), _ptr(kv.table), kv.table.shape[1], kv.ring, kv.page,
                                  batch.n_seqs, n_heads, n_kv_heads, mask, float(scale), n_slices,
                                  _ptr(part_o), _ptr(part_ml), _ptr(rt.status[1:2]), _stream())
        return _check(rc, "attn_decode_tma")
    rc = L.ub_attn_mma(1 if decode else 0, _ptr(q), q.stride(0), _ptr(out), out.stride(0), _ptr(kv.k), _ptr(kv.v),
                       _ptr(batch.seq_start), _ptr(batch.seq_before), _ptr(kv.table), kv.table.shape[1], kv.ring,
                       kv.page, batch.n_seqs, batch.max_new, n_heads, n_kv_heads, mask, float(scale),
                       n_slices, _ptr(part_o), _ptr(part_ml), _stream())
    _check(rc, "attn_mma")


def attention_ext(q, kv, out, batch, n_heads, n_kv_heads, head_dim, scale, rt, window=None, keep_first=0, sink=False,
                  slopes_log2=None, out_scale=1.0, gate=None, slices: int | None = None, softcap=None, dist_bias=None,
                  sink_vals=None):
    """The mma.sync kernels (prompts, and single tokens with groups of up to 16 heads) with the further options of
    the attention part: ``window`` with ``keep_first`` positions kept visible behind it, ``sink``, ``slopes_log2``
    (float32 [heads], slope * log2(e)), ``out_scale`` and ``gate`` (float32 [T, heads * head size], contiguous: one
    sigmoid gate an output element), ``softcap`` (a scaled score s becomes softcap * tanh(s / softcap)), ``dist_bias``
    (float32 [distances, heads]: the row of min(distance, rows - 1) is added behind the cap) and ``sink_vals`` (float32
    [heads]: the sink's term is exp(sink_vals[h])).  The cache holds every position or is a ring of the window's size."""
    tabled = softcap is not None or dist_bias is not None or sink_vals is not None
    if dist_bias is not None:
        assert dist_bias.dtype == torch.float32 and dist_bias.is_contiguous() and dist_bias.shape[1] == n_heads
    if sink_vals is not None:
        assert sink and sink_vals.dtype == torch.float32 and sink_vals.is_contiguous() and sink_vals.numel() == n_heads
    assert out.dtype == torch.bfloat16 and out.stride(1) == 1
    group = n_heads // n_kv_heads
    decode = batch.max_new == 1 and group <= 16
    if gate is not None:
        assert gate.dtype == torch.float32 and gate.stride(1) == 1 and gate.shape == (q.shape[0], n_heads * head_dim)
    # prompts without a window and without a bias by distance: the tcgen05 kernels know the sink, the scale and the gate
    if (not tabled and not decode and not window and not keep_first and slopes_log2 is None and tcgen05_fits(head_dim, n_heads, n_kv_heads)
            and out.stride(0) % 8 == 0 and out.data_ptr() % 16 == 0 and kv.k.is_contiguous() and kv.v.is_contiguous()
            and (gate is None or (gate.data_ptr() % 16 == 0 and gate.stride(0) % 4 == 0))):
        L = tc_lib(head_dim)
        T = q.shape[0]
        mq = _tc_map(("q", q.data_ptr(), T, n_heads, q.stride(0), group, head_dim),
                     lambda a: L.ub_attn_tc_map_q(a, q.data_ptr(), T, n_heads, q.stride(0), group))
        mk = _tc_map(("kv", kv.k.data_ptr(), kv.k.shape[0], n_kv_heads, head_dim),
                     lambda a: L.ub_attn_tc_map_kv(a, kv.k.data_ptr(), kv.k.shape[0], n_kv_heads, head_dim))
        mv = _tc_map(("kv", kv.v.data_ptr(), kv.v.shape[0], n_kv_heads, head_dim),
                     lambda a: L.ub_attn_tc_map_kv(a, kv.v.data_ptr(), kv.v.shape[0], n_kv_heads, head_dim))
        rc = L.ub_attn_tc_ext(mq, mk, mv, _ptr(out), out.stride(0), _ptr(batch.seq_start), _ptr(batch.seq_before),
                              _ptr(kv.table), kv.table.shape[1], kv.ring, kv.page, batch.n_seqs, batch.max_new, n_heads,
                              n_kv_heads, 0, float(scale), _ptr(rt.status[1:2]), 1 if sink else 0, float(out_scale),
                              _ptr(gate), gate.stride(0) if gate is not None else 0, _stream())
        return _check(rc, "attn_tc_ext")
    L = lib(head_dim)
    part_o = part_ml = None
    n_slices = 1
    if decode:
        reach = (int(window) + int(keep_first or 0)) if window else None
        n_slices = slices or decode_slices(batch.n_seqs, n_kv_heads, batch.max_after, reach)
        if n_slices > 1:
            part_o = rt.arena.alloc((batch.n_seqs, n_heads, n_slices, head_dim), torch.float32)
            part_ml = rt.arena.alloc((batch.n_seqs, n_heads, n_slices, 2), torch.float32)
    rc = L.ub_attn_mma_ext(1 if decode else 0, _ptr(q), q.stride(0), _ptr(out), out.stride(0), _ptr(kv.k), _ptr(kv.v),
                           _ptr(batch.seq_start), _ptr(batch.seq_before), _ptr(kv.table), kv.table.shape[1], kv.ring,
                           kv.page, batch.n_seqs, batch.max_new, n_heads, n_kv_heads, int(window or 0), float(scale),
                           n_slices, _ptr(part_o), _ptr(part_ml), int(keep_first or 0), 1 if sink else 0, _ptr(slopes_log2),
                           float(out_scale), _ptr(gate), gate.stride(0) if gate is not None else 0, float(softcap or 0.0),
                           _ptr(dist_bias), dist_bias.shape[0] if dist_bias is not None else 0, _ptr(sink_vals), _stream())
    _check(rc, "attn_mma_ext")
