"""What parts run on: the device, the element type of activations, scratch memory and the
choice of kernel for a matrix product or an attention call.

Parts never pick a kernel by model; they ask the runtime for "a product of these two
matrices with this epilogue" and the runtime picks by element type and shape.
"""
from __future__ import annotations

import torch

from ..kernels import ops


_ELEMENT_SIZE = {torch.float32: 4, torch.bfloat16: 2, torch.float16: 2, torch.int32: 4, torch.int64: 8,
                 torch.uint8: 1, torch.int8: 1, torch.float64: 8, torch.int16: 2, torch.bool: 1}


class Arena:
    """Scratch memory for one step: a bump allocator over one buffer, reset layer by layer.
    A request that does not fit gets a fresh, larger buffer (earlier tensors stay valid
    because they hold their buffer); that happens during warm-up only."""

    ALIGN = 256

    def __init__(self, device, nbytes: int = 1 << 20):
        self.device = device
        self._buf = torch.empty(max(nbytes, 1 << 16), dtype=torch.uint8, device=device)
        self._off = 0
        self.high_water = 0
        self._retired = []          # earlier buffers stay alive: captured graphs may point into them
        self._views = {}            # (offset, dtype, shape) -> the tensor over that place of the current buffer

    def reserve(self, nbytes: int) -> None:
        if nbytes > self._buf.numel():
            if self._off != 0:
                raise RuntimeError("arena can grow only when empty")
            self._retired.append(self._buf)
            self._views.clear()
            self._buf = torch.empty(nbytes, dtype=torch.uint8, device=self.device)

    def mark(self) -> int:
        return self._off

    def reset(self, mark: int = 0) -> None:
        self._off = mark

    def alloc(self, shape, dtype) -> torch.Tensor:
        n = 1
        for s in shape:
            n *= int(s)
        nbytes = n * _ELEMENT_SIZE[dtype]
        start = -(-self._off // self.ALIGN) * self.ALIGN
        if start + nbytes > self._buf.numel():
            size = max(2 * self._buf.numel(), start + nbytes + (1 << 20))
            self._retired.append(self._buf)
            self._views.clear()
            self._buf = torch.empty(size, dtype=torch.uint8, device=self.device)
            start = 0
        self._off = start + nbytes
        if self._off > self.high_water:
            self.high_water = self._off
        # layers reset the arena to the same mark, so the same (place, type, shape) comes again and again:
        # the tensor object made for it the first time is handed out again (making one costs microseconds)
        key = (start, dtype, tuple(shape))
        t = self._views.get(key)
        if t is None:
            if len(self._views) > 4096:
                self._views.clear()
            t = self._views[key] = self._buf[start:start + nbytes].view(dtype).view(*shape)
        return t


class Runtime:
    """dtype: torch.float32 (everything in true 32-bit: CUDA-core products, 32-bit cache) or
    torch.bfloat16 (16-bit activations, weights and cache; 32-bit residual stream, sums,
    softmax, norms and rotation)."""

    def __init__(self, device="cuda:0", dtype=torch.bfloat16, head_dims=()):
        self.device = torch.device(device)
        if dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"run dtype must be float32 or bfloat16, got {dtype}")
        self.dtype = dtype
        self.cache_dtype = dtype
        self.arena = Arena(self.device)
        self._shared: dict = {}
        self._carry: dict = {}
        self._carry_retired: list = []
        self.use_tensor_cores = dtype == torch.bfloat16
        self.launches = 0              # kernels of this library launched through the runtime
        self.pass_id = 0               # counts the passes through the layers (Model.forward); what an arrangement
                                       # keeps from layer to layer is valid within one pass only
        self.next_layer = None         # the layer that reads the stream behind the one that is running (set by Model.forward)
        # flags the kernels raise: [0] a token id outside the vocabulary, [1] a wait that ran out
        # (they are the head of a buffer whose tail takes the sampled token ids: one copy brings both)
        self.status_and_ids = torch.zeros(4 + 4096, dtype=torch.int32, device=self.device)
        self.status = self.status_and_ids[:4]
        self._status_ptr = self.status[1:2].data_ptr()

    def shared(self, key, make):
        """One object for all parts that ask with the same key (rotation tables and the like)."""
        if key not in self._shared:
            self._shared[key] = make()
        return self._shared[key]

    def carry(self, key, rows: int, cols: int, dtype):
        """A [rows, cols] array that one part of a pass fills and a later part of the same pass reads.  It lives outside the
        arena (which layers reset) at an address that stays the same from step to step, so a captured step may use it;
        when it has to grow, the old storage is kept alive for the graphs that point into it."""
        held = self._carry.get(key)
        n = int(rows) * int(cols)
        if held is None or held.dtype != dtype or held.numel() < n:
            if held is not None:
                self._carry_retired.append(held)
            held = self._carry[key] = torch.empty(max(n, 1), dtype=dtype, device=self.device)
        return held[:n].view(int(rows), int(cols))

    def check_status(self) -> None:
        """Read the flags the kernels raise (one small copy; waits for the stream)."""
        st = self.status.tolist()
        if any(st):
            self.status.zero_()
            if st[0]:
                raise RuntimeError("a token id outside the vocabulary reached the embedding kernel")
            raise RuntimeError("a wait inside a kernel ran out of time; the step's results are not valid")

    # ---- products ----------------------------------------------------------------------
    def matmul(self, a, w, out, epilogue=ops.EPI_STORE, w2=None, gate=None, unary=0, mul=None, unary_arg=0.0):
        """out (=, +=) a @ w.T with float32 accumulation; see kernels.ops for the epilogues.  ``gate`` =
        (limit, alpha, shift): the constants of a clamped gate product (tensor-core epilogues only).  ``unary``
        (ops.UNARY_*, ``unary_arg`` its constant where it has one): out = f(a @ w.T), the function taken of the float32 sums: in
        the tensor-core product's storing epilogue, elsewhere by a kernel behind the product.  ``mul`` = (gates, column step): the stored result times a sigmoid
        gate (see ``gemm_tc.mul_args``; tensor-core epilogues only)."""
        self.launches += 1
        if unary and (epilogue != ops.EPI_STORE or gate is not None):
            raise ops.KernelError("a function of the sums goes with the storing epilogue")
        if self.use_tensor_cores and a.dtype == torch.bfloat16 and w.dtype == torch.bfloat16:
            from ..kernels import gemm_tc
            if unary:
                gate = gemm_tc.unary_constants(unary, unary_arg)
            key = gemm_tc.launch_key(a, w, out, epilogue, w2, self._status_ptr, gate, mul)
            if gemm_tc.relaunch(key):
                return None
            if gemm_tc.accepts(a, w, out, epilogue, w2):
                return gemm_tc.gemm(a, w, out, epilogue, w2, self, key=key, gate=gate, mul=mul)
        if unary:
            sums = self.arena.alloc(tuple(out.shape), torch.float32)
            ops.gemm_simt(a, w, sums)
            self.launches += 1
            return ops.unary(sums, out, unary, unary_arg)
        if gate is not None or mul is not None:
            raise ops.KernelError("a clamped gate product, or a gate on the result, is an epilogue of the tensor-core product only")
        if epilogue == ops.EPI_SWIGLU_IL:
            raise ops.KernelError("the interleaved gate/up layout is for the tensor-core product only; "
                                  "this call does not fit it (operand alignment)")
        return ops.gemm_simt(a, w, out, epilogue, w2)

    def matmul_parts(self, a, w):
        """a @ w.T as a float32 [parts, T, N] whose sum over the first axis is the product (K is cut
        into slices so that a product with few tokens fills the GPU), or None when the product
        is better done whole."""
        if not (self.use_tensor_cores and a.dtype == torch.bfloat16 and w.dtype == torch.bfloat16):
            return None
        from ..kernels import gemm_tc
        T, N = a.shape[0], w.shape[0]
        parts = gemm_tc.store_splits(T, N, a.shape[1])
        if parts <= 1:
            return None
        out = self.arena.alloc((parts, T, N), torch.float32)
        if not gemm_tc.accepts(a, w, out[0], ops.EPI_STORE, None):
            return None
        self.launches += 1
        gemm_tc.gemm(a, w, out, ops.EPI_STORE, None, self, splits=parts)
        return out

    def matmul_heads(self, a, w, out, gate=None):
        """out[:, b, :] = a[:, b, :] @ w[b].T for every b (one small matrix a head): a [T, B, K], w [B, N, K], out
        [T, B, N]; a and out may be column ranges of wider rows.  ``gate`` float32 [T, B] or [T, B * N] (any row stride): the
        result times its sigmoid, a number a matrix or an element, in the tensor-core product's epilogue or behind the product
        (out is then contiguous)."""
        self.launches += 1
        if self.use_tensor_cores and a.dtype == torch.bfloat16 and w.dtype == torch.bfloat16:
            from ..kernels import gemm_tc
            if gemm_tc.accepts_batched(a, w, out):
                return gemm_tc.batched(a, w, out, self, gate=gate)
        ops.gemm_batched(a, w, out)
        if gate is not None:
            T, B, N = out.shape
            self.launches += 1
            if gate.shape[1] == B * N:
                ops.elem_gate(out.view(T, B * N), gate)
            else:
                ops.head_gate(out.view(T, B * N), gate, B, N)

    def matmul_grouped(self, a, w, out, plan, epilogue=ops.EPI_STORE, w2=None, unary=0, gate=None):
        """Sorted rows against the matrix their tile names (``plan``: a routed feed-forward's ``RoutePlan``):
        out[p] = a[plan.src_rows[p] or p] @ w[e].T, e the expert of the tile that holds sorted row p.  The tensor-core
        product takes rows that lie in the sorted order already (``plan.gather`` False); ``grouped_on_tensor_cores``
        says beforehand whether it will take a product.  ``unary`` (ops.UNARY_*): out = f(product), as in ``matmul``; ``gate`` =
        (limit, alpha, shift): the constants of a clamped gate product."""
        self.launches += 1
        if not plan.gather and self.grouped_on_tensor_cores(a, w, out, epilogue, w2):
            from ..kernels import gemm_tc
            return gemm_tc.grouped(a, w, out, plan, epilogue, w2, self, unary=unary, gate=gate)
        if unary:
            sums = self.arena.alloc(tuple(out.shape), torch.float32)
            ops.gemm_grouped(a, w, sums, plan.tiles, plan.n_tiles, plan.src_rows if plan.gather else None, plan.max_tiles,
                             epilogue, w2)
            self.launches += 1
            return ops.unary(sums, out, unary)
        return ops.gemm_grouped(a, w, out, plan.tiles, plan.n_tiles, plan.src_rows if plan.gather else None, plan.max_tiles,
                                epilogue, w2, gate=gate)

    def grouped_on_tensor_cores(self, a, w, out, epilogue=ops.EPI_STORE, w2=None) -> bool:
        if not (self.use_tensor_cores and a.dtype == torch.bfloat16 and w.dtype == torch.bfloat16):
            return False
        from ..kernels import gemm_tc
        return gemm_tc.accepts_grouped(a, w, out, epilogue, w2)

    # ---- attention ----------------------------------------------------------------------
    def attention_latent(self, q_lat, kv, batch, n_heads, row, rank, scale, window, sink_vals=None):
        """Attention of ``n_heads`` query heads [T, heads, row] over ONE key head whose rows [row] also hold the values
        (their leading ``rank`` columns); ``sink_vals`` float32 [heads]: the softmax's sum has one more term exp(sink).  Returns the heads' weighted sums as a view [T, heads, rank] (of a wider
        buffer where the kernel returns whole rows)."""
        T = q_lat.shape[0]
        q2 = q_lat.view(T, n_heads * row)
        self.launches += 1
        if self.use_tensor_cores and q_lat.dtype == torch.bfloat16:
            from ..kernels import attn_tc
            if attn_tc.accepts_latent(q_lat, kv, row, rank, n_heads, scale):
                o = self.arena.alloc((T, n_heads, rank), self.dtype)
                attn_tc.latent_attention(q_lat, kv, o, batch, n_heads, row, rank, scale, self, window=window, sink_vals=sink_vals)
                return o
            if attn_tc.accepts(q2, kv, row, n_heads, 1) and attn_tc.LATENT:
                o = self.arena.alloc((T, n_heads, row), self.dtype)
                o2 = o.view(T, n_heads * row)
                if sink_vals is not None:
                    attn_tc.attention_ext(q2, kv, o2, batch, n_heads, 1, row, scale, self, window=window, sink=True, sink_vals=sink_vals)
                else:
                    attn_tc.attention(q2, kv, o2, batch, n_heads, 1, row, scale, self, kernel="mma")
                return o[:, :, :rank]
        o = self.arena.alloc((T, n_heads, rank), self.dtype)
        ops.attn_simple(q2, kv.k, kv.k, o.view(T, n_heads * rank), batch.tok_pos, batch.tok_seq, kv.table, kv.ring, kv.page,
                        n_heads, 1, row, window, scale, v_head_dim=rank, v_row=row, sink=sink_vals is not None, sink_vals=sink_vals)
        return o

    def attention_from_qkv(self, qkv_parts, q_norm, k_norm, cos, sin, eps, kv, out, batch, n_heads, n_kv_heads,
                           head_dim, scale) -> bool:
        """Attention of a step of one token a sequence, straight from the float32 partial results of
        the fused q/k/v projection: one kernel sums them, prepares q and the new key, writes the new
        key and value and attends.  False when no kernel takes the case; the caller then prepares
        q and the cache itself and calls ``attention``."""
        if not (self.use_tensor_cores and qkv_parts is not None and batch.max_new == 1):
            return False
        from ..kernels import attn_tc
        done = attn_tc.decode_from_qkv(qkv_parts, q_norm, k_norm, cos, sin, eps, kv, out, batch, n_heads,
                                       n_kv_heads, head_dim, scale, self)
        if done:
            self.launches += 1
        return done

    def attention_fast(self, q, kv, out, batch, n_heads, n_kv_heads, head_dim, scale, block=None) -> bool:
        """The tensor-core attention kernels with a block mask (``block`` positions, counted from the
        sequence's start) or the cache's window, and values of the keys' size or another, where they take the case; False where
        they do not, and nothing was launched."""
        if not (self.use_tensor_cores and q.dtype == torch.bfloat16):
            return False
        from ..kernels import attn_tc
        if not attn_tc.accepts(q, kv, head_dim, n_heads, n_kv_heads) or not attn_tc.BLOCK_MASK \
                or not attn_tc.sizes_fit(head_dim, kv.v.shape[-1]):
            return False
        self.launches += 1
        attn_tc.attention(q, kv, out, batch, n_heads, n_kv_heads, head_dim, scale, self, block=block)
        return True

    def attention_ext(self, q, kv, out, batch, n_heads, n_kv_heads, head_dim, scale, **options) -> bool:
        """The tensor-core attention kernels with the attention part's further options (window with kept first
        positions, sink, bias by distance, output scale, a gate an element; see ``attn_tc.attention_ext``), where
        they take the case; False where they do not, and nothing was launched."""
        if not (self.use_tensor_cores and q.dtype == torch.bfloat16):
            return False
        from ..kernels import attn_tc
        if not attn_tc.accepts(q, kv, head_dim, n_heads, n_kv_heads) or not attn_tc.EXTENDED:
            return False
        self.launches += 1
        attn_tc.attention_ext(q, kv, out, batch, n_heads, n_kv_heads, head_dim, scale, self, **options)
        return True

    def attention(self, q, kv, out, batch, n_heads, n_kv_heads, head_dim, scale):
        self.launches += 1
        if self.use_tensor_cores and q.dtype == torch.bfloat16:
            from ..kernels import attn_tc
            if attn_tc.accepts(q, kv, head_dim, n_heads, n_kv_heads):
                return attn_tc.attention(q, kv, out, batch, n_heads, n_kv_heads, head_dim, scale, self)
        return ops.attn_simple(q, kv.k, kv.v, out, batch.tok_pos, batch.tok_seq, kv.table, kv.ring,
                               kv.page, n_heads, n_kv_heads, head_dim, kv.window, scale)
