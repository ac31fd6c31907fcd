"""Recurrent mixers whose state decays and takes up the token's key and value: gated linear attention and the matrix memory."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.spec import WeightSpec
from .base import Mixer, StateNeed, register_part


class _DecayedState(Mixer):
    """What the two share: for each head a matrix S [D, E] in float32, zero at a sequence's start, that a token decays and to
    which it adds k v^T; o = S^T q.  The projections of the mixer's input are ONE product [q | k | v | gate | ...] with float32
    sums; everything between it and the output projection is float32 (csrc/linear.cu).  A step of one token a sequence is one
    kernel between the two products, which takes the first one's K slices as they are; a longer one runs the recurrence with
    long sequences cut into chunks that are worked on side by side."""

    graph_safe = True
    silu_gate = False

    def __init__(self, width, n_heads, head_dim, v_head_dim, eps, out_scale=1.0):
        self.width, self.nh, self.hd, self.hdv = int(width), int(n_heads), int(head_dim), int(v_head_dim)
        self.eps, self.out_scale = float(eps), float(out_scale)
        self.q_scale = self.hd ** -0.5
        self.qk_width, self.v_width = self.nh * self.hd, self.nh * self.hdv
        if self.hd > 256 or self.hdv > 1024:
            raise ValueError(f"{self.kind}: key size {self.hd} or value size {self.hdv} is more than the kernels take (256, 1024)")

    def _projection_specs(self):
        W = WeightSpec
        return [W("q_proj.weight", (self.qk_width, self.width)), W("k_proj.weight", (self.qk_width, self.width)),
                W("v_proj.weight", (self.v_width, self.width)), W("gate_proj.weight", (self.v_width, self.width))]

    def kernel_needs(self, run_dtype):
        return [("linear.cu", ())]

    def _bind_input(self, tensors, names):
        """Stack the projections, padded with zero rows to a multiple of 8 (so that rows of sums start aligned); the columns where
        each of them starts."""
        ws = [tensors[n + ".weight"] for n in names]
        if len({w.dtype for w in ws}) != 1:
            raise ValueError(f"{self.kind}: the projections must share one element type")
        offs, at = [], 0
        for w in ws:
            offs.append(at)
            at += w.shape[0]
        if at % 8:
            ws.append(torch.zeros((8 - at % 8, self.width), dtype=ws[0].dtype, device=ws[0].device))
        self.w_in = torch.cat(ws, dim=0).contiguous()
        self.wo = tensors["o_proj.weight"].contiguous()
        self.o_norm = tensors["o_norm.weight"].float().contiguous()
        return offs

    def input_weight(self):
        return self.w_in

    def adopt_input_weight(self, w):
        self.w_in = w

    # what the two forms differ in
    def _step_options(self) -> dict:
        raise NotImplementedError

    def _prepare(self, p, T, states, batch, rt):
        """(decays or keep, put or None, floor or None) of a step's tokens."""
        raise NotImplementedError

    def forward(self, h, residual, batch, cache, rt, projected=None):
        T, f32, form = h.shape[0], torch.float32, self.form
        states = cache.states
        one_each = batch.max_new == 1 and batch.n_seqs == T
        p = projected if projected is not None else (rt.matmul_parts(h, self.w_in) if one_each else None)
        if p is None:
            p = rt.arena.alloc((T, self.w_in.shape[0]), f32)
            rt.matmul(h, self.w_in, p)
        elif p.dim() == 3 and not one_each:
            p = p.sum(0)                          # (an arrangement's product in K slices, for a few tokens of one sequence)
        oa = rt.arena.alloc((T, self.v_width), rt.dtype)
        if one_each:
            rt.launches += 1
            ops.lin_step(p, form, states, batch, self.o_norm, oa, self.q_scale, self.eps, self.out_scale, self.silu_gate,
                         **self._step_options())
        else:
            dec, put, floor = self._prepare(p, T, states, batch, rt)
            ew = self.hdv + (1 if form.head_form else 0)
            o = rt.arena.alloc((T, self.nh, ew), f32)
            chunks = ops.lin_chunks(form, batch.n_seqs, batch.max_new)
            work = decay = None
            if chunks[0] > 1:
                work = rt.arena.alloc((chunks[0], batch.n_seqs, self.nh, self.hd, ew), f32)
                decay = rt.arena.alloc((chunks[0], batch.n_seqs, self.nh, 1 if form.head_form else self.hd), f32)
            rt.launches += 2 + (2 if chunks[0] > 1 else 0)
            ops.lin_scan(p, form, dec, put, o, states[0], states[1] if form.head_form else None, batch, work, decay, chunks)
            ops.lin_finish(o, p, form, floor, self.o_norm, oa, self.q_scale, self.eps, self.out_scale, self.silu_gate)
        rt.matmul(oa, self.wo, residual, ops.EPI_ADD)


@register_part("mixer", "gated_linear")
class GatedLinear(_DecayedState):
    """Gated linear attention: S <- diag(a) S + k v^T, o = S^T q / sqrt(D), with one decay a head and key channel,
    a = sigmoid(decay_up(decay_down h) + decay_bias)^(1 / tau).  Each head's o passes an RMS norm over E with a weight the heads
    share, the heads side by side are multiplied by silu(gate_proj h) and go through the output projection.  ``out_scale``: a
    constant on what goes into it."""

    silu_gate = True

    def __init__(self, width: int, n_heads: int, head_dim: int, v_head_dim: int, decay_rank: int, tau: float, eps: float,
                 out_scale: float = 1.0):
        super().__init__(width, n_heads, head_dim, v_head_dim, eps, out_scale)
        self.rank, self.tau = int(decay_rank), float(tau)
        if not (1 <= self.rank <= 512):
            raise ValueError(f"gated_linear: a decay map of rank {self.rank} is not one the kernels take (1 to 512)")
        if not self.tau > 0:
            raise ValueError("gated_linear: tau must be positive")

    def weight_specs(self):
        W, V = WeightSpec, "vector"
        return self._projection_specs() + [
            W("decay_down.weight", (self.rank, self.width)), W("decay_up.weight", (self.qk_width, self.rank), "matrix", ("normal", 0.3)),
            W("decay_bias", (self.qk_width,), V, ("normal", 0.5)), W("o_norm.weight", (self.hdv,), V, ("one_plus_normal", 0.05)),
            W("o_proj.weight", (self.width, self.v_width))]

    def cache_need(self):
        return StateNeed((self.nh, self.hd, self.hdv), "float32")

    def bind(self, tensors, rt):
        q, k, v, g, a = self._bind_input(tensors, ("q_proj", "k_proj", "v_proj", "gate_proj", "decay_down"))
        self.up = tensors["decay_up.weight"].float().t().contiguous()               # [rank, H * D]
        self.decay_bias = tensors["decay_bias"].float().contiguous()
        self.form = ops.LinForm(self.nh, self.hd, self.hdv, (q, k, v, g, a, 0), rank=self.rank)

    def _step_options(self):
        return {"decay": (self.up, self.decay_bias, self.tau)}

    def _prepare(self, p, T, states, batch, rt):
        dec = rt.arena.alloc((T, self.qk_width), torch.float32)
        rt.launches += 1
        ops.lin_decay(p, self.form, self.up, self.decay_bias, dec, self.tau)
        return dec, None, None


@register_part("mixer", "matrix_memory")
class MatrixMemory(_DecayedState):
    """A matrix memory with exponential gates: for each head log gates i = c tanh((i_proj h + i_bias) / c) and
    f = logsigmoid(c tanh((f_proj h + f_bias) / c)), c = ``gate_cap``, and with a running maximum m (0 at a sequence's start)

        m' = max(f + m, i);   S <- exp(f + m - m') S + exp(i - m') k v^T;   n <- exp(f + m - m') n + exp(i - m') k
        o = S^T q / (max(|n . q|, exp(-m')) + 1e-6),     q scaled by D^-1/2

    Each head's o is divided by its root mean square (``eps``); the heads side by side are multiplied by a weight of all heads'
    size and by sigmoid(gate_proj h), and go through the output projection.  S, n and m are the sequence's state."""

    def __init__(self, width: int, n_heads: int, head_dim: int, v_head_dim: int, gate_cap: float, eps: float, out_scale: float = 1.0):
        super().__init__(width, n_heads, head_dim, v_head_dim, eps, out_scale)
        self.cap = float(gate_cap)
        if not self.cap > 0:
            raise ValueError("matrix_memory: the gates' cap must be positive")

    def weight_specs(self):
        W, V = WeightSpec, "vector"
        return self._projection_specs() + [
            W("i_proj.weight", (self.nh, self.width), "matrix", ("normal", 0.1)), W("i_bias", (self.nh,), V, ("normal", 1.0)),
            W("f_proj.weight", (self.nh, self.width), "matrix", ("normal", 0.1)), W("f_bias", (self.nh,), V, ("normal", 2.0)),
            W("o_norm.weight", (self.v_width,), V, ("one_plus_normal", 0.05)), W("o_proj.weight", (self.width, self.v_width))]

    def cache_need(self):
        return (StateNeed((self.nh, self.hd, self.hdv), "float32"), StateNeed((self.nh, self.hd), "float32"),
                StateNeed((self.nh,), "float32"))

    def bind(self, tensors, rt):
        offs = self._bind_input(tensors, ("q_proj", "k_proj", "v_proj", "gate_proj", "i_proj", "f_proj"))
        self.i_bias = tensors["i_bias"].float().contiguous()
        self.f_bias = tensors["f_bias"].float().contiguous()
        self.form = ops.LinForm(self.nh, self.hd, self.hdv, offs, head_form=True)

    def _step_options(self):
        return {"gates": (self.i_bias, self.f_bias, self.cap)}

    def _prepare(self, p, T, states, batch, rt):
        keep, put, floor = (rt.arena.alloc((T, self.nh), torch.float32) for _ in range(3))
        rt.launches += 1
        ops.lin_gates(p, self.form, self.i_bias, self.f_bias, self.cap, states[2], batch, keep, put, floor)
        return keep, put, floor
