"""Two mixers side by side."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.spec import WeightSpec
from .base import KVNeed, Mixer, PartSpec, StateNeed, build_part, register_part


@register_part("mixer", "side_by_side")
class SideBySide(Mixer):
    """left_scale * left(h) + right_scale * right(h): two mixers of any kind read the same input and add
    into the same stream.  Each applies its scale itself (its ``out_scale`` parameter, a constant on what
    goes into its output projection), so no buffer lies between them and the stream.  The tensors of the
    two stand under ``left.`` and ``right.``.  The run's cache is shared out: keys and values to the one
    that asks for them (at most one may), states in the order left, right.

    ``norm_outputs`` (an eps): left_scale * norm_l(left(h)) + right_scale * norm_r(right(h)), each side's result through an RMS
    norm over the width with a weight of its own (tensors ``left_out.weight``, ``right_out.weight``) first.  The two results then
    lie in buffers of their own, and ONE kernel norms, scales and adds them; an arrangement that norms the mixer's
    output takes the two buffers (``forward_apart``) and has that kernel apply its norm too."""

    def __init__(self, left: PartSpec, right: PartSpec, left_scale: float = 1.0, right_scale: float = 1.0,
                 norm_outputs: float | None = None):
        self.norm_eps = float(norm_outputs) if norm_outputs is not None else None
        self.scales = (float(left_scale), float(right_scale))
        def side(ps, scale):
            own = 1.0 if self.norm_eps is not None else float(scale)          # behind a norm the scale is the joining kernel's
            return build_part("mixer", PartSpec(ps.kind, tuple(sorted({**ps.as_dict(), "out_scale": own}.items()))))
        self.left, self.right = side(left, left_scale), side(right, right_scale)
        self.out_w = None
        self._stack = None
        self._needs = [self._list(self.left.cache_need()), self._list(self.right.cache_need())]
        if sum(isinstance(n, KVNeed) for ns in self._needs for n in ns) > 1:
            raise ValueError("side_by_side: at most one of the two mixers may keep keys and values")

    @staticmethod
    def _list(need):
        if need is None:
            return []
        return list(need) if isinstance(need, tuple) else [need]

    @property
    def graph_safe(self) -> bool:
        return bool(self.left.graph_safe and self.right.graph_safe)

    def weight_specs(self):
        s = [WeightSpec(side + s.name, s.shape, s.kind, s.init)
             for side, m in (("left.", self.left), ("right.", self.right)) for s in m.weight_specs()]
        if self.norm_eps is not None:
            s += [WeightSpec(f"{side}_out.weight", (m.width,), "vector", ("one_plus_normal", 0.05))
                  for side, m in (("left", self.left), ("right", self.right))]
        return s

    def cache_need(self):
        needs = tuple(n for ns in self._needs for n in ns)
        return needs or None

    def kernel_needs(self, run_dtype):
        return (list(self.left.kernel_needs(run_dtype)) + list(self.right.kernel_needs(run_dtype))
                + ([("rowwise.cu", ())] if self.norm_eps is not None else []))

    def bind(self, tensors, rt):
        for side, m in (("left.", self.left), ("right.", self.right)):
            m.bind({n[len(side):]: t for n, t in tensors.items() if n.startswith(side)}, rt)
        if self.norm_eps is not None:
            self.out_w = tuple(tensors[f"{side}_out.weight"].float().contiguous() for side in ("left", "right"))
            # both sides read the same input: one product for everything of it whose float32 sums they take
            w = self._both_inputs()
            if w is not None:
                self.adopt_input_weight(w)
                self._stack = w

    def input_weight(self):
        """Both sides' input matrices stacked, if both have one (with ``norm_outputs`` the product is this part's own)."""
        return None if self.norm_eps is not None else self._both_inputs()

    def _both_inputs(self):
        a, b = self.left.input_weight(), self.right.input_weight()
        if a is None or b is None or a.dtype != b.dtype or a.shape[1] != b.shape[1]:
            return None
        return torch.cat([a, b], dim=0)

    def adopt_input_weight(self, w):
        n = self.left.input_weight().shape[0]
        self.left.adopt_input_weight(w[:n])
        self.right.adopt_input_weight(w[n:])

    def _share(self, cache, which: int):
        """The part of the run's cache that belongs to one side."""
        if cache is None:
            return None
        before = sum(isinstance(n, StateNeed) for n in self._needs[0]) if which == 1 else 0
        mine = sum(isinstance(n, StateNeed) for n in self._needs[which])
        states = tuple(cache.states[before:before + mine])
        kv = cache.kv if any(isinstance(n, KVNeed) for n in self._needs[which]) else None
        return type(cache)(kv=kv, state=states[0] if states else None, owner=cache.owner, states=states)

    @property
    def apart(self) -> bool:
        """True: ``forward_apart`` leaves the two sides' results in two buffers."""
        return self.norm_eps is not None

    def forward_apart(self, h, y, y2, batch, cache, rt):
        """The two sides' results, not normed, added into y and y2 (cleared float32 [T, width])."""
        mark = rt.arena.mark()
        sums = None
        if self._stack is not None:
            # (a step of one token a sequence takes the product's K slices as they are; longer ones want whole sums)
            sums = rt.matmul_parts(h, self._stack) if batch.max_new == 1 and batch.n_seqs == h.shape[0] else None
            if sums is None:
                sums = rt.arena.alloc((h.shape[0], self._stack.shape[0]), torch.float32)
                rt.matmul(h, self._stack, sums)
        inner = rt.arena.mark()
        n = self.left.input_weight().shape[0] if sums is not None else 0
        for m, buf, which, cols in ((self.left, y, 0, slice(0, n)), (self.right, y2, 1, slice(n, None))):
            if sums is not None:
                m.forward(h, buf, batch, self._share(cache, which), rt, projected=sums[..., cols])
            else:
                m.forward(h, buf, batch, self._share(cache, which), rt)
            rt.arena.reset(inner)
        rt.arena.reset(mark)

    def join(self, y, y2, x, rt, after=None, h=None):
        """x += f(left_scale * norm_l(y) + right_scale * norm_r(y2)), both cleared; f: ``after`` = (weight, eps) of one more RMS norm,
        or nothing.  ``h`` receives the new x in its own type."""
        rt.launches += 1
        ops.norm_join_two(y, y2, x, self.out_w, self.scales, self.norm_eps, after=after, out=h)

    def forward(self, h, residual, batch, cache, rt, projected=None):
        mark = rt.arena.mark()
        if self.norm_eps is not None:
            y, y2 = (rt.arena.alloc(tuple(residual.shape), residual.dtype) for _ in range(2))
            y.zero_()
            y2.zero_()
            self.forward_apart(h, y, y2, batch, cache, rt)
            self.join(y, y2, residual, rt)
            rt.arena.reset(mark)
            return
        if projected is not None:
            n = self.left.input_weight().shape[0]
            self.left.forward(h, residual, batch, self._share(cache, 0), rt, projected=projected[..., :n])
            rt.arena.reset(mark)
            self.right.forward(h, residual, batch, self._share(cache, 1), rt, projected=projected[..., n:])
        else:
            self.left.forward(h, residual, batch, self._share(cache, 0), rt)
            rt.arena.reset(mark)
            self.right.forward(h, residual, batch, self._share(cache, 1), rt)
        rt.arena.reset(mark)
