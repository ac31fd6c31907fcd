"""The latent-attention mixer: keys and values kept as one small vector a position."""
from __future__ import annotations

import math

import torch

from ..kernels import ops
from ..weights.spec import WeightSpec
from .base import Mixer, KVNeed, register_part


@register_part("mixer", "latent_attention")
class LatentAttention(Mixer):
    """Every position keeps c = rms_norm(W_dkv h [:rank]) (weight ``kv_norm``, the layer's eps) and one rotated key
    part k_r = rotate(W_dkv h [rank:]) of ``rot_dim`` numbers that all heads share; nothing else is cached.  Head h of
    ``n_heads`` has a query [q_u (``head_dim`` numbers) | q_r (``rot_dim``, rotated)], the unrotated key W_uk[h] c and
    the value W_uv[h] c (``v_head_dim`` numbers); the score is (q_u . W_uk[h] c + q_r . k_r) * scale, the softmax
    ordinary, the window optional.  The rotation turns the pairs (2i, 2i + 1) of the first ``rotary_dim`` columns of a
    rotated part; its frequencies theta^(-2i/rotary_dim) may be rescaled (``yarn`` = (factor, original, fast, slow):
    with p(t) = rotary_dim ln(original / (2 pi t)) / (2 ln theta), lo = max(floor(p(fast)), 0), hi = min(ceil(p(slow)),
    rotary_dim - 1) and ramp_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1), frequency i becomes
    f_i / factor * ramp_i + f_i (1 - ramp_i), and cos and sin are multiplied by 0.1 ln(factor) + 1).

    Further parameters, each off by default:
      rot_dim = 0   no rotated part: queries and keys carry no positions (theta, rotary_dim, max_positions then stand idle)
      pairing       "halves": the pairs are (i, i + rotary_dim / 2) instead of neighbours.  The rows of the query and key
                    matrices are then held in the order that makes them neighbours: every score is the same sum in
                    another order
      q_rank        queries through a latent of their own: q = W_uq rms_norm(W_dq h) (tensors ``q_down.weight``,
                    ``q_down_norm.weight``, ``q_up.weight`` instead of ``q_proj.weight``)
      learned_sink  the softmax's sum has one more term exp(sink[h]) without key and value (tensor ``sink`` [heads])
      gate          "head": head h's output is multiplied by sigmoid(W_g h)_h; "element": the heads' outputs by
                    sigmoid(W_g h) element by element (tensor ``gate_proj.weight``)

    The attention runs in the latent space: q' = W_uk[h]^T q_u (``rank`` numbers) meets c directly, so all heads read
    ONE key row [c | k_r] a position and the weighted sum of the c goes through W_uv[h] afterwards.  Launches: one
    product [q | dkv | gate] with float32 sums (or [dq | dkv | gate], the placement kernel, then the product W_uq), the
    placement kernel (norm, rotation, cache row, query parts; without a rotated part W_uq writes the query parts itself),
    the heads' W_uk^T products as one batched product, attention over one key head whose values are the leading columns
    of the key rows, the heads' W_uv products as one batched product (the gate in its epilogue), the output product into
    the stream."""

    graph_safe = True

    def __init__(self, width: int, n_heads: int, head_dim: int, rot_dim: int, v_head_dim: int, rank: int, scale: float,
                 eps: float, theta: float = 0.0, rotary_dim: int = 0, max_positions: int = 0, window: int | None = None,
                 yarn: tuple | None = None, pairing: str = "neighbours", q_rank: int | None = None, learned_sink: bool = False,
                 gate: str | None = None):
        self.width, self.nh, self.hd, self.rot = int(width), int(n_heads), int(head_dim), int(rot_dim)
        self.hdv, self.rank, self.scale, self.eps = int(v_head_dim), int(rank), float(scale), float(eps)
        self.theta, self.rd, self.max_positions = float(theta), int(rotary_dim), int(max_positions)
        self.window = int(window) if window else None
        self.yarn = tuple(float(v) for v in yarn) if yarn else None
        self.row = self.rank + self.rot                    # a position's key row
        self.pairing, self.q_rank = str(pairing), int(q_rank) if q_rank else None
        self.learned_sink, self.gate = bool(learned_sink), gate
        if self.pairing not in ("neighbours", "halves") or gate not in (None, "head", "element"):
            raise ValueError("latent_attention: pairing is 'neighbours' or 'halves', gate None, 'head' or 'element'")
        if self.rot and (self.rd % 2 or not (2 <= self.rd <= self.rot)):
            raise ValueError(f"latent_attention: rotary size {self.rd} must be even and at most the rotated part {self.rot}")
        if self.row > 1024 or self.rank > 512:
            raise ValueError(f"latent_attention: a key row of {self.row} numbers (latent {self.rank}) is more than the "
                             f"attention kernels take (1,024 and 512)")
        self.gate_width = {None: 0, "head": self.nh, "element": self.nh * self.hdv}[gate]

    def weight_specs(self):
        W = WeightSpec
        q_rows = self.nh * (self.hd + self.rot)
        if self.q_rank:
            s = [W("q_down.weight", (self.q_rank, self.width)),
                 W("q_down_norm.weight", (self.q_rank,), "vector", ("one_plus_normal", 0.05)),
                 W("q_up.weight", (q_rows, self.q_rank), "matrix", ("normal", 0.08))]
        else:
            s = [W("q_proj.weight", (q_rows, self.width))]
        s += [W("kv_down.weight", (self.row, self.width)),
              W("kv_norm.weight", (self.rank,), "vector", ("one_plus_normal", 0.05)),
              W("k_up.weight", (self.nh * self.hd, self.rank), "matrix", ("normal", 0.08)),
              W("v_up.weight", (self.nh * self.hdv, self.rank), "matrix", ("normal", 0.08)),
              W("o_proj.weight", (self.width, self.nh * self.hdv))]
        if self.gate:
            s.append(W("gate_proj.weight", (self.gate_width, self.width)))
        if self.learned_sink:
            s.append(W("sink", (self.nh,), "vector", ("normal", 1.0)))
        return s

    def cache_need(self):
        return KVNeed(1, self.row, self.window, values_in_keys=True)

    def kernel_needs(self, run_dtype):
        from ..kernels import attn_tc
        out = [("latent.cu", ()), ("attn_simple.cu", ())]
        if run_dtype == torch.bfloat16:
            out += attn_tc.latent_needs(self.row, self.rank, self.nh)
        return out

    def frequencies(self):
        """(frequency of every pair, amplitude of cos and sin), float64."""
        half = self.rd // 2
        i = torch.arange(half, dtype=torch.float64)
        f = torch.pow(torch.tensor(self.theta, dtype=torch.float64), -2.0 * i / self.rd)
        amp = 1.0
        if self.yarn is not None:
            factor, original, fast, slow = self.yarn

            def where(t):
                return self.rd * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(self.theta))
            lo = max(math.floor(where(fast)), 0)
            hi = min(math.ceil(where(slow)), self.rd - 1)
            ramp = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
            f = f / factor * ramp + f * (1.0 - ramp)
            amp = 0.1 * math.log(factor) + 1.0
        return f, amp

    def _neighbours(self, w, parts: int):
        """The rows of ``w`` ([parts, rows a part] of which the last ``rot`` are a rotated part) with the rotated part's pairs
        next to each other."""
        if self.pairing == "neighbours" or not self.rot:
            return w
        half = self.rd // 2
        n = w.shape[0] // parts
        order = torch.arange(n)
        first = n - self.rot
        order[first:first + self.rd] = first + torch.stack([torch.arange(half), torch.arange(half) + half], dim=1).flatten()
        return w.view(parts, n, w.shape[1])[:, order.to(w.device)].reshape(w.shape).contiguous()

    def bind(self, tensors, rt):
        wq = tensors["q_down.weight"] if self.q_rank else self._neighbours(tensors["q_proj.weight"], self.nh)
        ws = [wq, self._neighbours(tensors["kv_down.weight"], 1)]
        if self.gate:
            ws.append(tensors["gate_proj.weight"])
        if len({w.dtype for w in ws}) != 1:
            raise ValueError("latent_attention: the projections must share one element type")
        self.w_in = torch.cat(ws, dim=0).contiguous()
        self.c_off = wq.shape[0]
        self.g_off = self.c_off + self.row
        if self.q_rank:
            self.w_uq = self._neighbours(tensors["q_up.weight"], self.nh)
            self.q_norm = tensors["q_down_norm.weight"].float().contiguous()
        self.kv_norm = tensors["kv_norm.weight"].float().contiguous()
        # a head's W_uk as the matrix its query part meets: [rank, head size]; W_uv as stored: [value size, rank]
        self.k_up_t = tensors["k_up.weight"].view(self.nh, self.hd, self.rank).transpose(1, 2).contiguous()
        self.v_up = tensors["v_up.weight"].view(self.nh, self.hdv, self.rank).contiguous()
        self.wo = tensors["o_proj.weight"].contiguous()
        self.sink_vals = tensors["sink"].float().contiguous() if self.learned_sink else None
        self.cos = self.sin = None
        if not self.rot:
            return
        key = ("latent_rotary", self.rd, self.theta, self.max_positions, self.yarn)

        def make():
            f, amp = self.frequencies()
            ang = torch.arange(self.max_positions, dtype=torch.float64)[:, None] * f[None, :]
            return ((torch.cos(ang) * amp).float().contiguous().to(rt.device),
                    (torch.sin(ang) * amp).float().contiguous().to(rt.device))
        self.cos, self.sin = rt.shared(key, make)

    def _project(self, a, w, T, rt):
        """a @ w.T with float32 sums: [parts, T, N] (few tokens: K in slices, summed by the placement kernel) or [T, N]."""
        x = rt.matmul_parts(a, w)
        if x is None:
            x = rt.arena.alloc((T, w.shape[0]), torch.float32)
            rt.matmul(a, w, x)
        return x

    def forward(self, h, residual, batch, cache, rt):
        T = h.shape[0]
        kv = cache.kv
        x = self._project(h, self.w_in, T, rt)
        q_plain = rt.arena.alloc((T, self.nh, self.hd), rt.dtype)
        q_lat = rt.arena.alloc((T, self.nh, self.row), rt.dtype)
        rotation = dict(cos=self.cos, sin=self.sin, rotary_dim=self.rd, tok_pos=batch.tok_pos)
        latent = dict(c_off=self.c_off, c_weight=self.kv_norm, k_cache=kv.k, table=kv.table, ring=kv.ring, page=kv.page,
                      tok_seq=batch.tok_seq, rank=self.rank, rot=self.rot, eps=self.eps)
        queries = dict(q_off=0, q_plain=q_plain, q_lat=q_lat, n_heads=self.nh, dim=self.hd)
        gate, gates = None, {}
        if self.gate and x.dim() == 3:
            gate = rt.arena.alloc((T, self.gate_width), torch.float32)
            gates = dict(g_off=self.g_off, gate_out=gate)
        elif self.gate:
            gate = x[:, self.g_off:]                       # read where the product put it
        rt.launches += 1
        if self.q_rank:
            c_q = rt.arena.alloc((T, self.q_rank), rt.dtype)
            ops.latent_place(x, **latent, **rotation, **gates, dq_off=0, dq_weight=self.q_norm, dq_out=c_q)
            if self.rot:
                xq = self._project(c_q, self.w_uq, T, rt)
                rt.launches += 1
                ops.latent_place(xq, **queries, **rotation, rank=self.rank, rot=self.rot)
            else:
                rt.matmul(c_q, self.w_uq, q_plain.view(T, self.nh * self.hd))
        else:
            ops.latent_place(x, **latent, **rotation, **gates, **queries)
        rt.matmul_heads(q_plain, self.k_up_t, q_lat[:, :, :self.rank])
        o_lat = rt.attention_latent(q_lat, kv, batch, self.nh, self.row, self.rank, self.scale, self.window, sink_vals=self.sink_vals)
        o = rt.arena.alloc((T, self.nh, self.hdv), rt.dtype)
        rt.matmul_heads(o_lat, self.v_up, o, gate=gate)
        rt.matmul(o.view(T, self.nh * self.hdv), self.wo, residual, ops.EPI_ADD)
