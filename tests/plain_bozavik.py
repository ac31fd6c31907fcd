"""A plain, slow implementation of the Bozavik design: one function for each mechanism, on whole-sequence matrices, on
the CPU.  It shares no code with the package: it takes config.json's dictionary and a dictionary of tensors by their
stored names.

``dt`` is the type everything is computed in (float64 for an oracle).  Nothing here keeps a cache: a sequence is always
run whole, and keys and values are formed head by head from the latent (no product is moved from one side of a score to
the other).
"""
from __future__ import annotations

import math

import torch

ALPHA = 1.702                               # steepness of an expert's gate


# ---------------------------------------------------------------------------------------
# norms
# ---------------------------------------------------------------------------------------
def layer_norm(x, w, b, eps):
    """Mean taken off, divided by the root of the mean squared deviation (+ eps), weight and bias."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


# ---------------------------------------------------------------------------------------
# rotation, mask, softmax
# ---------------------------------------------------------------------------------------
def rotate_halves(x, positions, base, dims):
    """x [T, ..., n]: of its first ``dims`` columns, column i and column i + dims/2 turn by position * base^(-2i/dims);
    the columns from ``dims`` on pass."""
    half = dims // 2
    f = torch.tensor(float(base), dtype=x.dtype) ** (-2.0 * torch.arange(half, dtype=x.dtype) / dims)
    a = positions.to(x.dtype)[:, None] * f[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [half]
    c, s = torch.cos(a).view(shape), torch.sin(a).view(shape)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def causal(T):
    i = torch.arange(T)
    return i[None, :] <= i[:, None]


def softmax_over_visible(scores, seen, sink=None):
    """Weights over the visible keys, scores [H, T, T]; ``sink`` [H]: the denominator has one more term exp(sink_h)."""
    s = scores.masked_fill(~seen[None], -math.inf)
    m = s.max(-1, keepdim=True).values
    if sink is not None:
        m = torch.maximum(m, sink[:, None, None])
    e = torch.exp(s - m)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink[:, None, None] - m)
    return e / den


# ---------------------------------------------------------------------------------------
# the two mixers
# ---------------------------------------------------------------------------------------
def latent_queries(h, W, eps, pre):
    """Queries through a latent of their own: up(rms_norm(down h))."""
    return rms_norm(h @ W[pre + "dq"].T, W[pre + "dq.norm"], eps) @ W[pre + "uq"].T


def heads_from_latent(c, w, H):
    """c [T, rank], w [H * n, rank] -> [T, H, n]."""
    return (c @ w.T).view(c.shape[0], H, -1)


def latent_attention_without_positions(h, W, m, eps, pre):
    T, H = h.shape[0], m["heads"]
    q = latent_queries(h, W, eps, pre).view(T, H, m["dim"])
    c = rms_norm(h @ W[pre + "dkv"].T, W[pre + "dkv.norm"], eps)
    k, v = heads_from_latent(c, W[pre + "uk"], H), heads_from_latent(c, W[pre + "uv"], H)
    p = softmax_over_visible(torch.einsum("ihd,jhd->hij", q, k) * m["scale"], causal(T), W[pre + "sink"])
    o = torch.einsum("hij,jhe->ihe", p, v).reshape(T, H * m["vdim"])
    return (o * torch.sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T              # a gate an output element


def latent_attention_with_rotated_part(h, W, m, eps, pre):
    T, H, d, rank = h.shape[0], m["heads"], m["dim"], m["kv_rank"]
    pos = torch.arange(T)
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = latent_queries(h, W, eps, pre).view(T, H, d + m["rot_dim"])
    q_plain, q_rot = q[..., :d], rotate_halves(q[..., d:], pos, base, dims)
    low = h @ W[pre + "dkv"].T
    c = rms_norm(low[:, :rank], W[pre + "dkv.norm"], eps)
    k_rot = rotate_halves(low[:, rank:], pos, base, dims)                        # one for all heads, not normed
    k, v = heads_from_latent(c, W[pre + "uk"], H), heads_from_latent(c, W[pre + "uv"], H)
    s = (torch.einsum("ihd,jhd->hij", q_plain, k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * m["scale"]
    p = softmax_over_visible(s, causal(T))
    o = torch.einsum("hij,jhe->ihe", p, v)
    o = o * torch.sigmoid(h @ W[pre + "g"].T)[:, :, None]                        # a gate a head
    return o.reshape(T, H * m["vdim"]) @ W[pre + "o"].T


MIXERS = {"latent_attention": latent_attention_without_positions, "latent_attention_2": latent_attention_with_rotated_part}


# ---------------------------------------------------------------------------------------
# the feed-forward
# ---------------------------------------------------------------------------------------
def clamped_expert(h, W, limit, pre):
    g = torch.clamp(h @ W[pre + "gate"].T, max=limit)
    u = torch.clamp(h @ W[pre + "up"].T, -limit, limit)
    return (g * torch.sigmoid(ALPHA * g) * (u + 1)) @ W[pre + "down"].T


def route(h, W, top, pre):
    """The chosen experts of every token and their weights, [T, top] each: softmax over the chosen logits only."""
    best = torch.topk(h @ W[pre + "router"].T, top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def routed_feed_forward(h, W, f, pre):
    idx, w = route(h, W, f["router"]["top"], pre)
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, k = torch.nonzero(idx == e, as_tuple=True)
        if t.numel():
            out.index_add_(0, t, w[t, k][:, None] * clamped_expert(h[t], W, f["expert"]["limit"], f"{pre}e{e}."))
    if f.get("shared"):
        out = out + torch.sigmoid(h @ W[pre + "shared.sg"].T) * clamped_expert(h, W, f["shared"]["limit"], pre + "shared.")
    return out


# ---------------------------------------------------------------------------------------
# layers and the model
# ---------------------------------------------------------------------------------------
def sublayer(x, W, pre, n, eps, mult, f):
    """x + mult * norm_after(f(norm_before(x)))."""
    a, b = f"{pre}norm{n}", f"{pre}norm{n}b"
    return x + mult * layer_norm(f(layer_norm(x, W[a], W[a + ".b"], eps)), W[b], W[b + ".b"], eps)


def forward(cfg, W, tokens, dt=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out``: a list that receives the residual stream after every layer."""
    W = {n: (t.to(dt) if t.is_floating_point() else t) for n, t in W.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, L in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = sublayer(x, W, pre, 1, eps, mult, lambda h: MIXERS[L["type"]](h, W, L["mixer"], eps, pre + "mix."))
        if L.get("mlp"):
            x = sublayer(x, W, pre, 2, eps, mult, lambda h: routed_feed_forward(h, W, L["mlp"], pre + "mlp."))
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["head"].T


def read_folder(model_dir: str):
    """(config.json's dictionary, stored name -> float64 tensor) read with nothing but the file format."""
    import json
    import os
    import struct

    import numpy as np
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(model_dir, "model.safetensors"), "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        data = f.read()
    header.pop("__metadata__", None)
    W = {}
    for name, e in header.items():
        raw = data[e["data_offsets"][0]:e["data_offsets"][1]]
        if e["dtype"] == "BF16":
            a = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32)
        elif e["dtype"] == "F32":
            a = np.frombuffer(raw, dtype="<f4")
        else:
            raise ValueError(f"plain reader: dtype {e['dtype']} of {name}")
        W[name] = torch.from_numpy(a.astype(np.float64).reshape(e["shape"]))
    return cfg, W


def logits(cfg, W, tokens):
    """float64 numpy [T, vocab]."""
    with torch.no_grad():
        return forward(cfg, W, tokens, torch.float64).numpy()
