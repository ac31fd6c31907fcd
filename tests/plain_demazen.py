"""A plain, slow implementation of the Demazen design: one function for each mechanism, on whole sequences, on the CPU.
It shares no code with the package: it takes config.json's dictionary and a dictionary of tensors by their stored names.

``dt`` is the type everything is computed in (float64 for an oracle).  Nothing here keeps a cache: a sequence is always
run whole, the recurrences token by token.
"""
from __future__ import annotations

import math

import torch


# ---------------------------------------------------------------------------------------
# norms and activations
# ---------------------------------------------------------------------------------------
def over_rms(x, eps):
    """x divided by its root mean square over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return over_rms(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def log_sigmoid(z):
    """ln(1 / (1 + e^-z)), without overflow on either side."""
    return torch.where(z > 0, -torch.log1p(torch.exp(-z.abs())), z - torch.log1p(torch.exp(-z.abs())))


# ---------------------------------------------------------------------------------------
# the matrix memory with exponential gates
# ---------------------------------------------------------------------------------------
def mlstm_gates(h, W, cap, pre):
    """(log input gate, log forget gate), [T, heads] each."""
    i = cap * torch.tanh((h @ W[pre + "i"].T + W[pre + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ W[pre + "f"].T + W[pre + "f.b"]) / cap))
    return i, f


def mlstm_memory(q, k, v, i, f):
    """q (scaled), k [T, H, D], v [T, H, E], log gates [T, H] -> [T, H, E], before any norm."""
    T, H, D = q.shape
    S, n, m = q.new_zeros(H, D, v.shape[-1]), q.new_zeros(H, D), q.new_zeros(H)
    out = []
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        m = m_new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hde,hd->he", S, q[t]) / den[:, None])
    return torch.stack(out)


def mlstm(h, W, m, eps, pre):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    q = (h @ W[pre + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ W[pre + "k"].T).view(T, H, D)
    v = (h @ W[pre + "v"].T).view(T, H, m["vdim"])
    i, f = mlstm_gates(h, W, m["gate_cap"], pre)
    o = over_rms(mlstm_memory(q, k, v, i, f), eps).reshape(T, -1) * W[pre + "norm"]
    return (o * torch.sigmoid(h @ W[pre + "g"].T)) @ W[pre + "o"].T


# ---------------------------------------------------------------------------------------
# windowed attention, gated linear attention, and the two side by side
# ---------------------------------------------------------------------------------------
def window_mask(T, size):
    """seen[i, j]: 0 <= i - j < size."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < size)


def attention_over_window(q, k, v, scale, size):
    """q [T, H, D], k [T, G, D], v [T, G, E]; query head h reads head h // (H / G) -> [T, H, E]."""
    r = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(r, dim=1), v.repeat_interleave(r, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~window_mask(q.shape[0], size)[None], -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return torch.einsum("hij,jhe->ihe", e / e.sum(-1, keepdim=True), v)


def window_attention(h, W, m, eps, pre):
    """Queries and keys are normed over all their heads at once; positions do not enter."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = rms_norm(h @ W[pre + "q"].T, W[pre + "q.norm"], eps).view(T, H, m["dim"])
    k = rms_norm(h @ W[pre + "k"].T, W[pre + "k.norm"], eps).view(T, G, m["dim"])
    v = (h @ W[pre + "v"].T).view(T, G, m["vdim"])
    return attention_over_window(q, k, v, m["scale"], m["mask"]["size"]).reshape(T, -1) @ W[pre + "o"].T


def channel_decay(h, W, tau, pre):
    """sigmoid(z)^(1/tau), z a low-rank map of h with a bias, [T, heads * dim]."""
    z = (h @ W[pre + "a1"].T) @ W[pre + "a2"].T + W[pre + "a2.b"]
    return torch.exp(log_sigmoid(z) / tau)


def decayed_memory(q, k, v, a):
    """q, k, a [T, H, D], v [T, H, E]: S <- diag(a) S + k v^T, o = S^T q -> [T, H, E]."""
    T, H, D = q.shape
    S = q.new_zeros(H, D, v.shape[-1])
    out = []
    for t in range(T):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out)


def gated_linear_attention(h, W, m, eps, pre):
    T, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ W[pre + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ W[pre + "k"].T).view(T, H, D)
    v = (h @ W[pre + "v"].T).view(T, H, E)
    o = rms_norm(decayed_memory(q, k, v, channel_decay(h, W, m["tau"], pre).view(T, H, D)), W[pre + "norm"], eps)
    return (o.reshape(T, H * E) * silu(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def side_by_side(h, W, m, eps, pre):
    a = rms_norm(window_attention(h, W, m["left"], eps, pre + "left."), W[pre + "left.out"], eps)
    b = rms_norm(gated_linear_attention(h, W, m["right"], eps, pre + "right."), W[pre + "right.out"], eps)
    return 0.5 * (a + b)


MIXERS = {"mlstm": mlstm, "parallel": side_by_side}


# ---------------------------------------------------------------------------------------
# feed-forwards
# ---------------------------------------------------------------------------------------
def gated_feed_forward(h, W, pre):
    return (silu(h @ W[pre + "gate"].T) * (h @ W[pre + "up"].T)) @ W[pre + "down"].T


def route(z, top):
    """The chosen experts of every token and their weights, [T, top] each: softmax over the chosen logits only."""
    best = torch.topk(z, top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def routed_feed_forward(h, W, f, pre):
    idx, w = route(h @ W[pre + "router"].T + W[pre + "router.b"], f["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, k = torch.nonzero(idx == e, as_tuple=True)
        if t.numel():
            out.index_add_(0, t, w[t, k][:, None] * gated_feed_forward(h[t], W, f"{pre}e{e}."))
    return out


def feed_forward(h, W, f, pre):
    return gated_feed_forward(h, W, pre) if f["kind"] == "dense" else routed_feed_forward(h, W, f, pre)


# ---------------------------------------------------------------------------------------
# the model
# ---------------------------------------------------------------------------------------
def owner(layers, i):
    """The layer whose tensors layer i uses."""
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def forward(cfg, W, tokens, dt=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out``: a list that receives the residual stream after every layer."""
    W = {n: (t.to(dt) if t.is_floating_point() else t) for n, t in W.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"][ids] + W["pos"][:len(ids)]
    for i, L in enumerate(cfg["layers"]):
        pre = f"l{owner(cfg['layers'], i)}."
        x = x + rms_norm(MIXERS[L["type"]](x, W, L["mixer"], eps, pre + "mix."), W[pre + "norm1"], eps)
        if L.get("mlp"):
            x = x + rms_norm(feed_forward(x, W, L["mlp"], pre + "mlp."), W[pre + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return capped(rms_norm(x, W["final.norm"], eps) @ W["embed"].T, cfg["logit_softcap"])


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
