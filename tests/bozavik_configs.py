"""Small Bozavik configurations for the tests.  They differ from one another in every size and constant: order of layers,
widths (one not a multiple of 8), heads, query, key, value and rotated sizes (equal and unequal, multiples of 8 and not),
rotations of the whole rotated part and of a part of it, latents whose key row takes one, two, three, four, five and nine
blocks of 64 or is one the tensor-core kernel does not take, experts, top 1 to all, limits (the shared expert's other than
the others'), with and without a shared expert, and layers without feed-forward."""


def _plain(heads, dim, vdim, q_rank, kv_rank, scale):
    return {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}


def _rotated(heads, dim, vdim, q_rank, kv_rank, scale, rot_dim, base, dims=None):
    return {**_plain(heads, dim, vdim, q_rank, kv_rank, scale), "rot_dim": rot_dim, "rot": {"base": base, "dims": dims or rot_dim}}


def _moe(experts, top, ff, limit, shared=None):
    f = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        f["shared"] = {"ff": shared[0], "limit": shared[1]}
    return f


def _layer(mixer, mlp=None):
    return {"type": "latent_attention_2" if "rot_dim" in mixer else "latent_attention", "mixer": mixer, "mlp": mlp}


def _model(layers, vocab=97, width=64, eps=1e-5, scale=3.0, mult=0.6):
    return {"architecture": "Bozavik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "residual_mult": mult, "layers": layers}


MIXED = _model([
    _layer(_rotated(3, 24, 40, 56, 48, 0.15, 16, 10000.0), _moe(6, 2, 40, 1.2, (64, 0.8))),
    _layer(_plain(5, 16, 24, 24, 64, 0.25), _moe(9, 3, 24, 2.0, (24, 3.0))),
    _layer(_rotated(2, 32, 16, 40, 88, 0.2, 32, 300.0, 12)),
    _layer(_plain(7, 8, 8, 64, 40, 0.4), _moe(5, 1, 64, 0.7)),
], vocab=300, width=72, eps=2e-5, scale=5.0, mult=0.45)

# sizes that no tensor-core kernel takes
ODD = _model([
    _layer(_plain(3, 20, 28, 22, 44, 0.2), _moe(5, 2, 36, 1.0)),
    _layer(_rotated(2, 10, 14, 31, 30, 0.3, 6, 50.0), _moe(4, 4, 50, 1.5, (20, 1.1))),
    _layer(_plain(1, 33, 12, 17, 52, 0.2)),
], vocab=257, width=100, eps=1e-6, scale=1.0, mult=1.0)

# heads, rows and feed-forwards of sizes the tensor-core kernels like; rows of 4 and 5 blocks
WIDE = _model([
    _layer(_rotated(8, 64, 64, 96, 192, 0.05, 64, 500000.0), _moe(8, 2, 64, 1.4, (128, 1.0))),
    _layer(_plain(16, 32, 48, 128, 256, 0.09), _moe(8, 2, 64, 1.4, (64, 1.6))),
    _layer(_rotated(4, 48, 32, 64, 264, 0.07, 48, 1000.0, 16), _moe(12, 3, 128, 2.5)),
], vocab=384, width=128, scale=8.0, mult=0.3)

# a row of nine blocks whose values take two passes (512 + 64), and one of one block
DEEP = _model([
    _layer(_rotated(2, 32, 24, 48, 512, 0.1, 64, 20000.0), _moe(3, 2, 32, 1.0, (32, 1.3))),
    _layer(_plain(20, 8, 16, 16, 64, 0.3), _moe(3, 1, 48, 1.8, (40, 0.9))),
], vocab=130, width=48, eps=1e-4, scale=0.7, mult=0.8)

CONFIGS = {"mixed": MIXED, "odd": ODD, "wide": WIDE, "deep": DEEP}
