"""Small Demazen configurations for the tests.  They differ from one another in every size and constant: order and number of
layers, widths (one not a multiple of 8), heads, kv heads (groups of one, several and all), key and value sizes (equal and
unequal, multiples of 16, of 4 and odd ones, every number of channels a lane of the scan holds), windows (below, at and above
a page, of one position), decay ranks and exponents, gate caps, experts, top 1 to all, dense and missing feed-forwards, and layers
that use another's tensors (once, twice, and one that comes later)."""
import copy


def _mem(heads, dim, vdim, cap):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def _par(left, right):
    """left: heads, kv_heads, dim, vdim, scale, window; right: heads, dim, vdim, tau, rank."""
    a = dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), left[:5]), mask={"size": left[5]})
    return {"type": "parallel", "mixer": {"left": a, "right": dict(zip(("heads", "dim", "vdim", "tau", "rank"), right))}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def _layer(mixer, mlp=None, of=None):
    L = {**copy.deepcopy(mixer), "mlp": mlp}
    if of is not None:
        L["weights_of"] = of
    return L


def _model(layers, vocab=97, width=64, eps=1e-5, cap=20.0, positions=512):
    return {"architecture": "Demazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap,
            "max_positions": positions, "layers": layers}


_A = _par((6, 3, 32, 48, 0.2, 40), (3, 24, 40, 8.0, 8))
_B = _mem(3, 40, 24, 9.0)

MIXED = _model([
    _layer(_B, _moe(7, 2, 40)),
    _layer(_A, _dense(96)),
    _layer(_mem(2, 16, 64, 15.0)),
    _layer(_B, _moe(7, 2, 40), of=0),
    _layer(_par((4, 1, 16, 16, 0.4, 70), (2, 64, 32, 2.0, 24)), _moe(5, 1, 24)),
    _layer(_A, _dense(96), of=1),
], vocab=300, width=72, eps=2e-5, cap=24.0)

# sizes that no tensor-core kernel and no vector load takes
ODD = _model([
    _layer(_par((3, 3, 20, 28, 0.3, 33), (5, 7, 11, 5.0, 3)), _moe(5, 3, 21)),
    _layer(_mem(3, 13, 9, 4.0), _dense(50)),
    _layer(_par((5, 1, 9, 6, 0.5, 1), (1, 30, 21, 1.0, 13))),
    _layer(_mem(3, 13, 9, 4.0), _dense(50), of=1),
], vocab=257, width=100, eps=1e-6, cap=17.5)

# sizes the tensor-core kernels like; keys of 64 and 128 with values of the same size and twice that
WIDE = _model([
    _layer(_par((4, 2, 64, 128, 0.12, 96), (2, 128, 64, 16.0, 16)), _moe(8, 3, 64)),
    _layer(_mem(2, 128, 128, 12.0), _dense(192)),
    _layer(_par((3, 1, 128, 128, 0.09, 130), (4, 32, 64, 4.0, 32)), _moe(12, 12, 64)),
    _layer(_par((2, 2, 128, 256, 0.08, 64), (1, 96, 160, 6.0, 40)), _dense(64)),
], vocab=384, width=128, cap=25.0)

# large state: keys of 256, values over a block of columns; a layer that uses one that comes later, and one used three times
DEEP = _model([
    _layer(_mem(1, 256, 96, 6.0), _dense(40), of=2),
    _layer(_par((2, 1, 48, 16, 0.2, 100), (1, 256, 72, 3.0, 20)), _moe(3, 2, 32)),
    _layer(_mem(1, 256, 96, 6.0), _dense(40)),
    _layer(_mem(1, 256, 96, 6.0), _dense(40), of=0),
], vocab=130, width=48, eps=1e-4, cap=50.0)

CONFIGS = {"mixed": MIXED, "odd": ODD, "wide": WIDE, "deep": DEEP}
