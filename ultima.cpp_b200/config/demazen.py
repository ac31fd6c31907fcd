"""Demazen: the typed configuration, read from the design's own config.json keys.

    architecture     "Demazen"
    vocab, width     sizes of the embedding table
    max_positions    rows of the table of position vectors (the longest context)
    norm.eps         the eps of every norm of the model
    logit_softcap    the cap on the logits
    layers           a list; each entry has
        type         "mlstm" or "parallel"
        mixer        the mixer's sizes and constants (below)
        mlp          null, {"kind": "dense", "ff"} or {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}}
        weights_of   optional: the number of an equal layer whose tensors this one uses
    mlstm mixer:     heads, dim, vdim, gate_cap
    parallel mixer:  left  {heads, kv_heads, dim, vdim, scale, mask {"size"}}
                     right {heads, dim, vdim, tau}

The inner size of the decay's low-rank map stands in no key: it is the shape of the stored tensors
(``with_tensor_shapes``); a configuration written by this package carries it as ``right.rank``, so that a random model
can be made from it.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Optional

from .base import ConfigError

MLSTM, PARALLEL = "mlstm", "parallel"


def _int(d: dict, key: str, where: str, minimum: int = 1) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, int):
        raise ConfigError(f"config.json: {where}'{key}' must be an integer, got {v!r}")
    if v < minimum:
        raise ConfigError(f"config.json: {where}'{key}' must be >= {minimum}, got {v}")
    return v


def _num(d: dict, key: str, where: str, positive: bool = False) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: {where}'{key}' must be a number, got {v!r}")
    if positive and not v > 0:
        raise ConfigError(f"config.json: {where}'{key}' must be positive, got {v}")
    return float(v)


def _obj(d: dict, key: str, where: str, keys: str) -> dict:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}{key} must be an object with {keys}")
    return v


@dataclass(frozen=True)
class MatrixMemoryMixer:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class WindowAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None


@dataclass(frozen=True)
class GatedLinear:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: Optional[int] = None               # inner size of the decay's map; from the tensors' shapes when the file has no key


@dataclass(frozen=True)
class ParallelMixer:
    left: WindowAttention
    right: GatedLinear


@dataclass(frozen=True)
class FeedForwardConfig:
    ff: int
    experts: Optional[int] = None            # None: one dense feed-forward
    top: Optional[int] = None


@dataclass(frozen=True)
class DemazenLayer:
    kind: str
    mixer: object
    mlp: Optional[FeedForwardConfig]
    weights_of: Optional[int] = None


def _read_mixer(kind, m: dict, where: str):
    if kind == MLSTM:
        return MatrixMemoryMixer(_int(m, "heads", where), _int(m, "dim", where), _int(m, "vdim", where),
                                 _num(m, "gate_cap", where, positive=True))
    if kind != PARALLEL:
        raise ConfigError(f"config.json: {where[:-6]}type must be '{MLSTM}' or '{PARALLEL}', got {kind!r}")
    a = _obj(m, "left", where, "'heads', 'kv_heads', 'dim', 'vdim', 'scale' and 'mask'")
    r = _obj(m, "right", where, "'heads', 'dim', 'vdim' and 'tau'")
    wl, wr = where + "left.", where + "right."
    heads, kv_heads = _int(a, "heads", wl), _int(a, "kv_heads", wl)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {wl}heads must be a multiple of kv_heads")
    window = None
    if a.get("mask") is not None:
        window = _int(_obj(a, "mask", wl, "'size'"), "size", wl + "mask.")
    left = WindowAttention(heads, kv_heads, _int(a, "dim", wl), _int(a, "vdim", wl), _num(a, "scale", wl), window)
    right = GatedLinear(_int(r, "heads", wr), _int(r, "dim", wr), _int(r, "vdim", wr), _num(r, "tau", wr, positive=True),
                        None if r.get("rank") is None else _int(r, "rank", wr))
    return ParallelMixer(left, right)


def _read_mlp(f, where: str) -> Optional[FeedForwardConfig]:
    if f is None:
        return None
    kind = f.get("kind") if isinstance(f, dict) else f
    if kind == "dense":
        return FeedForwardConfig(_int(f, "ff", where))
    if kind != "moe":
        raise ConfigError(f"config.json: {where}kind must be 'dense' or 'moe', got {kind!r}")
    r, e = _obj(f, "router", where, "'experts' and 'top'"), _obj(f, "expert", where, "'ff'")
    experts, top = _int(r, "experts", where + "router."), _int(r, "top", where + "router.")
    if top > experts:
        raise ConfigError(f"config.json: {where}router.top is more than the router has experts")
    return FeedForwardConfig(_int(e, "ff", where + "expert."), experts, top)


@dataclass(frozen=True)
class DemazenConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple
    logit_softcap: Optional[float] = None
    max_position_embeddings: int = 0         # 0: from the shape of the stored table of position vectors
    torch_dtype: str = "bfloat16"
    eos_token_id: tuple = ()
    architecture: str = "Demazen"
    model_type: str = "demazen"

    # ---- reading ---------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: dict) -> "DemazenConfig":
        vocab, width = _int(d, "vocab", ""), _int(d, "width", "")
        eps = _num(_obj(d, "norm", "", "'eps'"), "eps", "norm.")
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(L, dict) or not isinstance(L.get("mixer"), dict):
                raise ConfigError(f"config.json: {where}mixer must be an object")
            of = None if L.get("weights_of") is None else _int(L, "weights_of", where, 0)
            layers.append(DemazenLayer(L.get("type"), _read_mixer(L.get("type"), L["mixer"], where + "mixer."),
                                       _read_mlp(L.get("mlp"), where + "mlp."), of))
        eos = d.get("eos_token_id")
        eos = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(eos))
        cfg = cls(vocab=vocab, width=width, eps=eps, layers=tuple(layers),
                  logit_softcap=None if d.get("logit_softcap") is None else _num(d, "logit_softcap", "", positive=True),
                  max_position_embeddings=0 if d.get("max_positions") is None else _int(d, "max_positions", ""),
                  torch_dtype=str(d.get("torch_dtype", "bfloat16")), eos_token_id=eos)
        for i, L in enumerate(layers):
            j = cfg.owner(i)
            a, b = replace(L, weights_of=None), replace(layers[j], weights_of=None)
            if a != b:
                raise ConfigError(f"config.json: layers[{i}].weights_of names layer {j}, whose sizes differ from its own")
        return cfg

    def owner(self, i: int) -> int:
        """The layer whose tensors layer ``i`` uses (itself, unless it says ``weights_of``)."""
        seen = set()
        while self.layers[i].weights_of is not None:
            seen.add(i)
            i = self.layers[i].weights_of
            if i >= len(self.layers) or i in seen:
                raise ConfigError(f"config.json: 'weights_of' must lead to a layer with tensors of its own; {i} does not")
        return i

    # ---- sizes that only the tensors give ------------------------------------------------------
    @property
    def needs_tensor_shapes(self) -> bool:
        return not self.max_position_embeddings or any(L.kind == PARALLEL and L.mixer.right.rank is None for L in self.layers)

    def with_tensor_shapes(self, shapes: dict) -> "DemazenConfig":
        """The configuration with the ranks of the decay maps and the number of position vectors read from the stored
        tensors' shapes (``shapes``: stored name -> shape)."""
        def rows(name):
            if name not in shapes or len(shapes[name]) != 2:
                raise ConfigError(f"the model's files hold no matrix '{name}', whose shape gives a size of the model")
            return int(shapes[name][0])
        layers = []
        for i, L in enumerate(self.layers):
            m = L.mixer
            if L.kind == PARALLEL and m.right.rank is None:
                m = replace(m, right=replace(m.right, rank=rows(f"l{self.owner(i)}.mix.right.a1")))
            layers.append(replace(L, mixer=m))
        return replace(self, layers=tuple(layers), max_position_embeddings=self.max_position_embeddings or rows("pos"))

    # ---- writing ---------------------------------------------------------------------------
    def to_dict(self) -> dict:
        out = []
        for L in self.layers:
            m = L.mixer
            if L.kind == MLSTM:
                d = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap}
            else:
                a, r = m.left, m.right
                left = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
                if a.window is not None:
                    left["mask"] = {"size": a.window}
                right = {"heads": r.heads, "dim": r.dim, "vdim": r.vdim, "tau": r.tau}
                if r.rank is not None:
                    right["rank"] = r.rank
                d = {"left": left, "right": right}
            mlp = None
            if L.mlp is not None:
                f = L.mlp
                mlp = {"kind": "dense", "ff": f.ff} if f.experts is None else \
                    {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
            entry = {"type": L.kind, "mixer": d, "mlp": mlp}
            if L.weights_of is not None:
                entry["weights_of"] = L.weights_of
            out.append(entry)
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
             "layers": out, "torch_dtype": self.torch_dtype}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.max_position_embeddings:
            d["max_positions"] = self.max_position_embeddings
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        return d
