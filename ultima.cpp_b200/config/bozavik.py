"""Bozavik: the typed configuration, read from the design's own config.json keys.

    architecture     "Bozavik"
    vocab, width     sizes of the embedding table
    norm.eps         the eps of every norm of the model
    embedding.scale  a constant on the embedding's rows
    residual_mult    a constant on what a sublayer adds to the stream
    layers           a list; each entry has
        type         "latent_attention" or "latent_attention_2"
        mixer        the mixer's sizes and constants (below)
        mlp          null, or {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top"},
                     "shared": {"ff", "limit"}}
    latent_attention mixer:    heads, dim, vdim, q_rank, kv_rank, scale
    latent_attention_2 mixer:  the same and rot_dim, rot {"base", "dims"}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .base import ConfigError

LATENT, LATENT_ROTATED = "latent_attention", "latent_attention_2"


def _int(d: dict, key: str, where: str, minimum: int = 1) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, int):
        raise ConfigError(f"config.json: {where}'{key}' must be an integer, got {v!r}")
    if v < minimum:
        raise ConfigError(f"config.json: {where}'{key}' must be >= {minimum}, got {v}")
    return v


def _num(d: dict, key: str, where: str) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: {where}'{key}' must be a number, got {v!r}")
    return float(v)


def _obj(d: dict, key: str, where: str, keys: str) -> dict:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}{key} must be an object with {keys}")
    return v


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_dim: int = 0                         # 0: no rotated part
    rot_base: float = 0.0
    rot_dims: int = 0


@dataclass(frozen=True)
class ExpertConfig:
    ff: int
    limit: float


@dataclass(frozen=True)
class RoutedConfig:
    experts: int
    top: int
    expert: ExpertConfig
    shared: Optional[ExpertConfig] = None


@dataclass(frozen=True)
class BozavikLayer:
    kind: str
    mixer: LatentMixer
    mlp: Optional[RoutedConfig]


def _read_mixer(kind, m: dict, where: str) -> LatentMixer:
    if kind not in (LATENT, LATENT_ROTATED):
        raise ConfigError(f"config.json: {where[:-6]}type must be '{LATENT}' or '{LATENT_ROTATED}', got {kind!r}")
    sizes = [_int(m, k, where) for k in ("heads", "dim", "vdim", "q_rank", "kv_rank")]
    scale = _num(m, "scale", where)
    if kind == LATENT:
        return LatentMixer(*sizes, scale)
    rot = _obj(m, "rot", where, "'base' and 'dims'")
    rot_dim, dims = _int(m, "rot_dim", where, 2), _int(rot, "dims", where + "rot.", 2)
    if dims % 2 or dims > rot_dim:
        raise ConfigError(f"config.json: {where}rot.dims must be even and at most rot_dim")
    return LatentMixer(*sizes, scale, rot_dim, _num(rot, "base", where + "rot."), dims)


def _read_expert(d: dict, where: str) -> ExpertConfig:
    limit = _num(d, "limit", where)
    if limit <= 0:
        raise ConfigError(f"config.json: {where}limit must be positive")
    return ExpertConfig(_int(d, "ff", where), limit)


def _read_mlp(f, where: str) -> Optional[RoutedConfig]:
    if f is None:
        return None
    if not isinstance(f, dict) or f.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}kind must be 'moe', got {f.get('kind') if isinstance(f, dict) else f!r}")
    r, e = _obj(f, "router", where, "'experts' and 'top'"), _obj(f, "expert", where, "'ff' and 'limit'")
    experts, top = _int(r, "experts", where + "router."), _int(r, "top", where + "router.")
    if top > experts:
        raise ConfigError(f"config.json: {where}router.top is more than the router has experts")
    shared = None if f.get("shared") is None else _read_expert(_obj(f, "shared", where, "'ff' and 'limit'"), where + "shared.")
    return RoutedConfig(experts, top, _read_expert(e, where + "expert."), shared)


@dataclass(frozen=True)
class BozavikConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    max_position_embeddings: int = 131072
    torch_dtype: str = "bfloat16"
    eos_token_id: tuple = ()
    architecture: str = "Bozavik"
    model_type: str = "bozavik"

    # ---- reading ---------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: dict) -> "BozavikConfig":
        vocab, width = _int(d, "vocab", ""), _int(d, "width", "")
        eps = _num(_obj(d, "norm", "", "'eps'"), "eps", "norm.")
        scale = 1.0
        if d.get("embedding") is not None:
            scale = _num(_obj(d, "embedding", "", "'scale'"), "scale", "embedding.")
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(L, dict) or not isinstance(L.get("mixer"), dict):
                raise ConfigError(f"config.json: {where}mixer must be an object")
            layers.append(BozavikLayer(L.get("type"), _read_mixer(L.get("type"), L["mixer"], where + "mixer."),
                                       _read_mlp(L.get("mlp"), where + "mlp.")))
        eos = d.get("eos_token_id")
        eos = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(eos))
        return cls(vocab=vocab, width=width, eps=eps, layers=tuple(layers), embedding_scale=scale,
                   residual_mult=_num(d, "residual_mult", "") if d.get("residual_mult") is not None else 1.0,
                   max_position_embeddings=int(d.get("max_positions", 131072)),
                   torch_dtype=str(d.get("torch_dtype", "bfloat16")), eos_token_id=eos)

    # ---- writing ---------------------------------------------------------------------------
    def to_dict(self) -> dict:
        out = []
        for L in self.layers:
            m = L.mixer
            d = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank, "scale": m.scale}
            if L.kind == LATENT_ROTATED:
                d.update(rot_dim=m.rot_dim, rot={"base": m.rot_base, "dims": m.rot_dims})
            mlp = None
            if L.mlp is not None:
                f = L.mlp
                mlp = {"kind": "moe", "expert": {"ff": f.expert.ff, "limit": f.expert.limit},
                       "router": {"experts": f.experts, "top": f.top}}
                if f.shared is not None:
                    mlp["shared"] = {"ff": f.shared.ff, "limit": f.shared.limit}
            out.append({"type": L.kind, "mixer": d, "mlp": mlp})
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
             "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult, "layers": out,
             "max_positions": self.max_position_embeddings, "torch_dtype": self.torch_dtype}
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        return d
