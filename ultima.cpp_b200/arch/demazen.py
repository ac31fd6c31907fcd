"""Demazen as data: layers of two kinds in the order the configuration lists them, some of them run again with a cache of
their own; the tensor names of its files.

A layer norms what its sublayers put out: x += norm1(mixer(x)); x += norm2(feed_forward(x)) (arrangement ``norm_after``).
The mixer is a matrix memory with exponential gates (part ``matrix_memory``), or two mixers side by side (part
``side_by_side`` with ``norm_outputs``): attention over a window, its queries and keys normed over all heads at once, no
positions (part ``attention``), and gated linear attention (part ``gated_linear``).  The feed-forward is ``gated_silu`` or
``routed_experts`` whose router has a bias and weighs the chosen logits.  A learned vector of its position is added to a
token's row of the embedding table; the head is that table, its logits capped.  A layer that names another's tensors is
that layer, once more in the run list.
"""
from __future__ import annotations

from ..config.base import ArchitectureEntry, register_architecture
from ..config.demazen import MLSTM, PARALLEL, DemazenConfig
from ..parts.base import ModelSpec, Run, layer, part

_NAMES = {"mixer": "mix.", "mixer_norm": "norm1.", "feed_forward": "mlp.", "feed_forward_norm": "norm2."}

# part's own tensor name -> the name below the role's prefix in the files
_MEMORY_NAMES = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "gate_proj.weight": "g", "o_proj.weight": "o",
                 "o_norm.weight": "norm", "i_proj.weight": "i", "i_bias": "i.b", "f_proj.weight": "f", "f_bias": "f.b"}
_LEFT_NAMES = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o", "q_norm.weight": "q.norm",
               "k_norm.weight": "k.norm"}
_RIGHT_NAMES = {"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "gate_proj.weight": "g", "o_proj.weight": "o",
                "o_norm.weight": "norm", "decay_down.weight": "a1", "decay_up.weight": "a2", "decay_bias": "a2.b"}
_PARALLEL_NAMES = {**{f"left.{a}": f"left.{b}" for a, b in _LEFT_NAMES.items()},
                   **{f"right.{a}": f"right.{b}" for a, b in _RIGHT_NAMES.items()},
                   "left_out.weight": "left.out", "right_out.weight": "right.out"}
_DENSE_NAMES = {"gate_proj.weight": "gate", "up_proj.weight": "up", "down_proj.weight": "down"}
SIDE_SCALE = 0.5                                   # half the sum of the two sides


def _mixer(cfg: DemazenConfig, L):
    m = L.mixer
    if L.kind == MLSTM:
        return part("matrix_memory", width=cfg.width, n_heads=m.heads, head_dim=m.dim, v_head_dim=m.vdim, gate_cap=m.gate_cap,
                    eps=cfg.eps), _MEMORY_NAMES
    if L.kind != PARALLEL:
        raise ValueError(f"Demazen: unknown layer type {L.kind!r}")
    a, r = m.left, m.right
    left = part("attention", width=cfg.width, n_heads=a.heads, n_kv_heads=a.kv_heads, head_dim=a.dim, v_head_dim=a.vdim,
                qk_norm=True, norm_whole=True, eps=cfg.eps, position=None, window=a.window, scale=a.scale)
    right = part("gated_linear", width=cfg.width, n_heads=r.heads, head_dim=r.dim, v_head_dim=r.vdim, decay_rank=r.rank, tau=r.tau,
                 eps=cfg.eps)
    return part("side_by_side", left=left, right=right, left_scale=SIDE_SCALE, right_scale=SIDE_SCALE,
                norm_outputs=cfg.eps), _PARALLEL_NAMES


def build_spec(cfg: DemazenConfig, max_positions: int | None = None) -> ModelSpec:
    if cfg.needs_tensor_shapes:
        raise ValueError("Demazen: the rank of a decay map or the number of position vectors is not known; read the "
                         "configuration with config_from_dir (which takes them from the tensors' shapes) or give 'rank' and "
                         "'max_positions'")
    max_pos = min(int(max_positions or cfg.max_position_embeddings), cfg.max_position_embeddings)
    norm = part("rms", width=cfg.width, eps=cfg.eps)
    layers, index, runs, optional = [], {}, [], []
    renames = [("embed.weight", "embed"), ("embed.positions", "pos"), ("final.norm.weight", "final.norm")]
    for i, L in enumerate(cfg.layers):
        if L.weights_of is not None:
            continue
        pre = f"l{i}."
        mixer, names = _mixer(cfg, L)
        renames += [(f"{pre}mix.{a}", f"{pre}mix.{b}") for a, b in names.items()]
        renames.append((f"{pre}norm1.weight", f"{pre}norm1"))
        roles = {"mixer": mixer, "mixer_norm": norm}
        kind = "norm_after_mixer_only"
        if L.mlp is not None:
            f = L.mlp
            kind = "norm_after"
            renames.append((f"{pre}norm2.weight", f"{pre}norm2"))
            if f.experts is None:
                ff = part("gated_silu", width=cfg.width, inner=f.ff)
                renames += [(f"{pre}mlp.{a}", f"{pre}mlp.{b}") for a, b in _DENSE_NAMES.items()]
            else:
                ff = part("routed_experts", width=cfg.width, inner=f.ff, n_experts=f.experts, top=f.top, correction=False,
                          score="logits", logit_bias=True)
                renames += [(f"{pre}mlp.router.weight", f"{pre}mlp.router"), (f"{pre}mlp.router.bias", f"{pre}mlp.router.b")]
                for e in range(f.experts):
                    renames += [(f"{pre}mlp.experts.{e}.{a}", f"{pre}mlp.e{e}.{b}") for a, b in _DENSE_NAMES.items()]
            roles.update(feed_forward=ff, feed_forward_norm=norm)
        else:
            optional.append(f"{pre}norm2")         # a file may carry it for a layer without feed-forward
        index[i] = len(layers)
        layers.append(layer(part(kind), prefix=pre, names=tuple((r, _NAMES[r]) for r in roles), **roles))
    runs = tuple(Run(index[cfg.owner(i)]) for i in range(len(cfg.layers)))
    return ModelSpec(
        width=cfg.width, vocab_size=cfg.vocab, max_positions=max_pos,
        embedding=part("token_table", vocab_size=cfg.vocab, width=cfg.width, positions=cfg.max_position_embeddings),
        embedding_name="embed.", layers=tuple(layers), runs=runs, final_norm=norm, final_norm_name="final.norm.",
        head=part("linear", vocab_size=cfg.vocab, width=cfg.width, tied=True, softcap=cfg.logit_softcap), head_name="head.",
        stop_token_ids=tuple(cfg.eos_token_id), renames=tuple(renames), optional_tensors=tuple(optional))


register_architecture(ArchitectureEntry(
    name="Demazen", model_type="demazen", supported=True,
    notes="Demazen: matrix memories with exponential gates, windowed attention beside gated linear attention, dense and routed "
          "feed-forwards, norms behind the sublayers, layers run again, learned positions and capped logits",
    config_cls=DemazenConfig, build_spec=build_spec))
