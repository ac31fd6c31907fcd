"""Bozavik as data: layers of latent attention in two forms, in the order the configuration lists them; the tensor names
of its files.

A layer has a layer norm (weight and bias) on what each sublayer reads and one on what it puts out, and a constant on what
it adds: x += m * norm1b(mixer(norm1(x))); x += m * norm2b(feed_forward(norm2(x))) (arrangement ``norm_both``).  Both mixers
are the part ``latent_attention`` with queries through a latent of their own: "latent_attention" without positions, with a
learned sink and a gate an output element; "latent_attention_2" with a rotated part (pairs of halves) and a gate a head.  The
feed-forward is ``routed_experts`` with clamped gated experts, weights from a softmax over the chosen logits, and a shared
expert behind a sigmoid gate.  The embedding's rows are multiplied by a constant.
"""
from __future__ import annotations

from ..config.base import ArchitectureEntry, register_architecture
from ..config.bozavik import LATENT, LATENT_ROTATED, BozavikConfig
from ..parts.base import ModelSpec, Run, layer, part

EXPERT_ALPHA, EXPERT_SHIFT = 1.702, 1.0      # an expert is down(g sigmoid(ALPHA g) (u + SHIFT))

_NAMES = {"mixer_norm": "norm1.", "mixer": "mix.", "mixer_norm_after": "norm1b.", "feed_forward_norm": "norm2.",
          "feed_forward": "mlp.", "feed_forward_norm_after": "norm2b."}

# part's own tensor name -> the name below the role's prefix in the files
_LATENT_NAMES = {"q_down.weight": "dq", "q_down_norm.weight": "dq.norm", "q_up.weight": "uq", "kv_down.weight": "dkv",
                 "kv_norm.weight": "dkv.norm", "k_up.weight": "uk", "v_up.weight": "uv", "gate_proj.weight": "g",
                 "o_proj.weight": "o", "sink": "sink"}
_EXPERT_NAMES = {"gate_proj.weight": "gate", "up_proj.weight": "up", "down_proj.weight": "down"}


def _norm_renames(name: str) -> list:
    return [(f"{name}.weight", name), (f"{name}.bias", f"{name}.b")]


def build_spec(cfg: BozavikConfig, max_positions: int | None = None) -> ModelSpec:
    max_pos = int(max_positions or cfg.max_position_embeddings)
    norm = part("layer", width=cfg.width, eps=cfg.eps, with_bias=True)
    layers, runs, optional = [], [], []
    renames = [("embed.weight", "embed"), ("head.weight", "head")] + _norm_renames("final.norm")
    for i, L in enumerate(cfg.layers):
        m, pre = L.mixer, f"l{i}."
        common = dict(width=cfg.width, n_heads=m.heads, head_dim=m.dim, v_head_dim=m.vdim, rank=m.kv_rank, q_rank=m.q_rank,
                      scale=m.scale, eps=cfg.eps)
        if L.kind == LATENT:
            mixer = part("latent_attention", rot_dim=0, learned_sink=True, gate="element", **common)
        elif L.kind == LATENT_ROTATED:
            mixer = part("latent_attention", rot_dim=m.rot_dim, theta=m.rot_base, rotary_dim=m.rot_dims, max_positions=max_pos,
                         pairing="halves", gate="head", **common)
        else:
            raise ValueError(f"Bozavik: unknown layer type {L.kind!r}")
        renames += [(f"{pre}mix.{a}", f"{pre}mix.{b}") for a, b in _LATENT_NAMES.items()]
        renames += _norm_renames(f"{pre}norm1") + _norm_renames(f"{pre}norm1b")
        roles = {"mixer_norm": norm, "mixer": mixer, "mixer_norm_after": norm}
        second = [f"{pre}norm2", f"{pre}norm2b"]
        if L.mlp is not None:
            f = L.mlp
            roles.update(feed_forward_norm=norm, feed_forward_norm_after=norm)
            roles["feed_forward"] = part(
                "routed_experts", width=cfg.width, inner=f.expert.ff, n_experts=f.experts, top=f.top, correction=False,
                score="logits", expert="gated_clamped", clamp=(f.expert.limit, EXPERT_ALPHA, EXPERT_SHIFT),
                shared_inner=f.shared.ff if f.shared else None, shared_limit=f.shared.limit if f.shared else None,
                shared_gate=f.shared is not None)
            for n in second:
                renames += _norm_renames(n)
            renames += [(f"{pre}mlp.router.weight", f"{pre}mlp.router"), (f"{pre}mlp.shared.out_gate.weight", f"{pre}mlp.shared.sg")]
            for e in range(f.experts):
                renames += [(f"{pre}mlp.experts.{e}.{a}", f"{pre}mlp.e{e}.{b}") for a, b in _EXPERT_NAMES.items()]
            renames += [(f"{pre}mlp.shared.{a}", f"{pre}mlp.shared.{b}") for a, b in _EXPERT_NAMES.items()]
            kind = "norm_both"
        else:
            optional += [t for n in second for t in (n, f"{n}.b")]       # a file may carry them for a layer without feed-forward
            kind = "norm_both_mixer_only"
        layers.append(layer(part(kind, mult=cfg.residual_mult), prefix=pre, names=tuple((r, _NAMES[r]) for r in roles), **roles))
        runs.append(Run(i))
    return ModelSpec(
        width=cfg.width, vocab_size=cfg.vocab, max_positions=max_pos,
        embedding=part("token_table", vocab_size=cfg.vocab, width=cfg.width, scale=cfg.embedding_scale), embedding_name="embed.",
        layers=tuple(layers), runs=tuple(runs), final_norm=norm, final_norm_name="final.norm.",
        head=part("linear", vocab_size=cfg.vocab, width=cfg.width, tied=False), head_name="head.",
        stop_token_ids=tuple(cfg.eos_token_id), renames=tuple(renames), optional_tensors=tuple(optional))


register_architecture(ArchitectureEntry(
    name="Bozavik", model_type="bozavik", supported=True,
    notes="Bozavik: latent attention with queries through a latent, with and without a rotated part, gates and a sink, between "
          "layer norms before and after; routed clamped experts with a gated shared one",
    config_cls=BozavikConfig, build_spec=build_spec))
