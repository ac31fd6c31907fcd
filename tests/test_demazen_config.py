"""Demazen without a GPU: the configuration read and written back, refusals that name the key, sizes taken from the tensors'
shapes, the model as data (arrangements, parts, run list, tensor names, cache needs), a random model folder that the plain reader
takes, the plain implementation held to itself, and how the scan cuts sequences."""
import copy
import os
import sys

import numpy as np
import pytest

from demazen_configs import CONFIGS, DEEP, MIXED, ODD, WIDE


def test_configuration_reads_and_writes_back():
    import ultima_b200 as u
    for name, raw in CONFIGS.items():
        cfg = u.config_from_dict(raw)
        assert cfg.architecture == "Demazen" and len(cfg.layers) == len(raw["layers"])
        assert u.config_from_dict(cfg.to_dict()) == cfg, name
    cfg = u.config_from_dict(MIXED)
    assert cfg.logit_softcap == 24.0 and cfg.eps == 2e-5 and cfg.max_position_embeddings == 512
    assert cfg.layers[0].mixer.gate_cap == 9.0 and cfg.layers[1].mixer.left.window == 40 and cfg.layers[1].mixer.right.tau == 8.0
    assert cfg.layers[1].mlp.experts is None and cfg.layers[2].mlp is None and cfg.layers[4].mlp.top == 1
    assert [cfg.owner(i) for i in range(6)] == [0, 1, 2, 0, 4, 1]
    assert [u.config_from_dict(DEEP).owner(i) for i in range(4)] == [2, 1, 2, 2]


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "attention", "type"), (("layers", 0, "mixer", "gate_cap"), 0.0, "gate_cap"),
    (("layers", 0, "mixer", "dim"), 0, "dim"), (("layers", 1, "mixer", "left"), None, "left"),
    (("layers", 1, "mixer", "left", "kv_heads"), 4, "kv_heads"), (("layers", 1, "mixer", "left", "scale"), "1", "scale"),
    (("layers", 1, "mixer", "left", "mask"), 40, "mask"), (("layers", 1, "mixer", "right", "tau"), -1, "tau"),
    (("layers", 0, "mlp", "kind"), "gated", "kind"), (("layers", 0, "mlp", "router", "top"), 8, "top"),
    (("layers", 3, "weights_of"), 1, "weights_of"), (("layers", 3, "weights_of"), 3, "weights_of"),
    (("layers", 3, "weights_of"), 9, "weights_of"), (("layers", 3, "mixer", "heads"), 4, "weights_of"),
    (("norm",), 1e-5, "norm"), (("logit_softcap",), 0.0, "logit_softcap"), (("max_positions",), "x", "max_positions"),
    (("layers",), [], "layers")])
def test_refusals_name_the_key(path, value, word):
    import ultima_b200 as u
    raw = copy.deepcopy(MIXED)
    d = raw
    for k in path[:-1]:
        d = d[k]
    d[path[-1]] = value
    with pytest.raises(u.ConfigError) as e:
        u.config_from_dict(raw)
    assert word in str(e.value)


def test_sizes_that_only_the_tensors_give(tmp_path):
    import json
    import ultima_b200 as u
    from ultima_b200.config.base import config_from_dir
    full = u.config_from_dict(MIXED)
    d = u.write_random_model(str(tmp_path / "m"), full, seed=1, dtype="bfloat16")
    with open(os.path.join(d, "config.json")) as f:
        raw = json.load(f)
    del raw["max_positions"]
    for L in raw["layers"]:
        if L["type"] == "parallel":
            del L["mixer"]["right"]["rank"]
    with pytest.raises(ValueError):
        u.model_spec_for(u.config_from_dict(raw))
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(raw, f)
    cfg = config_from_dir(d)
    assert cfg == full and cfg.layers[5].mixer.right.rank == 8


def test_the_model_as_data():
    import torch
    import ultima_b200 as u
    from ultima_b200.arch import model_spec_for
    from ultima_b200.parts.base import KVNeed, StateNeed, build_part
    spec = model_spec_for(u.config_from_dict(MIXED))
    assert [L.arrangement.kind for L in spec.layers] == ["norm_after", "norm_after", "norm_after_mixer_only", "norm_after"]
    assert [r.layer for r in spec.runs] == [0, 1, 2, 0, 3, 1] and all(r.cache_from is None for r in spec.runs)
    names = {w.name: tuple(w.shape) for w in spec.weight_specs()}
    assert names["embed"] == (300, 72) and names["pos"] == (512, 72) and "head" not in names and names["final.norm"] == (72,)
    assert names["l0.mix.q"] == (120, 72) and names["l0.mix.g"] == (72, 72) and names["l0.mix.norm"] == (72,)
    assert names["l0.mix.i"] == (3, 72) and names["l0.mix.f.b"] == (3,) and names["l0.mix.o"] == (72, 72)
    assert names["l1.mix.left.q.norm"] == (192,) and names["l1.mix.left.k.norm"] == (96,) and names["l1.mix.left.v"] == (144, 72)
    assert names["l1.mix.right.a1"] == (8, 72) and names["l1.mix.right.a2"] == (72, 8) and names["l1.mix.right.a2.b"] == (72,)
    assert names["l1.mix.right.norm"] == (40,) and names["l1.mix.left.out"] == names["l1.mix.right.out"] == (72,)
    assert names["l0.mlp.router"] == (7, 72) and names["l0.mlp.router.b"] == (7,) and names["l0.mlp.e6.down"] == (72, 40)
    assert names["l1.mlp.up"] == (96, 72) and not any(n.startswith(("l3.", "l5.")) for n in names)
    assert "l2.norm2" not in names and "l2.norm2" in spec.optional_tensors
    assert build_part("mixer", spec.layers[0].part("mixer")).cache_need() == (
        StateNeed((3, 40, 24)), StateNeed((3, 40)), StateNeed((3,)))
    assert build_part("mixer", spec.layers[1].part("mixer")).cache_need() == (KVNeed(3, 32, 40, 48), StateNeed((3, 24, 40)))
    # what is compiled: attention once for each pair of sizes the tensor-core kernels take
    pairs = {d for s, d in spec.kernel_needs(torch.bfloat16) if s == "attn_mma.cu"}
    assert pairs == {("HEAD_DIM=32", "HEAD_DIM_V=48"), ("HEAD_DIM=16",)}
    wide = {d for s, d in model_spec_for(u.config_from_dict(WIDE)).kernel_needs(torch.bfloat16) if s == "attn_tcgen05.cu"}
    assert wide == {("HEAD_DIM=64", "HEAD_DIM_V=128"), ("HEAD_DIM=128",), ("HEAD_DIM=128", "HEAD_DIM_V=256")}
    assert not any(s == "attn_mma.cu" for s, _ in model_spec_for(u.config_from_dict(ODD)).kernel_needs(torch.bfloat16))
    assert not any(s == "attn_mma.cu" for s, _ in spec.kernel_needs(torch.float32))


def test_a_random_folder_is_read_by_the_plain_reader(tmp_path):
    import plain_demazen as P
    import ultima_b200 as u
    d = u.write_random_model(str(tmp_path / "m"), u.config_from_dict(ODD), seed=3, dtype="bfloat16")
    cfg, W = P.read_folder(d)
    assert cfg["architecture"] == "Demazen" and W["l0.mix.right.a2"].shape == (35, 3) and W["l1.mlp.gate"].shape == (50, 100)
    out = P.logits(cfg, W, [1, 2, 3, 4, 5])
    assert out.shape == (5, 257) and 0 < abs(out).max() < cfg["logit_softcap"]
    # causal: a longer sequence has the same first rows
    assert np.allclose(P.logits(cfg, W, [1, 2, 3, 4, 5, 6, 7])[:5], out, atol=1e-9)


def test_the_plain_recurrences_against_their_sums_written_out():
    """Without their running maximum the exponential gates are plain sums: S_t = sum_s exp(F_t - F_s + i_s) k_s v_s^T with F the sum of
    the log forget gates; the decayed memory likewise with the product of the decays."""
    import torch
    import plain_demazen as P
    g = torch.Generator().manual_seed(1)
    T, H, D, E = 9, 2, 3, 4
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (D, D, E))
    i, f = torch.randn(T, H, generator=g, dtype=torch.float64) * 2 - 1, -torch.rand(T, H, generator=g, dtype=torch.float64)
    got = P.mlstm_memory(q, k, v, i, f)
    F = torch.cumsum(f, 0)
    a = torch.rand(T, H, D, generator=g, dtype=torch.float64)
    got2 = P.decayed_memory(q, k, v, a)
    for t in range(T):
        w = torch.exp(F[t] - F[:t + 1] + i[:t + 1])                             # [t + 1, H]
        qk = torch.einsum("hd,shd->sh", q[t], k[:t + 1])
        num, nq = torch.einsum("sh,she->he", w * qk, v[:t + 1]), (w * qk).sum(0)
        # both divided by exp(m): the denominator's floor is then 1 (and its small constant exp(m) times as large)
        m = torch.maximum(F[t], (F[t] - F[:t + 1] + i[:t + 1]).max(0).values)
        den = torch.maximum(nq.abs(), torch.ones(H, dtype=torch.float64)) + 1e-6 * torch.exp(m)
        assert torch.allclose(got[t], num / den[:, None], atol=1e-12)
        ref = torch.zeros(H, E, dtype=torch.float64)
        for s in range(t + 1):
            ref += ((q[t] * k[s] * a[s + 1:t + 1].prod(0)).sum(-1))[:, None] * v[s]
        assert torch.allclose(got2[t], ref, atol=1e-12)


def test_a_long_sequence_is_cut_into_chunks_that_cover_it():
    from ultima_b200.kernels import ops
    form = ops.LinForm(16, 64, 128, (0, 1024, 2048, 4096, 6144, 0), rank=16)
    for n_seqs in (1, 2, 7, 40, 3000):
        for longest in (1, 2, 63, 64, 255, 256, 257, 1000, 2048, 2049, 8192):
            n, size = ops.lin_chunks(form, n_seqs, longest, n_sms=148)
            assert n >= 1 and n * size >= longest and (n - 1) * size < longest and n * n_seqs <= 65535
            assert n == 1 or (n >= 4 and size >= ops.LIN_CHUNK and size % 8 == 0)
    assert ops.lin_chunks(form, 1, 2048, n_sms=148)[0] > 8 and ops.lin_chunks(form, 40, 2048, n_sms=148)[0] == 1


def test_the_bench_models_are_configurations_of_equal_active_size():
    """The models that ``bench.py --only demazen`` times: a token's chosen experts together have the dense models' inner size."""
    sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    import bench
    import ultima_b200 as u
    from ultima_b200.kernels import attn_tc
    for z in bench.SUGIZEN_SIZES.values():
        cfg = u.config_from_dict(bench.demazen_config(z))
        assert len(u.model_spec_for(cfg).layers) == z["layers"]
        for L in cfg.layers:
            assert L.mlp.ff * (L.mlp.top or 1) == z["ff"]
            if L.kind == "parallel":
                assert attn_tc.sizes_fit(L.mixer.left.dim, L.mixer.left.vdim)
