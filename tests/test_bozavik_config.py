"""Bozavik without a GPU: the configuration read and written back, refusals that name the key, the model as data
(arrangements, parts, tensor names, cache needs), a random model folder that the plain reader takes, and the plain
implementation held to itself."""
import copy

import numpy as np
import pytest

from bozavik_configs import CONFIGS, DEEP, MIXED, ODD, WIDE


def test_configuration_reads_and_writes_back():
    import ultima_b200 as u
    for name, raw in CONFIGS.items():
        cfg = u.config_from_dict(raw)
        assert cfg.architecture == "Bozavik" and len(cfg.layers) == len(raw["layers"])
        assert u.config_from_dict(cfg.to_dict()) == cfg, name
    cfg = u.config_from_dict(MIXED)
    assert cfg.embedding_scale == 5.0 and cfg.residual_mult == 0.45 and cfg.eps == 2e-5
    assert cfg.layers[0].mixer.rot_dim == 16 and cfg.layers[2].mixer.rot_dims == 12 and cfg.layers[1].mixer.rot_dim == 0
    assert cfg.layers[0].mlp.expert.limit == 1.2 and cfg.layers[0].mlp.shared.limit == 0.8 and cfg.layers[3].mlp.shared is None
    assert cfg.layers[2].mlp is None


@pytest.mark.parametrize("path,value,word", [
    (("layers", 0, "type"), "attention", "type"), (("layers", 0, "mixer", "q_rank"), 0, "q_rank"),
    (("layers", 0, "mixer", "rot", "dims"), 18, "rot.dims"), (("layers", 0, "mixer", "rot"), None, "rot"),
    (("layers", 1, "mixer", "scale"), "1", "scale"), (("layers", 0, "mlp", "kind"), "dense", "kind"),
    (("layers", 0, "mlp", "router", "top"), 7, "top"), (("layers", 0, "mlp", "expert", "limit"), 0.0, "limit"),
    (("layers", 0, "mlp", "shared"), 3, "shared"), (("norm",), 1e-5, "norm"), (("embedding",), 2.0, "embedding"),
    (("residual_mult",), "x", "residual_mult"), (("layers",), [], "layers")])
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


def test_the_model_as_data():
    import torch
    import ultima_b200 as u
    from ultima_b200.arch import model_spec_for
    from ultima_b200.parts.base import KVNeed, build_part
    spec = model_spec_for(u.config_from_dict(MIXED))
    assert [L.arrangement.kind for L in spec.layers] == ["norm_both", "norm_both", "norm_both_mixer_only", "norm_both"]
    assert spec.layers[0].arrangement.get("mult") == 0.45 and spec.embedding.get("scale") == 5.0
    names = {w.name: tuple(w.shape) for w in spec.weight_specs()}
    assert names["l0.mix.dq"] == (56, 72) and names["l0.mix.dq.norm"] == (56,) and names["l0.mix.uq"] == (3 * 40, 56)
    assert names["l0.mix.dkv"] == (64, 72) and names["l0.mix.uv"] == (120, 48) and names["l0.mix.g"] == (3, 72)
    assert "l0.mix.sink" not in names and names["l1.mix.sink"] == (5,) and names["l1.mix.g"] == (120, 72)
    assert names["l0.norm1"] == names["l0.norm1.b"] == names["l0.norm2b.b"] == names["final.norm.b"] == (72,)
    assert names["l0.mlp.router"] == (6, 72) and names["l0.mlp.shared.sg"] == (1, 72) and names["l0.mlp.e5.down"] == (72, 40)
    assert "l3.mlp.shared.sg" not in names and "l3.mlp.shared.up" not in names and "l2.norm2" not in names
    assert names["head"] == (300, 72)
    assert {"l2.norm2", "l2.norm2.b", "l2.norm2b", "l2.norm2b.b"} == set(spec.optional_tensors)
    assert build_part("mixer", spec.layers[0].part("mixer")).cache_need() == KVNeed(1, 64, None, values_in_keys=True)
    assert build_part("mixer", spec.layers[1].part("mixer")).cache_need() == KVNeed(1, 64, None, values_in_keys=True)
    # what is compiled: the tensor-core attention once for each number of blocks a key row takes, and only where it fits
    blocks = {d for s, d in spec.kernel_needs(torch.bfloat16) if s == "attn_latent.cu"}
    assert blocks == {("ROW_BLOCKS=1",), ("ROW_BLOCKS=2",)}
    assert not any(s == "attn_latent.cu" for s, _ in spec.kernel_needs(torch.float32))
    deep = model_spec_for(u.config_from_dict(DEEP)).kernel_needs(torch.bfloat16)
    assert {d for s, d in deep if s == "attn_latent.cu"} == {("ROW_BLOCKS=9",), ("ROW_BLOCKS=1",)}
    assert not any(s == "attn_latent.cu" for s, _ in model_spec_for(u.config_from_dict(ODD)).kernel_needs(torch.bfloat16))


def test_a_random_folder_is_read_by_the_plain_reader(tmp_path):
    import plain_bozavik as P
    import ultima_b200 as u
    from ultima_b200.arch import model_spec_for
    from ultima_b200.weights.loader import WeightError, check_weights
    from ultima_b200.weights.safetensors_io import write_safetensors
    import torch
    d = u.write_random_model(str(tmp_path / "m"), u.config_from_dict(ODD), seed=3, dtype="bfloat16")
    cfg, W = P.read_folder(d)
    assert cfg["architecture"] == "Bozavik" and W["l1.mix.dkv"].shape == (36, 100) and W["l2.norm1b.b"].shape == (100,)
    out = P.logits(cfg, W, [1, 2, 3, 4, 5])
    assert out.shape == (5, 257) and abs(out).max() > 0
    # causal: a longer sequence has the same first rows
    assert np.allclose(P.logits(cfg, W, [1, 2, 3, 4, 5, 6, 7])[:5], out, atol=1e-9)
    # the second sublayer's norms may stand in the file for a layer without feed-forward; anything else may not
    spec = model_spec_for(u.config_from_dict(ODD))
    more = {n: t.to(torch.bfloat16) for n, t in W.items()}
    more["l2.norm2"] = torch.ones(100, dtype=torch.bfloat16)
    write_safetensors(str(tmp_path / "m" / "model.safetensors"), more)
    check_weights(d, spec.weight_specs(), spec.optional_tensors)
    more["l2.norm3"] = more["l2.norm2"]
    write_safetensors(str(tmp_path / "m" / "model.safetensors"), more)
    with pytest.raises(WeightError):
        check_weights(d, spec.weight_specs(), spec.optional_tensors)


def test_slices_of_a_latent_decode_step_follow_from_what_a_captured_step_is_looked_up_by():
    """Two steps with the same key must want the same number of slices, whatever the sequences' lengths."""
    from ultima_b200.kernels import attn_tc
    for B in (1, 2, 5, 8, 33, 200):
        for parts in (1, 2):
            seen = {}
            for longest in range(1, 9000, 37):
                key = attn_tc.decode_slices(B, 1, longest, None, n_sms=148, cap=attn_tc.LATENT_SLICE_CAP)
                n = attn_tc.latent_slices(B, longest, None, parts, n_sms=148)
                assert seen.setdefault(key, n) == n and 1 <= n <= attn_tc.LATENT_SLICE_CAP


def test_a_stored_product_with_few_output_rows_spreads_over_smaller_token_tiles():
    from ultima_b200.kernels import gemm_tc
    from ultima_b200.kernels.ops import EPI_ADD, EPI_STORE
    assert gemm_tc.spread_tile(2048, 33, EPI_STORE, 148) == 64 and gemm_tc.spread_tile(2048, 33, EPI_ADD, 148) == 256
    assert gemm_tc.spread_tile(2048, 1024, EPI_STORE, 148) == 128 and gemm_tc.spread_tile(2048, 4096, EPI_STORE, 148) == 256
    assert gemm_tc.spread_tile(20, 33, EPI_STORE, 148) == 32


def test_the_bench_models_are_configurations_of_equal_active_size():
    """The models that ``bench.py --only bozavik`` times: chosen and shared experts together have the dense models' inner
    size, and every layer's attention is one the tensor-core kernel takes."""
    import os
    import sys
    sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    import bench
    import ultima_b200 as u
    from ultima_b200.kernels import attn_tc
    for z in bench.SUGIZEN_SIZES.values():
        cfg = u.config_from_dict(bench.bozavik_config(z))
        assert len(u.model_spec_for(cfg).layers) == z["layers"]
        for L in cfg.layers:
            m, f = L.mixer, L.mlp
            assert f.top * f.expert.ff + f.shared.ff == z["ff"]
            assert m.kv_rank + m.rot_dim == 256 and attn_tc.latent_fits(m.kv_rank + m.rot_dim, m.kv_rank, m.heads)
