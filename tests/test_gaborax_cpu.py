"""Gaborax decoders without a GPU: configuration, frequencies, tensors, cache geometry, the oracle itself.  The numbers are
checked in test_gpu_gaborax.py."""
import json
import math

import pytest
import torch

from art_b200.engine.kv_cache import HybridCache
from art_b200.models.config import ModelConfig, config_from_dict, resolve_config
from art_b200.models.hybrid import HYBRID_PRESETS, HybridConfig, LayerSpec, init_hybrid_weights, rope_frequencies, tensor_shapes
from art_b200.models.weights import init_base_weights, load_base_weights
from . import gaborax_oracle as oracle
from .hybrid_models import capped, gaborax, gated_heads, relu2_moe, small_gaborax, yarn


def test_config_is_read_from_its_dictionary_and_found_by_the_registry(tmp_path):
    d = small_gaborax()
    (tmp_path / "config.json").write_text(json.dumps(d))
    cfg = ModelConfig.from_pretrained_dir(str(tmp_path))
    assert isinstance(cfg, HybridConfig) and cfg.family == "gaborax" and not cfg.recurrent
    assert (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps) == (d["vocab"], d["width"], d["norm"]["eps"])
    assert not cfg.pre_norms and cfg.post_norms and cfg.layer_scale and cfg.tie_word_embeddings and cfg.norm_offset == 1 and cfg.norm_names(2) == (None, "norm2")
    assert not (cfg.depth_average or cfg.embed_norm) and cfg.embed_scale == 1 and cfg.position_base == 0
    for i, (s, e) in enumerate(zip(cfg.layers, d["layers"])):
        m, p, first = e["mixer"], e["mlp"], e["type"] == "attention"
        assert (s.heads, s.kv_heads, s.dim, s.vdim, s.rot_dim, s.rope_base, s.scale) == (m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]["dims"],
                                                                                         m["rot"]["base"], m["scale"])
        assert s.qk_norm and (s.rot_pairs, s.biases, s.head_gate) == (("half", False, True) if first else ("next", True, False)) and not s.out_bias
        assert s.softcap == m.get("softcap", 0) and s.kv_from == m.get("kv_from", -1) and cfg.kv_layer(i) == m.get("kv_from", i)
        sc = m["rot"].get("scaling")
        assert s.rope_scaling == (sc and (sc["factor"], sc["original"], sc["fast"], sc["slow"]))
        if p is None:
            assert not s.has_mlp
        else:
            r = p["router"]
            assert (s.mlp, s.act, s.glu, s.router) == ("moe", "relu2", False, "scores")
            assert (s.experts, s.identity, s.top, s.expert_ff, s.shared_ff, s.shared_gate) == (r["experts"], r["identity"], r["top"], p["expert"]["ff"],
                                                                                              p["shared"]["ff"], True)
    for name in ("gaborax-tiny", "gaborax-2b-a1b", "gaborax-14b-a4b"):
        assert resolve_config(name).family == "gaborax" and HYBRID_PRESETS[name].num_params() > 0
        assert any(s.kv_from >= 0 for s in resolve_config(name).layers)
    for name in ("nikelix-1b", "naselorn-2b-a1b"):                        # the other designs keep their frames
        assert resolve_config(name).pre_norms and not resolve_config(name).layer_scale


def test_what_the_configuration_leaves_out():
    e = gated_heads(mlp={"kind": "moe", "router": {"experts": 4, "top": 2}, "expert": {"ff": 8}})
    cfg = config_from_dict(gaborax([e]))
    s = cfg.layers[0]
    assert (s.identity, s.shared_ff, s.shared_gate, s.softcap, s.rope_scaling, s.kv_from) == (0, 0, False, 0.0, None, -1)
    shapes = tensor_shapes(cfg)
    assert not any("shared" in k for k in shapes) and shapes["l0.mlp.router"] == (4, 92) and "l0.ls2" in shapes


@pytest.mark.parametrize("change,match", [
    (lambda d: d["layers"][0].update(type="hgrn2"), "mixer"), (lambda d: d["layers"][1]["mixer"].update(kv_heads=3), "key heads"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=22), "rot.dims"), (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=3), "rot.dims"),
    (lambda d: d["layers"][0]["mlp"].update(kind="dense"), "feed-forward"), (lambda d: d["layers"][0]["mlp"]["router"].update(top=9), "experts"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(identity=252), "experts"), (lambda d: d["layers"][0]["mixer"].update(mask={"size": 8}), "mask"),
    (lambda d: d["layers"][2]["mixer"].update(kv_from=2), "kv_from"), (lambda d: d["layers"][2]["mixer"].update(kv_from=-1), "kv_from"),
    (lambda d: d["layers"][4]["mixer"].update(kv_from=2), "kv_from"), (lambda d: d["layers"][2]["mixer"].update(dim=24), "differ")])
def test_what_the_kernels_do_not_compute_is_refused(change, match):
    d = json.loads(json.dumps(small_gaborax()))
    change(d)
    with pytest.raises(ValueError, match=match):
        config_from_dict(d)


@pytest.mark.parametrize("dims,base,scaling", [(64, 1e4, None), (10, 300.0, yarn()), (64, 5e5, yarn(4.0, 8192, 32.0, 1.0)), (6, 20.0, yarn(8.0, 16, 2.0, 1.9)),
                                               (16, 1e4, yarn(1.0, 4096, 32, 1)), (4, 2.0, yarn(2.0, 100000, 1.0, 0.001))])
def test_frequencies_of_plain_and_scaled_rotations(dims, base, scaling):
    s = LayerSpec("attention", 1, dims, dims, kv_heads=1, rot_dim=dims, rope_base=base)
    if scaling:
        s.rope_scaling = tuple(scaling[k] for k in ("factor", "original", "fast", "slow"))
    want, m = oracle.frequencies({"dims": dims, "base": base, "scaling": scaling})
    got, scale = rope_frequencies(s)
    assert len(got) == dims // 2 and all(math.isclose(a, b, rel_tol=1e-12) for a, b in zip(got, want)) and math.isclose(scale, m)
    if scaling and scaling["factor"] > 1 and dims == 64:           # fast pairs are kept, slow ones interpolated
        assert got[0] == 1.0 and math.isclose(got[-1], base ** (-62 / 64) / scaling["factor"]) and scale > 1


def test_tensor_names_and_loading(tmp_path):
    from safetensors.torch import save_file

    d = small_gaborax()
    cfg = config_from_dict(d)
    shapes = tensor_shapes(cfg)
    mix = lambda i: {k[len(f"l{i}.mix."):] for k in shapes if k.startswith(f"l{i}.mix.")}      # noqa: E731
    assert {"embed", "final.norm", "l0.norm1", "l0.norm2", "l0.ls1", "l0.ls2", "l3.norm1", "l3.ls1"} <= set(shapes)
    assert not {"head", "l0.norm1b", "l3.norm2", "l3.ls2", "l0.dwa"} & set(shapes)
    assert mix(0) == {"q", "k", "v", "o", "q.b", "k.b", "v.b", "q.norm", "k.norm"} and mix(1) == {"q", "k", "v", "o", "q.norm", "k.norm", "g"}
    assert mix(2) == {"q", "o", "q.norm", "g"} and mix(5) == {"q", "o", "q.b", "q.norm"}          # keys and values are another layer's
    assert shapes["l0.mix.q.norm"] == (42,) and shapes["l0.mix.k"] == (42, 92) and shapes["l0.mix.v.b"] == (66,) and shapes["l2.mix.g"] == (6, 92)
    assert {k for k in shapes if k.startswith("l0.mlp.e1.")} == {"l0.mlp.e1.up", "l0.mlp.e1.down"}
    assert shapes["l0.mlp.router"] == (8, 92) and shapes["l0.mlp.correction"] == (8,) and shapes["l0.mlp.shared.sg"] == (1, 92)
    w = init_base_weights(cfg, seed=3, dtype=torch.bfloat16)
    assert {k: tuple(t.shape) for k, t in w.items()} == shapes
    assert abs(float(w["l0.norm1"].float().mean())) < 0.2 and float(w["l0.mix.q.norm"].float().mean()) > 0.8      # stored around zero / as it is
    (tmp_path / "config.json").write_text(json.dumps(d))
    save_file(w, str(tmp_path / "model.safetensors"))
    got = load_base_weights(str(tmp_path), cfg)
    assert all(torch.equal(got[k], w[k]) for k in w)
    save_file({k: v for k, v in w.items() if k != "l2.ls1"}, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError, match="ls1"):
        load_base_weights(str(tmp_path), cfg)


def test_a_layer_that_shares_keys_and_values_has_no_pages_of_its_own():
    cfg = config_from_dict(small_gaborax())
    kv = HybridCache(cfg, num_blocks=6, block_size=16, num_slots=2, device=torch.device("cpu"), dtype=torch.float32)
    assert kv.state_slots is None and [set(L) for L in kv.layers] == [{"kv"}, {"kv"}, set(), {"kv"}, set(), set()]
    assert kv.part(2, 0)["kv"] is kv.layers[1]["kv"] and kv.part(4, 0)["kv"] is kv.layers[1]["kv"] and kv.part(5, 0)["kv"] is kv.layers[3]["kv"]
    assert kv.layers[0]["kv"].shape == (6, 16, 3 * (16 + 32)) and kv.layers[3]["kv"].shape == (6, 16, 64 + 64)
    total = sum(t.numel() * t.element_size() for L in kv.layers for t in L.values())
    assert total == 6 * HybridCache.bytes_per_block(cfg, 16, 4) and HybridCache.bytes_per_slot(cfg) == 0
    kv.offload()
    kv.restore()
    assert kv.part(2, 0)["kv"] is kv.layers[1]["kv"]


def test_oracle_is_causal_and_its_choices_follow_the_correction():
    d = small_gaborax()
    w = init_hybrid_weights(config_from_dict(d), seed=1)
    toks = torch.randint(0, 199, (40,), generator=torch.Generator().manual_seed(0)).tolist()
    full = oracle.forward(d, w, toks)
    assert torch.allclose(full[:17], oracle.forward(d, w, toks[:17]), atol=1e-10)
    p = relu2_moe(3, 2, 2)
    h = torch.eye(5, dtype=torch.float64)
    m = {"router": torch.zeros(5, 5, dtype=torch.float64), "correction": torch.tensor([0.0, 0.3, 0.0, 0.2, 0.0], dtype=torch.float64)}
    best, a = oracle.route(h, m, p)
    assert best.tolist() == [[1, 3]] * 5 and torch.allclose(a, torch.full_like(a, 0.5))      # the weights know nothing of it


def test_oracle_rotation_keeps_relative_positions_in_both_layouts():
    x = torch.randn(1, 1, 12, dtype=torch.float64, generator=torch.Generator().manual_seed(0)).expand(30, 1, 12).contiguous()
    for interleaved in (False, True):
        r = oracle.rotate(x, {"dims": 8, "base": 30.0}, interleaved)
        s = r[:, 0] @ r[:, 0].T
        assert torch.allclose(s[3:, 3:], s[:-3, :-3]) and torch.equal(r[..., 8:], x[..., 8:]) and not torch.allclose(s[0, 1], s[0, 2])


def test_softcap_of_the_oracle_bounds_scores():
    q = torch.tensor([[[100.0]], [[100.0]]], dtype=torch.float64)
    v = torch.tensor([[[1.0]], [[0.0]]], dtype=torch.float64)
    k = torch.tensor([[[1.0]], [[-1.0]]], dtype=torch.float64)
    got = oracle.attend(q, k, v, 1.0, 2.0)[1, 0, 0]
    assert math.isclose(float(got), 1 / (1 + math.exp(-4.0)), rel_tol=1e-9)
