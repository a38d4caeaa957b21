"""Naselorn decoders without a GPU: configuration, tensors, cache geometry, key masks, the oracle itself.  The numbers are
checked in test_gpu_naselorn.py."""
import json

import pytest
import torch

from art_b200.engine.kv_cache import HybridCache
from art_b200.models.config import ModelConfig, config_from_dict, resolve_config
from art_b200.models.hybrid import HYBRID_PRESETS, HybridConfig, init_hybrid_weights, tensor_shapes
from art_b200.models.weights import init_base_weights, load_base_weights
from . import naselorn_oracle as oracle
from .hybrid_models import lightning, moe, naselorn, parallel, small_naselorn


def test_config_is_read_from_its_dictionary_and_found_by_the_registry(tmp_path):
    d = small_naselorn()
    (tmp_path / "config.json").write_text(json.dumps(d))
    cfg = ModelConfig.from_pretrained_dir(str(tmp_path))
    assert isinstance(cfg, HybridConfig) and cfg.family == "naselorn" and cfg.recurrent
    assert (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps, cfg.embed_scale) == (d["vocab"], d["width"], d["norm"]["eps"], d["embedding"]["scale"])
    assert not (cfg.post_norms or cfg.depth_average or cfg.tie_word_embeddings or cfg.embed_norm) and cfg.norm_offset == 1 and cfg.position_base == 10000
    for s, e in zip(cfg.layers, d["layers"]):
        m, p = e["mixer"], e["mlp"]
        if e["type"] == "lightning":
            assert (s.heads, s.dim, s.vdim, list(s.decay)) == (m["heads"], m["dim"], m["vdim"], m["decay"])
        else:
            a, r = s.parts
            x, y = m["left"], m["right"]
            assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.chunk, a.window) == (x["heads"], x["kv_heads"], x["dim"], x["vdim"], x["scale"],
                                                                                         x["mask"]["size"], 0)
            assert (r.heads, r.heads * r.dim, r.conv) == (y["blocks"], y["width"], y["conv"]) and s.part_scales == (m["left_scale"], m["right_scale"])
            assert s.recurrent and r.recurrent and not a.recurrent
        if p is None:
            assert not s.has_mlp
        elif p["kind"] == "dense":
            assert (s.mlp, s.act, s.ff, s.experts) == ("gated", "relu", p["ff"], 0)
        else:
            assert (s.experts, s.top, s.expert_ff, s.shared_ff) == (p["router"]["experts"], p["router"]["top"], p["expert"]["ff"], p["shared"]["ff"])
    for name in ("naselorn-tiny", "naselorn-2b-a1b", "naselorn-14b-a4b"):
        assert resolve_config(name).family == "naselorn" and HYBRID_PRESETS[name].num_params() > 0
    assert resolve_config("nikelix-1b").post_norms                        # the other design keeps its frame


@pytest.mark.parametrize("change,match", [
    (lambda d: d["layers"][0].update(type="hgrn2"), "mixer"), (lambda d: d["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
    (lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=3), "key heads"), (lambda d: d["layers"][0]["mixer"]["right"].update(blocks=4), "blocks"),
    (lambda d: d["layers"][0]["mlp"].update(kind="poly"), "feed-forward"), (lambda d: d["layers"][0]["mlp"]["router"].update(top=99), "experts")])
def test_what_the_kernels_do_not_compute_is_refused(change, match):
    d = json.loads(json.dumps(small_naselorn()))
    change(d)
    with pytest.raises(ValueError, match=match):
        config_from_dict(d)


def test_tensor_names_and_loading(tmp_path):
    from safetensors.torch import save_file

    d = naselorn([parallel(mlp=moe(2, 1)), lightning()])
    cfg = config_from_dict(d)
    shapes = tensor_shapes(cfg)
    assert {"embed", "head", "final.norm", "l0.norm1", "l0.norm2", "l1.norm1"} <= set(shapes) and "l1.norm2" not in shapes
    assert {k[len("l0.mix.left."):] for k in shapes if k.startswith("l0.mix.left.")} == {k + b for k in "qkvo" for b in ("", ".b")}
    assert {k[len("l0.mix.right."):] for k in shapes if k.startswith("l0.mix.right.")} == {
        "y", "y.b", "x", "x.b", "conv", "conv.b", "ra", "ra.b", "ri", "ri.b", "lam", "o"}
    assert shapes["l0.mix.right.ra"] == (3, 14, 14) and shapes["l0.mix.left.o"] == (84, 80) and shapes["l1.mix.norm"] == (42,)
    assert {k for k in shapes if k.startswith("l0.mlp.e1.")} == {"l0.mlp.e1.gate", "l0.mlp.e1.up", "l0.mlp.e1.down"}
    w = init_base_weights(cfg, seed=3, dtype=torch.bfloat16)
    assert {k: tuple(t.shape) for k, t in w.items()} == shapes
    assert abs(float(w["final.norm"].float().mean())) < 0.2 and float(w["l1.mix.norm"].float().mean()) > 0.8      # stored around zero / as it is
    (tmp_path / "config.json").write_text(json.dumps(d))
    save_file(w, str(tmp_path / "model.safetensors"))
    got = load_base_weights(str(tmp_path), cfg)
    assert all(torch.equal(got[k], w[k]) for k in w)
    save_file({k: v for k, v in w.items() if k != "l0.mix.right.lam"}, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError, match="lam"):
        load_base_weights(str(tmp_path), cfg)


def test_cache_geometry_of_a_layer_with_pages_and_state():
    cfg = config_from_dict(small_naselorn())
    kv = HybridCache(cfg, num_blocks=6, block_size=16, num_slots=2, device=torch.device("cpu"), dtype=torch.float32)
    assert set(kv.layers[0]) == {"0.kv", "1.state", "1.conv"} and set(kv.part(0, 1)) == {"state", "conv"} and set(kv.part(1, 0)) == {"state"}
    assert kv.part(0, 0)["kv"].shape == (6, 16, 2 * (16 + 32)) and kv.part(0, 1)["conv"].shape == (2, 2, 42) and kv.part(0, 1)["state"].dtype == torch.float32
    assert kv.part(3, 0)["kv"].shape[2] == 2 * (64 + 64)                  # value columns as the prompt kernel of these sizes reads them
    total = sum(t.numel() * t.element_size() for L in kv.layers for t in L.values())
    assert total == 6 * HybridCache.bytes_per_block(cfg, 16, 4) + 2 * HybridCache.bytes_per_slot(cfg)
    one_tap = config_from_dict(naselorn([parallel(conv=1)]))
    HybridCache(one_tap, 1, 16, 1, torch.device("cpu")).offload()


def test_first_key_and_plans_of_chunks():
    from art_b200.ops.hybrid import first_key, plan_prefill

    assert [first_key(p, 0, 10) for p in (0, 9, 10, 19, 20, 25)] == [0, 0, 10, 10, 20, 20]
    assert [first_key(p, 4, 10) for p in (9, 10, 12, 15)] == [6, 10, 10, 12]
    assert [first_key(p, 0, 0) for p in (0, 99)] == [0, 0] and [first_key(p, 1, 0) for p in (0, 99)] == [0, 99]
    plan = plan_prefill([(0, 0, 5), (2, 100, 300), (3, 64, 1)], 0, "cpu", chunk=64)
    assert plan.key_pos0.tolist() == [0, 64, 64] and plan.key_cnt.tolist() == [5, 336, 1] and plan.key_off.tolist() == [0, 8, 344]


def test_oracle_is_causal_and_a_changed_token_ends_with_its_chunk():
    d = naselorn([parallel(chunk=10, right=0.0)])
    w = init_hybrid_weights(config_from_dict(d), seed=1)
    toks = torch.randint(0, 211, (40,), generator=torch.Generator().manual_seed(0)).tolist()
    full = oracle.forward(d, w, toks)
    assert torch.allclose(full[:17], oracle.forward(d, w, toks[:17]), atol=1e-10)
    toks[23] = (toks[23] + 1) % 211
    seen = ((oracle.forward(d, w, toks) - full).abs().amax(-1) > 1e-9).nonzero().flatten().tolist()
    assert seen == list(range(23, 30))


def test_oracle_recurrences_forget_at_their_decay():
    p = lightning(heads=1, dim=2, vdim=2, decay=[0.5])["mixer"]
    w = {k: torch.eye(2, dtype=torch.float64) for k in "qkvo"}
    w.update(g=torch.zeros(2, 2, dtype=torch.float64), norm=torch.ones(2, dtype=torch.float64))
    h = torch.zeros(3, 2, dtype=torch.float64)
    h[0, 0] = 2.0
    h[2, 0] = 2.0
    s = float(oracle.silu(torch.tensor(2.0, dtype=torch.float64)))
    out = oracle.lightning(h, w, p, 0.0)
    # o_2 = (0.25 + 1) s^3 on the first column, normed over the row, halved by the gate's sigmoid(0)
    assert torch.allclose(out[2], torch.tensor([2 ** 0.5 / 2, 0.0], dtype=torch.float64)) and s > 0
