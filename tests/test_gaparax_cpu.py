"""Gaparax decoders without a GPU: configuration, tables, tensors, cache geometry, stream boundaries, the oracle itself.  The
numbers of the kernels are checked in test_gpu_gaparax.py."""
import json
import math

import pytest
import torch

from art_b200.engine.hybrid_runner import HybridRunner, kernel_sources
from art_b200.engine.kv_cache import HybridCache
from art_b200.models.config import ModelConfig, config_from_dict, resolve_config
from art_b200.models.hybrid import HYBRID_PRESETS, HybridConfig, check_weights, distance_buckets, init_hybrid_weights, tensor_shapes
from art_b200.models.weights import init_base_weights, load_base_weights
from art_b200.ops import hybrid as hy
from . import gaparax_oracle as oracle
from .hybrid_models import gaparax, group_moe, relu2_dense, sigmoid_heads, sink_latent, small_gaparax


def test_config_is_read_from_its_dictionary_and_found_by_the_registry(tmp_path):
    d = small_gaparax()
    (tmp_path / "config.json").write_text(json.dumps(d))
    cfg = ModelConfig.from_pretrained_dir(str(tmp_path))
    assert isinstance(cfg, HybridConfig) and cfg.family == "gaparax" and not cfg.recurrent
    assert (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps, cfg.streams) == (d["vocab"], d["width"], d["norm"]["eps"], d["streams"])
    assert cfg.pre_norms and cfg.residual_gate and not (cfg.post_norms or cfg.layer_scale or cfg.tie_word_embeddings or cfg.depth_average or cfg.embed_norm)
    assert cfg.norm_offset == 0 and cfg.embed_scale == 1 and cfg.residual_mult == 1 and cfg.norm_names(2) == ("norm2", None)
    for s, e in zip(cfg.layers, d["layers"]):
        m, p = e["mixer"], e["mlp"]
        assert (s.type, s.heads, s.dim, s.vdim, s.scale) == (e["type"], m["heads"], m["dim"], m["vdim"], m["scale"])
        if e["type"] == "attention":
            assert (s.kv_heads, s.chunk, s.softcap, s.bias_max, s.rot_dim) == (m["kv_heads"], m["mask"]["size"], m["softcap"], m["bias_max"], 0)
            assert s.sigmoid and s.qk_norm and s.qk_norm_heads and s.head_temp and s.out_gate and not (s.sink or s.biases or s.head_gate)
        else:
            sc = m["rot"]["scaling"]
            assert (s.kv_rank, s.rot_dim, s.rope_base, s.rot_pairs, s.window) == (m["kv_rank"], m["rot_dim"], m["rot"]["base"], "half", 0) and s.sink
            assert s.rope_scaling == (sc and (sc["factor"], sc["original"], sc["fast"], sc["slow"])) and not s.sigmoid
        if p is None:
            assert not s.has_mlp
        elif p["kind"] == "dense":
            assert (s.mlp, s.act, s.ff) == ("plain", "relu2", p["ff"])
        else:
            r = p["router"]
            assert (s.mlp, s.act, s.glu, s.router) == ("moe", "silu", True, "softmax")
            assert (s.experts, s.top, s.expert_ff, s.groups, s.group_keep, s.router_scale) == (r["experts"], r["top"], p["expert"]["ff"], r["groups"]["count"],
                                                                                              r["groups"]["keep"], r["scale"])
    for name in ("gaparax-tiny", "gaparax-2b-a1b", "gaparax-14b-a4b"):
        assert resolve_config(name).family == "gaparax" and HYBRID_PRESETS[name].num_params() > 0
    for name in ("nikelix-1b", "naselorn-2b-a1b", "gaborax-2b-a1b"):       # the other designs keep their frames and rotations
        c = resolve_config(name)
        assert not c.streams and not c.residual_gate and not any(m.sigmoid or m.sink for s in c.layers for m in s.mixers())
        assert all(m.rot_pairs == "next" for s in c.layers for m in s.mixers() if m.type == "latent_attention")
    assert {"latent_decode", "gqa_attn", "moe", "hybrid_rows"} <= kernel_sources(cfg) and "rglru" not in kernel_sources(cfg)


@pytest.mark.parametrize("change,match", [
    (lambda d: d["layers"][0].update(type="hgrn2"), "mixer"), (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "key heads"),
    (lambda d: d["layers"][1]["mixer"]["rot"].update(dims=4), "rot.dims"), (lambda d: d["layers"][1]["mixer"].update(mask={"size": 9}), "mask"),
    (lambda d: d["layers"][0]["mixer"].update(rot={"base": 10.0}), "rot"), (lambda d: d["layers"][0]["mixer"].update(bias_max=0), "bias_max"),
    (lambda d: d["layers"][0]["mlp"].update(kind="gated"), "feed-forward"), (lambda d: d["layers"][0]["mlp"].update(shared={"ff": 8}), "shared"),
    (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(count=4), "groups"), (lambda d: d["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "groups"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=5), "fewer"), (lambda d: d["layers"][0]["mlp"]["router"].update(bias=True), "bias"),
    (lambda d: d.update(streams=9), "streams")])
def test_what_the_kernels_do_not_compute_is_refused(change, match):
    d = json.loads(json.dumps(small_gaparax()))
    change(d)
    with pytest.raises(ValueError, match=match):
        config_from_dict(d)


@pytest.mark.parametrize("rows,reach", [(2, 2), (8, 5), (8, 64), (32, 128), (24, 500), (10, 11), (64, 4096), (9, 30)])
def test_distance_buckets_against_the_oracle(rows, reach):
    got = distance_buckets(rows, reach)
    assert got == [oracle.bucket(n, rows, reach) for n in range(len(got))] and got[-1] == rows - 1 and len(got) <= reach + 1
    assert all(oracle.bucket(n, rows, reach) == rows - 1 for n in range(len(got), 3 * reach)) and (len(got) == 1 or got[-2] < rows - 1)
    assert distance_buckets(rows, reach, 3) == got[:3]
    with pytest.raises(ValueError, match="distance"):
        distance_buckets(rows, rows // 2)


def test_distance_table_holds_the_bias_by_distance_in_base_two():
    rel, pb = torch.randn(6, 2), torch.randn(2)
    t = hy.distance_table(rel, distance_buckets(6, 20), pb)
    n = t.shape[1] - 2 * hy.BIAS_PAD
    for dist in (0, 1, 2, 3, 7, 19, 20, 150):
        want = (rel[oracle.bucket(dist, 6, 20)] + pb) / math.log(2)
        assert torch.allclose(t[:, hy.BIAS_PAD + min(dist, n - 1)], want, atol=1e-6)
        if dist < n + hy.BIAS_PAD:
            assert torch.allclose(t[:, hy.BIAS_PAD + dist], want, atol=1e-6)
    assert bool(torch.isfinite(t).all())


def test_tensor_names_and_loading(tmp_path):
    from safetensors.torch import save_file

    d = small_gaparax()
    cfg = config_from_dict(d)
    w = init_base_weights(cfg, seed=3, dtype=torch.bfloat16)
    shapes = tensor_shapes(cfg)
    assert {k: tuple(t.shape) for k, t in w.items()} == shapes
    mix = lambda i: {k[len(f"l{i}.mix."):] for k in shapes if k.startswith(f"l{i}.mix.")}      # noqa: E731
    assert mix(0) == {"q", "k", "v", "o", "q.norm", "k.norm", "g", "rel", "temp", "pb"} and mix(1) == {"q", "dkv", "dkv.norm", "uk", "uv", "o", "sink"}
    assert shapes["l0.mix.q.norm"] == (20,) and shapes["l0.mix.g"] == (48, 84) and shapes["l0.mix.rel"][1] == 4 and shapes["l1.mix.sink"] == (3,)
    assert {"head", "l0.hc1.in", "l0.hc1.out", "l0.hc2.mix", "l0.rg1", "l0.rg1.b", "l0.rg2", "l0.norm1", "l0.norm2"} <= set(shapes)
    assert not {"embed.norm", "l0.norm1b", "l3.norm2", "l3.hc2.in", "l3.rg2", "l0.mlp.router.b", "l0.mlp.correction"} & set(shapes)
    assert {k for k in shapes if k.startswith("l0.mlp.e1.")} == {"l0.mlp.e1.gate", "l0.mlp.e1.up", "l0.mlp.e1.down"}
    assert {k for k in shapes if k.startswith("l1.mlp.")} == {"l1.mlp.up", "l1.mlp.down"} and shapes["l0.hc2.mix"] == (3, 3)
    w["l0.mix.rel"] = torch.randn(10, 4).bfloat16()                # the rows of a distance bias are the tensor's
    (tmp_path / "config.json").write_text(json.dumps(d))
    save_file(w, str(tmp_path / "model.safetensors"))
    fresh = config_from_dict(d)
    got = load_base_weights(str(tmp_path), fresh)
    check_weights(fresh, got)
    assert all(torch.equal(got[k], w[k]) for k in w) and fresh.layers[0].bias_rows == 10
    for bad, match in (({k: v for k, v in w.items() if k != "l2.rg1.b"}, "rg1.b"), ({**w, "l1.mix.sink": torch.zeros(4).bfloat16()}, "sink"),
                       ({**w, "l4.mix.rel": torch.zeros(30, 5).bfloat16()}, "distance")):
        save_file(bad, str(tmp_path / "model.safetensors"))
        with pytest.raises(ValueError, match=match):
            check_weights(config_from_dict(d), load_base_weights(str(tmp_path), config_from_dict(d)))


def test_cache_geometry():
    cfg = config_from_dict(small_gaparax())
    kv = HybridCache(cfg, num_blocks=6, block_size=16, num_slots=2, device=torch.device("cpu"), dtype=torch.float32)
    assert kv.state_slots is None and [set(L) for L in kv.layers] == [{"kv"}, {"latent"}] * 3
    assert kv.layers[0]["kv"].shape == (6, 16, 2 * (32 + 16)) and kv.layers[1]["latent"].shape == (6, 16, 48 + 16)
    assert sum(t.numel() * t.element_size() for L in kv.layers for t in L.values()) == 6 * HybridCache.bytes_per_block(cfg, 16, 4)


@pytest.mark.parametrize("streams", [1, 2, 5])
def test_boundaries_of_streams_equal_the_oracles(streams):
    """One copy in front of the first sublayer and behind the last one stands for all of them."""
    d = gaparax([sigmoid_heads(mlp=relu2_dense()), sink_latent(), sigmoid_heads()], streams=streams)
    cfg = config_from_dict(d)
    w = init_hybrid_weights(cfg, seed=2)
    run = HybridRunner(cfg, None, w, device="cpu", dtype=torch.float32)
    g = torch.Generator().manual_seed(0)
    e = torch.randn(4, 84, generator=g)
    xs, mine = e.expand(streams, -1, -1), [e]
    assert run._embed_streams.n_in == 0 and torch.allclose(run._embed_streams.coef[1] * e, sum(a * e for a in w["l0.hc1.in"]), atol=1e-5)
    subs = [(0, 1), (0, 2), (1, 1), (2, 1)]
    for n, (i, k) in enumerate(subs):
        st, y = run.layers[i][f"hc{k}"], torch.randn(4, 84, generator=g)
        assert (st.n_in, st.n_out) == (1 if n == 0 else streams, 1 if n == 3 else streams)
        mix, out, nxt = st.coef[:st.n_in * st.n_out].view(st.n_in, st.n_out), st.coef[-2 * st.n_out:-st.n_out], st.coef[-st.n_out:]
        mine = [sum(mix[s, t] * mine[s] for s in range(st.n_in)) + out[t] * y for t in range(st.n_out)]
        hc = oracle.part(w, f"l{i}.hc{k}")
        xs = [sum(hc["mix"][s, t] * xs[s] for s in range(streams)) + hc["out"][t] * y for t in range(streams)]
        want = sum(xs) if n == 3 else sum(a * x for a, x in zip(w["l{}.hc{}.in".format(*subs[n + 1])], xs))
        assert torch.allclose(sum(a * x for a, x in zip(nxt, mine)), want, atol=1e-4)


def test_oracle_is_causal_and_ends_at_chunks():
    d = small_gaparax()
    w = init_hybrid_weights(config_from_dict(d), seed=1)
    toks = torch.randint(0, 193, (60,), generator=torch.Generator().manual_seed(0)).tolist()
    full = oracle.forward(d, w, toks)
    assert torch.allclose(full[:17], oracle.forward(d, w, toks[:17]), atol=1e-10)
    m = oracle.chunk_mask(9, 4)
    assert m[7].tolist() == [False] * 4 + [True] * 4 + [False] and m[4].tolist() == [False] * 4 + [True] + [False] * 4
    d = gaparax([sigmoid_heads(chunk=10)])                             # nothing of an earlier chunk is seen
    w = init_hybrid_weights(config_from_dict(d), seed=1)
    assert torch.allclose(oracle.forward(d, w, toks[:20])[10:], oracle.forward(d, w, [5] * 10 + toks[10:20])[10:], atol=1e-10)


def test_oracle_sink_groups_and_bias():
    s = torch.tensor([[1.0, 2.0, -math.inf]], dtype=torch.float64)
    p = oracle.sink_softmax(s, torch.tensor(0.5, dtype=torch.float64))
    z = math.exp(1) + math.exp(2) + math.exp(0.5)
    assert torch.allclose(p, torch.tensor([[math.exp(1) / z, math.exp(2) / z, 0.0]], dtype=torch.float64))
    r = group_moe(6, 3, 1, 2, scale=3.0)["router"]
    z = torch.tensor([[0.0, 1.0, 1.4, -5.0, 1.3, 1.2]], dtype=torch.float64)
    top, a = oracle.route(torch.eye(1, dtype=torch.float64), {"router": z.T}, r)      # the group of the best one, with its worst
    assert top.tolist() == [[2, 3]] and torch.allclose(a, 3 * torch.softmax(z, -1)[:, [2, 3]])
    assert [oracle.bucket(n, 8, 16) for n in (0, 3, 4, 5, 6, 8, 12, 15, 16, 99)] == [0, 3, 4, 4, 5, 6, 7, 7, 7, 7]
