"""Hybrid decoders without a GPU: configuration and registry, weight loading, cache geometry, state slots, the scheduler's
handling of state and mixed batches, trace replay.  The numbers are checked in test_gpu_hybrid.py."""
import asyncio
import json

import pytest
import torch

from art_b200.engine.engine import Engine, SamplingParams
from art_b200.engine.kv_cache import BlockManager, HybridCache, StateSlots
from art_b200.engine.replay import Replay
from art_b200.models.config import ModelConfig, config_from_dict, resolve_config
from art_b200.models.hybrid import HYBRID_PRESETS, HybridConfig, init_hybrid_weights, tensor_shapes
from art_b200.models.weights import init_base_weights, load_base_weights
from . import nikelix_oracle as oracle
from .hybrid_models import small_design


def test_config_is_read_from_its_dictionary_and_found_by_the_registry(tmp_path):
    d = small_design()
    (tmp_path / "config.json").write_text(json.dumps(d))
    cfg = ModelConfig.from_pretrained_dir(str(tmp_path))
    assert isinstance(cfg, HybridConfig) and cfg.family == "nikelix" and cfg.vocab_size == d["vocab"]
    assert isinstance(resolve_config(str(tmp_path)), HybridConfig)
    assert isinstance(resolve_config("x", architecture=d), HybridConfig)
    assert [s.type for s in cfg.layers] == [e["type"] for e in d["layers"]]
    la = next(s for s in cfg.layers if s.type == "latent_attention")
    src = next(e for e in d["layers"] if e["type"] == "latent_attention")["mixer"]
    assert (la.window, la.scale, la.rope_base, la.kv_rank) == (src["mask"]["size"], src["scale"], src["rot"]["base"], src["kv_rank"])
    assert any(s.ff == 0 for s in cfg.layers)                    # a layer without feed-forward
    wk = next(s for s in cfg.layers if s.type == "wkv")
    assert wk.vdim == wk.dim
    assert isinstance(resolve_config("nikelix-7b"), HybridConfig) and HYBRID_PRESETS["nikelix-7b"].num_params() > 5e9
    with pytest.raises(ValueError, match="architecture"):
        config_from_dict({"architecture": "Unknown"})
    bad = small_design()
    bad["layers"][0]["type"] = "mamba"
    with pytest.raises(ValueError, match="mixer"):
        config_from_dict(bad)
    assert isinstance(config_from_dict({"num_attention_heads": 4, "vocab_size": 64, "hidden_size": 32, "num_hidden_layers": 1}), ModelConfig)


def test_weights_load_from_safetensors_and_are_checked(tmp_path):
    from safetensors.torch import save_file

    d = small_design()
    (tmp_path / "config.json").write_text(json.dumps(d))
    cfg = config_from_dict(d)
    w = init_base_weights(cfg, seed=3, dtype=torch.bfloat16)
    assert set(w) == set(tensor_shapes(cfg))
    save_file(w, str(tmp_path / "model.safetensors"))
    fresh = ModelConfig.from_pretrained_dir(str(tmp_path))
    got = load_base_weights(str(tmp_path), fresh)
    assert set(got) == set(w) and all(torch.equal(got[k], w[k]) for k in w)
    assert [s.decay_rank for s in fresh.layers] == [s.decay_rank for s in cfg.layers]      # read off the tensors
    cut = {k: v for k, v in w.items() if not k.endswith("norm1b")}
    save_file(cut, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError, match="norm1b"):
        load_base_weights(str(tmp_path), ModelConfig.from_pretrained_dir(str(tmp_path)))
    save_file({**w, "final.norm": torch.ones(3, dtype=torch.bfloat16)}, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError, match="final.norm"):
        load_base_weights(str(tmp_path), ModelConfig.from_pretrained_dir(str(tmp_path)))


def test_oracle_forward_is_causal_and_counts_positions_from_zero():
    """The oracle itself: a later token changes no earlier logits; a prefix alone gives the same logits."""
    d = small_design()
    cfg = config_from_dict(d)
    w = init_hybrid_weights(cfg, seed=1)
    toks = torch.randint(0, cfg.vocab_size, (40,), generator=torch.Generator().manual_seed(0)).tolist()
    full = oracle.forward(d, w, toks, torch.float64)
    part = oracle.forward(d, w, toks[:17], torch.float64)
    assert torch.allclose(full[:17], part, atol=1e-10)
    toks[30] = (toks[30] + 1) % cfg.vocab_size
    other = oracle.forward(d, w, toks, torch.float64)
    assert torch.allclose(full[:30], other[:30], atol=1e-10) and not torch.allclose(full[30], other[30], atol=1e-3)


def test_state_slots_and_cache_geometry():
    s = StateSlots(3)
    a = [s.alloc() for _ in range(3)]
    assert sorted(a) == [0, 1, 2] and s.alloc() is None
    s.free(a[1])
    assert s.num_free == 1 and s.alloc() == a[1]
    s.free(a[0])
    with pytest.raises(ValueError):
        s.free(a[0])
    cfg = config_from_dict(small_design())
    kv = HybridCache(cfg, num_blocks=6, block_size=16, num_slots=2, device=torch.device("cpu"), dtype=torch.float32)
    for spec, L in zip(cfg.layers, kv.layers):
        if spec.type == "latent_attention":
            assert L["latent"].shape[:2] == (6, 16) and L["latent"].shape[2] % 16 == 0
        else:
            assert L["state"].shape[:3] == (2, spec.heads, spec.vdim) and L["state"].dtype == torch.float32
            assert ("shift" in L) == (spec.type == "wkv")
    total = sum(t.numel() * t.element_size() for L in kv.layers for t in L.values())
    assert total == 6 * HybridCache.bytes_per_block(cfg, 16, 4) + 2 * HybridCache.bytes_per_slot(cfg)
    kv.layers[0][next(iter(kv.layers[0]))].fill_(2.0)
    kv.offload()
    assert not kv.resident
    kv.restore()
    assert float(kv.layers[0][next(iter(kv.layers[0]))].min()) == 2.0
    kv.discard()
    kv.restore()
    assert float(kv.layers[0][next(iter(kv.layers[0]))].abs().max()) == 0.0


class CountingRunner:
    """Stands in for a recurrent model on the CPU: its "state" is the sum of the tokens a slot has seen, which only comes
    out right if every token is fed exactly once, in order, to the slot its sequence holds."""

    mixed_steps = True
    device = torch.device("cpu")

    class cfg:
        vocab_size = 1000

    def __init__(self, n_slots: int):
        self.sum, self.seen = [0] * n_slots, [0] * n_slots
        self.batches: list[list[int]] = []

    def _feed(self, v) -> int:
        n1 = len(v.tokens) if v.upto is None else v.upto
        if v.num_cached == 0:
            self.sum[v.state_slot] = self.seen[v.state_slot] = 0
        assert self.seen[v.state_slot] == v.num_cached and len(v.blocks) * 4 >= n1
        self.sum[v.state_slot] += sum(v.tokens[v.num_cached:n1])
        self.seen[v.state_slot] = n1
        return self.sum[v.state_slot] % 997

    def prefill(self, seqs):
        slots = [v.state_slot for v in seqs]
        assert len(set(slots)) == len(slots)
        self.batches.append([(len(v.tokens) if v.upto is None else v.upto) - v.num_cached for v in seqs])
        out = [self._feed(v) for v in seqs]
        return [None if v.partial else t for v, t in zip(seqs, out)], [0.0] * len(seqs)

    def decode(self, seqs, n):
        toks = []
        work = [list(v.tokens) for v in seqs]
        for _ in range(n):
            step = []
            for v, w in zip(seqs, work):
                assert self.seen[v.state_slot] == len(w) - 1
                self.sum[v.state_slot] += w[-1]
                self.seen[v.state_slot] += 1
                step.append(self.sum[v.state_slot] % 997)
                w.append(step[-1])
            toks.append(step)
        return toks, [[0.0] * len(seqs) for _ in range(n)]

    def score_view(self, view, n_prompt):
        assert view.state_slot >= 0 and view.blocks
        self.seen[view.state_slot] = -1
        return [float(len(view.tokens) - n_prompt)]

    def set_adapter(self, slot, state):
        raise ValueError("no adapters")


class Slots:
    arena = None

    def __init__(self, n):
        self.state_slots = StateSlots(n)


def expected_tokens(prompt, n):
    s, out = sum(prompt), []
    for _ in range(n):
        out.append(s % 997)
        s += out[-1]
    return out


def make_engine(slots=4, blocks=64, **kw):
    kv = Slots(slots)
    run = CountingRunner(slots)
    return Engine(run, BlockManager(blocks, 4, True), eos_token_id=None, kv_cache=kv, **kw), run, kv


def drain(eng, seqs):
    for _ in range(10000):
        if all(s.finished for s in seqs):
            break
        eng.step()
    eng.step()
    assert all(s.finished for s in seqs)


def test_scheduler_gives_every_sequence_its_state_and_takes_it_back():
    eng, run, kv = make_engine(num_scheduler_steps=3)
    prompts = [list(range(3, 3 + n)) for n in (5, 9, 1, 30, 17, 2)]
    seqs = [eng.add_request(p, SamplingParams(max_tokens=11, temperature=0.0)) for p in prompts]      # more than slots
    drain(eng, seqs)
    for p, s in zip(prompts, seqs):
        assert s.output_ids == expected_tokens(p, 11)
    assert kv.state_slots.num_free == 4 and eng.bm.num_free == 64
    again = eng.generate_sync(prompts[3], SamplingParams(max_tokens=4, temperature=0.0))     # prefix cache stays out of it
    assert again.output_ids == expected_tokens(prompts[3], 4) and again.prefix_hit_tokens == 0
    assert eng.bm.stats()["prefix_hits"] == 0


def test_prompt_portions_share_steps_with_decoded_tokens():
    eng, run, kv = make_engine(num_scheduler_steps=2, max_num_batched_tokens=8)
    a = eng.add_request([1, 2, 3], SamplingParams(max_tokens=30, temperature=0.0))
    eng.step()
    b = eng.add_request(list(range(50)), SamplingParams(max_tokens=5, temperature=0.0))
    drain(eng, [a, b])
    assert a.output_ids == expected_tokens([1, 2, 3], 30) and b.output_ids == expected_tokens(list(range(50)), 5)
    assert any(1 in n and max(n) > 1 for n in run.batches)       # a mixed step happened: a portion beside a single token


def test_preempted_and_aborted_sequences_return_state_and_blocks():
    eng, run, kv = make_engine(slots=3, blocks=12, num_scheduler_steps=4)
    seqs = [eng.add_request(list(range(i, i + 8)), SamplingParams(max_tokens=14, temperature=0.0)) for i in range(3)]
    drain(eng, seqs)
    assert eng.stats.preemptions > 0
    assert all(s.output_ids == expected_tokens(list(range(i, i + 8)), 14) for i, s in enumerate(seqs))
    live = eng.add_request([5, 6], SamplingParams(max_tokens=40, temperature=0.0))
    eng.step()
    assert kv.state_slots.num_free == 2
    eng.abort(live)
    eng.step()
    assert kv.state_slots.num_free == 3 and eng.bm.num_free == 12


def test_scoring_borrows_a_slot_and_sleep_recomputes_states():
    eng, run, kv = make_engine()
    assert asyncio.run(eng.score([1, 2, 3], [4, 5])) == [2.0]
    assert kv.state_slots.num_free == 4 and eng.bm.num_free == 64
    kv.resident, kv.discard, kv.restore, kv.offload = True, lambda: None, lambda: None, lambda: None
    s = eng.add_request([9, 9, 9], SamplingParams(max_tokens=8, temperature=0.0))
    eng.step()
    eng.sleep(2)                                                 # memory is given up: the request starts over from its tokens
    assert kv.state_slots.num_free == 4
    eng.wake_up()
    drain(eng, [s])
    assert s.output_ids == expected_tokens([9, 9, 9], 8)


def test_replay_admits_continues_and_ends_requests():
    class LogitRunner(CountingRunner):
        def step_logits(self, views, want):
            rows = []
            for v, w in zip(views, want):
                t = self._feed(v)
                rows += [torch.full((1, 1000), float(t)) for _ in w]
            return torch.cat(rows) if rows else torch.empty(0, 1000)

    kv = Slots(2)
    rep = Replay(LogitRunner(2), BlockManager(8, 4, False), kv)
    out = rep.step([{"id": "a", "tokens": [1, 2, 3], "want": [2]}, {"id": "b", "tokens": [10], "want": []}])
    assert out.shape == (1, 1000) and float(out[0, 0]) == 6
    assert rep.step([{"id": "b", "tokens": [5], "want": [0]}])[0, 0] == 15       # "a" is left out of this step
    assert rep.step([{"id": "a", "tokens": [4], "want": [0]}], ["b"])[0, 0] == 10
    assert rep.step([{"id": "c", "tokens": [7], "want": [0]}], ["a", "c"])[0, 0] == 7      # b's slot again
    assert rep.bm.num_free == 8 and kv.state_slots.num_free == 2
    with pytest.raises(ValueError, match="ids below"):
        rep.step([{"id": "d", "tokens": [1000]}])
    rep.step([{"id": "e", "tokens": [1] * 20}, {"id": "f", "tokens": [1]}])
    with pytest.raises(RuntimeError, match="state slot"):
        rep.step([{"id": "g", "tokens": [1]}])
    with pytest.raises(RuntimeError, match="cache block"):
        rep.step([{"id": "e", "tokens": [1] * 40}])


def test_prefill_plan_covers_every_row_and_window():
    from art_b200.ops.hybrid import PREFILL_ROWS, plan_prefill

    portions = [(0, 0, 5), (2, 100, 300), (3, 7, 129)]
    plan = plan_prefill(portions, window=33, device="cpu")
    assert plan.key_pos0.tolist() == [0, 68, 0]
    assert plan.key_cnt.tolist() == [5, 332, 136]
    assert plan.key_off.tolist() == [0, 8, 8 + 336] and plan.n_keys == 8 + 336 + 136          # starts at multiples of 8
    assert plan.row_end.tolist() == [5, 305, 434] and plan.row_pos0.tolist() == [0, 95, -298]
    rows = []
    for s, r in zip(plan.tile_seq.tolist(), plan.tile_row.tolist()):
        rows += range(r, min(r + PREFILL_ROWS, plan.row_end.tolist()[s]))
    assert rows == list(range(434))
    assert plan_prefill(portions, window=0, device="cpu").key_pos0.tolist() == [0, 0, 0]


def test_a_process_that_needs_few_kernels_compiles_few(tmp_path, monkeypatch):
    """Every kernel a design's front-ends may call lies in the sources its layers ask for; one that is missing all the same
    is taken from the complete library."""
    import re

    from art_b200 import build
    from art_b200.engine.hybrid_runner import KERNEL_SOURCES, kernel_sources
    from art_b200.models.config import resolve_config
    from art_b200.ops import _lib

    everything = {p.stem for p in build.kernel_sources()}
    assert all(v <= everything for v in KERNEL_SOURCES.values())
    for name in ("nikelix-tiny", "naselorn-tiny", "gaborax-tiny"):
        assert {"hybrid_rows", "gemm_tcgen05"} <= kernel_sources(resolve_config(name)) < everything
    assert "linear_scan" not in kernel_sources(resolve_config("gaborax-tiny")) and "linear_scan" in kernel_sources(resolve_config("naselorn-tiny"))
    exported = {s: p.stem for p in build.kernel_sources() for s in re.findall(r"ARTB_EXPORT \w+ (artb_\w+)\(", p.read_text())}
    from art_b200.ops import hybrid as hy

    everyone = set().union(*(kernel_sources(resolve_config(n)) for n in ("nikelix-tiny", "naselorn-tiny", "gaborax-tiny")))
    assert {exported[s] for s in hy._sigs} <= everyone

    class Lib:
        artb_one = 1

    class Full:
        artb_two = 2

    monkeypatch.setattr(_lib, "_load", lambda name: Full)
    part = _lib._Part(Lib)
    assert part.artb_one == 1 and part.artb_two == 2
    with pytest.raises(AttributeError):
        part.artb_three
