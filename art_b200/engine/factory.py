"""One place that turns a configuration and its weights into a rollout engine's parts: cache, runner, block manager.

The model family decides: Hugging Face families run on :class:`~art_b200.engine.runner.NativeRunner` over a
:class:`~art_b200.engine.kv_cache.KVCache`, hybrid designs on :class:`~art_b200.engine.hybrid_runner.HybridRunner` over a
:class:`~art_b200.engine.kv_cache.HybridCache`.
"""
from __future__ import annotations

import torch

from ..models.hybrid import HybridConfig
from ..models.weights import LoraConfig
from .engine import Engine
from .kv_cache import BlockManager, HybridCache, KVCache


class UnsupportedPrecision(ValueError):
    """The model family does not run in the requested number format."""


def build_runner(cfg, base: dict[str, torch.Tensor] | None, *, num_blocks: int, block_size: int = 16, num_slots: int = 256,
                 device: torch.device | str = "cuda", dtype: torch.dtype = torch.bfloat16, lora_cfg: LoraConfig | None = None,
                 max_loras: int = 4, tp_group=None, decoder=None, use_arena: bool = False):
    """``(runner, cache)`` on ``device``.  ``num_slots`` bounds the sequences that hold recurrent state at once."""
    dev = torch.device(device)
    if dev.type == "cuda" and dev.index is None:       # the engine's stepping thread selects it by number
        dev = torch.device("cuda", torch.cuda.current_device())
    if isinstance(cfg, HybridConfig):
        from .hybrid_runner import HybridRunner

        if tp_group is not None and torch.distributed.get_world_size(tp_group) > 1:
            raise ValueError("hybrid models run on one GPU per replica")
        kv = HybridCache(cfg, num_blocks, block_size, num_slots, dev, dtype)
        return HybridRunner(cfg, kv, base, device=dev, dtype=dtype), kv
    from .runner import NativeRunner

    if dtype != torch.bfloat16:
        raise UnsupportedPrecision(f"{cfg.family} models run in bfloat16")
    tp = 1 if tp_group is None else torch.distributed.get_world_size(tp_group)
    args = (cfg.num_layers, num_blocks, block_size, cfg.num_kv_heads // tp, cfg.head_dim, dev)
    try:
        kv = KVCache(*args, use_arena=use_arena)
    except RuntimeError:   # no VMM support: plain tensors; Engine.sleep() then drops the captured graphs
        if not use_arena:
            raise
        kv = KVCache(*args)
    return NativeRunner(cfg, lora_cfg or LoraConfig(), kv, decoder=decoder, base=base, max_loras=max_loras, device=dev,
                        tp_group=tp_group), kv


def cache_bytes(cfg, block_size: int, tp: int = 1) -> tuple[int, int]:
    """(bytes of one cache block, bytes of one state slot) over all layers."""
    if isinstance(cfg, HybridConfig):
        return max(1, HybridCache.bytes_per_block(cfg, block_size)), HybridCache.bytes_per_slot(cfg)
    return KVCache.bytes_per_block(cfg.num_layers, block_size, cfg.num_kv_heads // tp, cfg.head_dim), 0


def build_engine(cfg, base: dict[str, torch.Tensor], *, num_blocks: int, block_size: int = 16, max_num_seqs: int = 256,
                 max_loras: int = 4, device="cuda", dtype: torch.dtype = torch.bfloat16, lora_cfg: LoraConfig | None = None,
                 enable_prefix_caching: bool = True, eos_token_id: int | None = None, **engine_kw) -> Engine:
    """A rollout engine of either family on one GPU; ``engine_kw`` goes to :class:`Engine`."""
    runner, kv = build_runner(cfg, base, num_blocks=num_blocks, block_size=block_size, num_slots=max_num_seqs, device=device,
                              dtype=dtype, lora_cfg=lora_cfg, max_loras=max_loras)
    return Engine(runner, BlockManager(num_blocks, block_size, enable_prefix_caching), eos_token_id=eos_token_id,
                  max_num_seqs=max_num_seqs, max_loras=max_loras, kv_cache=kv, **engine_kw)
