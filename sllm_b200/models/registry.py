"""Model registry: family name -> model class, cache class and seeded initialiser; source architecture name -> reader of
its config.json and tensors.  Engine construction (`build_engine`, the command line, the server, the trace runner) goes
through here."""
from __future__ import annotations

import json
import os
from typing import Optional

import torch

from .config import ModelConfig

# CUDA translation units of a family, for callers that build no more than they run (None: the whole library)
KERNEL_UNITS = {
    "zokuvik": ("elementwise", "gemm_tcgen05", "gemm_simt", "group_norm", "latent_attention", "latent_decode", "latent_prefill",
                "delta_rule", "state_scan"),
    "sepedra": ("elementwise", "gemm_tcgen05", "gemm_simt", "group_norm", "attention", "kv_attention", "short_conv", "latent_prefill", "rglru", "moe",
                "moe_dense"),
    "kegorax": ("elementwise", "gemm_tcgen05", "gemm_simt", "group_norm", "attention", "kv_attention", "short_conv", "latent_prefill",
                "linear_state", "state_scan", "moe", "moe_dense"),
    "fekolorn": ("elementwise", "gemm_tcgen05", "gemm_simt", "hyper_streams", "poly_norm", "attention", "kv_attention", "short_conv",
                 "latent_prefill", "linear_state", "state_scan"),
}

# families whose configuration lists its layers (ModelConfig.layer_specs): modules with ARCHITECTURE, config_from_source,
# pack_weights, named_tensors and make_cache.  They run on one GPU, in bf16 or fp32
LAYERED = ("zokuvik", "sepedra", "kegorax", "fekolorn")


def layered(family: str):
    """The module of a family in LAYERED."""
    import importlib
    return importlib.import_module(f".{family}", __package__)


def make_model(cfg: ModelConfig, weights, tp=None, ep=None):
    if cfg.family == "qwen35":
        from .qwen35 import Qwen35Model
        return Qwen35Model(cfg, weights, tp, ep)
    if cfg.family == "moe":
        from .moe import MoeModel
        return MoeModel(cfg, weights, tp, ep)
    if cfg.family == "zokuvik":
        from .zokuvik import ZokuvikModel
        return ZokuvikModel(cfg, weights, tp)
    if cfg.family == "sepedra":
        from .sepedra import SepedraModel
        return SepedraModel(cfg, weights, tp)
    if cfg.family == "kegorax":
        from .kegorax import KegoraxModel
        return KegoraxModel(cfg, weights, tp)
    if cfg.family == "fekolorn":
        from .fekolorn import FekolornModel
        return FekolornModel(cfg, weights, tp)
    from .llama import LlamaModel
    return LlamaModel(cfg, weights, tp)


def make_cache(cfg: ModelConfig, model, num_pages: int, device, max_seqs: int):
    """The family's cache: ``num_pages`` pages and, where layers are recurrent, ``max_seqs`` state slots."""
    if cfg.family == "qwen35":
        from ..cache.hybrid import HybridCache
        return HybridCache(cfg, num_pages, device, max_seqs=max_seqs, kv_heads=model.local_kv_heads, tp_size=model.tp.size)
    if cfg.family in LAYERED:
        return layered(cfg.family).make_cache(cfg, model, num_pages, device, max_seqs)
    from ..cache.paged import PagedKVCache
    return PagedKVCache(cfg, num_pages, device, kv_heads=model.local_kv_heads)


def init_random_weights(cfg: ModelConfig, device, seed: int = 0, tp_size: int = 1, tp_rank: int = 0, ep_size: int = 1,
                        ep_rank: int = 0):
    if cfg.family == "qwen35":
        from .qwen35 import init_random_qwen35_weights
        return init_random_qwen35_weights(cfg, device, seed, tp_size=tp_size, tp_rank=tp_rank, ep_size=ep_size, ep_rank=ep_rank)
    if cfg.family == "moe":
        from .moe import init_random_moe_weights
        return init_random_moe_weights(cfg, device, seed, tp_size, tp_rank, ep_size, ep_rank)
    if cfg.family == "zokuvik":
        from .zokuvik import init_random_zokuvik_weights
        return init_random_zokuvik_weights(cfg, device, seed)
    if cfg.family == "sepedra":
        from .sepedra import init_random_sepedra_weights
        return init_random_sepedra_weights(cfg, device, seed)
    if cfg.family == "kegorax":
        from .kegorax import init_random_kegorax_weights
        return init_random_kegorax_weights(cfg, device, seed)
    if cfg.family == "fekolorn":
        from .fekolorn import init_random_fekolorn_weights
        return init_random_fekolorn_weights(cfg, device, seed)
    from .llama import init_random_weights as init
    return init(cfg, device, seed, tp_size, tp_rank)


# ------------------------------------------------------------------------------------------ model folders
class ModelFolderError(RuntimeError):
    pass


def read_folder_config(path: str, dtype: str = "bf16", max_context: Optional[int] = None) -> ModelConfig:
    """ModelConfig of a folder with config.json, chosen by its ``architecture``."""
    readers = {m.ARCHITECTURE: m.config_from_source for m in map(layered, LAYERED)}
    try:
        with open(os.path.join(path, "config.json"), "r", encoding="utf-8") as f:
            d = json.load(f)
        read = readers.get(d.get("architecture"))
        if read is None:
            raise ModelFolderError(f"no model of architecture {d.get('architecture')!r} (known: {sorted(readers)})")
        name = os.path.basename(os.path.abspath(path)) or "model"
        return read(d, name=name, dtype=dtype, **({"max_context": max_context} if max_context else {}))
    except (OSError, ValueError, KeyError, TypeError) as exc:
        raise ModelFolderError(f"{path}: unusable config.json: {type(exc).__name__}: {exc}") from None


def load_folder_weights(path: str, cfg: ModelConfig, device):
    """Resident weights of a folder with model.safetensors."""
    from ..formats.safetensors import SafetensorsError, SafetensorsFile
    try:
        with SafetensorsFile(os.path.join(path, "model.safetensors")) as f:
            return layered(cfg.family).pack_weights(cfg, f.tensor, torch.device(device))
    except (OSError, ValueError, SafetensorsError) as exc:
        raise ModelFolderError(f"{path}: unusable model.safetensors: {exc}") from None
