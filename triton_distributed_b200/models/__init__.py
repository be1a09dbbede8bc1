"""Models, KV caches, weight loading and the serving engine (the reference's ``triton_dist.models``)."""
from .config import ArchConfig, ModelConfig, PRESETS  # noqa: F401
from .kv_cache import (DeltaSpec, GroupSpec, HybridCache, KV_Cache, KVSpec, LatentSpec, PagedKVCache, SharedSpec, StateSpec,  # noqa: F401
                       StepPlan, TiedKVSpec, WindowKVSpec)
from .safetensors_io import SafetensorsFile, ShardedCheckpoint, save_file  # noqa: F401
from .dense import DenseLLM, DenseLLMLayer  # noqa: F401
from .engine import Engine  # noqa: F401
from .qwen_moe import Qwen3MoE, Qwen3MoELayer  # noqa: F401
from .bagasun import BAGASUN_PRESETS, BagasunConfig, BagasunLLM  # noqa: F401
from .lisenex import LISENEX_PRESETS, LisenexConfig, LisenexLLM  # noqa: F401
from .tazitar import TAZITAR_PRESETS, TazitarConfig, TazitarLLM  # noqa: F401
from .vasolix import VASOLIX_PRESETS, VasolixConfig, VasolixLLM  # noqa: F401

# "architecture" of a config.json -> (configuration class, model class); configurations without that key are read as
# Hugging Face ones (DenseLLM / Qwen3MoE).
ARCHITECTURES = {"Vasolix": (VasolixConfig, VasolixLLM), "Lisenex": (LisenexConfig, LisenexLLM), "Tazitar": (TazitarConfig, TazitarLLM),
                 "Bagasun": (BagasunConfig, BagasunLLM)}


def all_presets() -> dict:
    return {**PRESETS, **VASOLIX_PRESETS, **LISENEX_PRESETS, **TAZITAR_PRESETS, **BAGASUN_PRESETS}


class AutoLLM:
    """``AutoLLM.from_pretrained(ModelConfig)`` picks the model class (python/triton_dist/models/__init__.py:33-59)."""

    @staticmethod
    def from_pretrained(model_config: ModelConfig, group=None):
        arch = model_config.arch()
        for config_cls, model_cls in ARCHITECTURES.values():
            if isinstance(arch, config_cls):
                return model_cls(model_config, group)
        if arch.is_moe:
            from .qwen_moe import Qwen3MoE
            return Qwen3MoE(model_config, group)
        return DenseLLM(model_config, group)


def smoke_decode():
    """One prefill + two decode steps of a tiny Qwen3-shaped model, and of tiny layered ones, on the current device."""
    import torch

    from ..runtime import get_runtime

    rt = get_runtime()
    for name in ("tiny-dense", "tiny-vasolix", "tiny-lisenex", "tiny-tazitar", "tiny-bagasun"):
        cfg = ModelConfig(model_name=name, max_length=64, rank=rt.rank, world_size=rt.world_size)
        eng = Engine(cfg)
        eng.backend = "triton_dist_gemm_ar"
        ids = torch.randint(0, 1000, (2, 8), device=rt.device)
        out = eng.serve(ids, 3)
        assert out.shape == (2, 3)
