"""Model families and the preset zoo."""
from .config import (ModelConfig, LlamaConfig, MistralConfig, Qwen2Config, DeepSeekV2Config, get_model_config,  # noqa: F401
                     config_from_name, extend_context, list_models)
from .llama import LlamaForCausalLM, MistralForCausalLM, Qwen2ForCausalLM, create_model  # noqa: F401


def build_model(cfg, dtype=None, device=None):
    """Instantiate the model class that ``cfg.architecture`` names."""
    arch = cfg.architecture
    if arch == "transformer":
        return LlamaForCausalLM(cfg, dtype=dtype, device=device)
    if arch == "mamba2":
        from .mamba2 import Mamba2ForCausalLM
        return Mamba2ForCausalLM(cfg, dtype=dtype, device=device)
    if arch == "hss_ser":
        from .hss_ser import HSSSERForCausalLM
        return HSSSERForCausalLM(cfg, dtype=dtype, device=device)
    if arch == "deepseek_moe":
        from .deepseek import DeepSeekV2ForCausalLM
        return DeepSeekV2ForCausalLM(cfg, dtype=dtype, device=device)
    hybrid = _hybrid_class(arch)
    if hybrid is not None:
        return hybrid(cfg, dtype=dtype, device=device)
    raise ValueError(f"unknown architecture '{arch}'")


def _hybrid_class(arch):
    """Class of a hybrid decoder family, None for other architectures."""
    if arch == "rilenex":
        from .rilenex import RilenexForCausalLM
        return RilenexForCausalLM
    if arch == "tibalorn":
        from .tibalorn import TibalornForCausalLM
        return TibalornForCausalLM
    return None


def complete_config(cfg, tensors):
    """Fill in the sizes that a checkpoint gives only through its tensors' shapes (a no-op for most families)."""
    hybrid = _hybrid_class(cfg.architecture)
    return hybrid.config_from_tensors(cfg, tensors) if hybrid is not None else cfg
