from . import fozelix, polosun, tonilix, vobotar
from .hybrid import HybridConfig, HybridModel
from .llama import GenerateConfig, LlamaConfig, LlamaModel, llama_local_to_hf_name
from .registry import architectures, load_config, load_model, load_pretrained
from .sampler import MT19937_64, Sampler, SamplingParams, sample_from_logits

__all__ = ["GenerateConfig", "HybridConfig", "HybridModel", "architectures", "load_config", "load_model", "load_pretrained",
           "LlamaConfig", "LlamaModel", "llama_local_to_hf_name", "MT19937_64", "Sampler",
           "SamplingParams", "sample_from_logits"]
