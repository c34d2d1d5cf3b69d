"""Fimodra adapter: text only, no adapters, 16-bit (or 32-bit) cache rows, long prefill chunks.  Recurrent state cannot
be restored from cached KV blocks, so the prefix cache stays off."""
from ..engine.errors import InvalidRequestError
from .base import ModelAdapter, ModelCapabilities, RuntimeModelPolicy


class FimodraAdapter(ModelAdapter):
    name = "fimodra"

    @classmethod
    def matches(cls, arch) -> bool:
        return arch.family == "fimodra"

    def runtime_policy(self, runtime_config) -> RuntimeModelPolicy:
        return RuntimeModelPolicy(force_kv_cache_dtype="model", prefill_chunk_size=2048)

    def detect(self, model) -> ModelCapabilities:
        return ModelCapabilities(supports_lora=False, supports_multimodal=False, supports_prefix_cache=False)

    def validate_request(self, sampling_params, prompt_len, lora_request=None, multi_modal_data=None) -> None:
        if lora_request is not None:
            raise InvalidRequestError("this model does not support LoRA adapters")
        if multi_modal_data:
            raise InvalidRequestError("this model is text only")
