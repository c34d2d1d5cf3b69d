"""Luzerax adapter: text only, no adapters, 16-bit (or 32-bit) cache rows, long prefill chunks.  Everything a request
leaves behind lives in its KV pages, so cached prefixes can be used."""
from .base import ModelAdapter, ModelCapabilities
from .fimodra import FimodraAdapter


class LuzeraxAdapter(FimodraAdapter):
    name = "luzerax"

    @classmethod
    def matches(cls, arch) -> bool:
        return arch.family == "luzerax"

    def detect(self, model) -> ModelCapabilities:
        return ModelAdapter.detect(self, model)
