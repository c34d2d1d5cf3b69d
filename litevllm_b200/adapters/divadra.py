"""Divadra adapter: text only, no adapters, 16-bit (or 32-bit) cache rows, long prefill chunks.  Recurrent state cannot
be restored from cached KV blocks, so the prefix cache stays off."""
from .fimodra import FimodraAdapter


class DivadraAdapter(FimodraAdapter):
    name = "divadra"

    @classmethod
    def matches(cls, arch) -> bool:
        return arch.family == "divadra"
