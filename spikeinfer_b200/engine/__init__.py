"""Decode-side engine pieces: the paged pools, the on-GPU batch state and its host-side block ledger."""
from .batch_state import DecodeBatchState
from .block_ledger import BlockLedger
from .kv_state_cache import PagedKVStateCache
from .spike_cache import PagedSpikeCache

__all__ = ["DecodeBatchState", "BlockLedger", "PagedSpikeCache", "PagedKVStateCache", "PagedDecodeEngine", "SpikeDecodeEngine"]


def __getattr__(name):
    if name in ("PagedDecodeEngine", "SpikeDecodeEngine"):  # imported lazily: they pull in the attention operators
        from . import decode_engine

        return getattr(decode_engine, name)
    raise AttributeError(name)
