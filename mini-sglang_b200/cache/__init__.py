from .manager import CacheManager, KVGroup, OutOfSlots, PagedKVNeed, StateNeed, keys_seen
from .pages import OutOfPages, PagePool
from .radix import PrefixTree

__all__ = ["CacheManager", "KVGroup", "OutOfSlots", "PagedKVNeed", "StateNeed", "keys_seen", "OutOfPages", "PagePool", "PrefixTree"]
