from .cache import PAGE_SIZE, Cache, CacheEntries, CacheEntry, CacheSpec, KVGroup, KVSpec, StateGroup, StateSpec, shared_spec
from .pages import CacheError, CacheFull, PagePool, SlotTable

__all__ = ["PAGE_SIZE", "Cache", "CacheEntries", "CacheEntry", "CacheSpec", "KVGroup", "KVSpec", "StateGroup", "StateSpec",
           "shared_spec", "CacheError", "CacheFull", "PagePool", "SlotTable"]
