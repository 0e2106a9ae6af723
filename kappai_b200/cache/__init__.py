from .spec import CompositeSpec, PagedKVSpec, StateSpec, leaf_specs
from .manager import (CacheManager, PagePool, SlotPool, CacheError, OutOfPages, OutOfSlots, RELEASED)

__all__ = ["PagedKVSpec", "StateSpec", "CompositeSpec", "leaf_specs", "CacheManager", "PagePool", "SlotPool", "CacheError", "OutOfPages",
           "OutOfSlots", "RELEASED"]
