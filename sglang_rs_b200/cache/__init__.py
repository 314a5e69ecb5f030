from .manager import (CacheManager, JointLayerCache, OutOfPages, OutOfStateSlots, PageAllocator, PagedLayerCache, RequestCache,
                      StateLayerCache, group_key)

from .radix import PrefixTree

__all__ = ["PrefixTree", "CacheManager", "JointLayerCache", "OutOfPages", "OutOfStateSlots", "PageAllocator", "PagedLayerCache", "RequestCache",
           "StateLayerCache", "group_key"]
