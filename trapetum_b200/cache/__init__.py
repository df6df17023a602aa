from .slots import CacheError, CacheFull, Pool
from .kv import BothView, Cache, KVGroup, KVLineView, StateView, pages_for

__all__ = ["BothView", "Cache", "CacheError", "CacheFull", "KVGroup", "KVLineView", "Pool", "StateView", "pages_for"]
