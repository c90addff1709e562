from .config import NipuraxConfig
from .model import NipuraxModel, init_random_, load_into

__all__ = ["NipuraxConfig", "NipuraxModel", "init_random_", "load_into"]
