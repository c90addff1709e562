from .config import KivezenConfig
from .model import KivezenModel, init_random_, load_into

__all__ = ["KivezenConfig", "KivezenModel", "init_random_", "load_into"]
