from .config import TatizenConfig
from .model import TatizenModel, init_random_, load_into

__all__ = ["TatizenConfig", "TatizenModel", "init_random_", "load_into"]
