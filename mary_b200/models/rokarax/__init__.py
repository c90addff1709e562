from .config import RokaraxConfig
from .model import RokaraxModel, init_random_, load_into

__all__ = ["RokaraxConfig", "RokaraxModel", "init_random_", "load_into"]
