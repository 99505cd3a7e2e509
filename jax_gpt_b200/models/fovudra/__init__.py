from .config import FovudraConfig
from .engine import FovudraEngine
from .model import forward, generate, init_params, make_cache
from .weight_loader import load_from_state_dict, random_state_dict

__all__ = ["FovudraConfig", "FovudraEngine", "forward", "generate", "init_params", "make_cache", "load_from_state_dict",
           "random_state_dict"]
