from .config import MopalornConfig
from .engine import MopalornEngine
from .model import forward, generate, init_params, make_cache
from .weight_loader import load_from_state_dict, random_state_dict

__all__ = ["MopalornConfig", "MopalornEngine", "forward", "generate", "init_params", "make_cache", "load_from_state_dict",
           "random_state_dict"]
