from .config import FikizenConfig, tiny_config_dict  # noqa: F401
from .decoder import FikizenDecoder  # noqa: F401
from .model import FikizenForCausalLM, build_fikizen  # noqa: F401
