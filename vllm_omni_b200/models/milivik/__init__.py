from .config import MilivikConfig, tiny_config_dict  # noqa: F401
from .decoder import MilivikDecoder  # noqa: F401
from .model import MilivikForCausalLM, build_milivik  # noqa: F401
