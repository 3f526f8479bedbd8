from .config import TavulixConfig, tiny_config_dict  # noqa: F401
from .decoder import TavulixDecoder  # noqa: F401
from .model import TavulixForCausalLM, build_tavulix  # noqa: F401
