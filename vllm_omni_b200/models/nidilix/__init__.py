from .config import NidilixConfig, tiny_config_dict  # noqa: F401
from .decoder import NidilixDecoder  # noqa: F401
from .model import NidilixForCausalLM, build_nidilix  # noqa: F401
