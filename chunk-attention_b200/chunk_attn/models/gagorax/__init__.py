from .configuration_gagorax import GagoraxConfig  # noqa: F401
from .modeling_gagorax import GagoraxForCausalLM  # noqa: F401
