from .configuration_bikelix import BikelixConfig  # noqa: F401
from .modeling_bikelix import BikelixForCausalLM  # noqa: F401
