from . import duratar, fegidra, fudelorn, kodulix, llama, logirax, pozirax  # noqa: F401  (registers Duratar, Fegidra, Fudelorn, Kodulix, LlamaForCausalLM, Logirax, Pozirax)
from .registry import Architecture, architecture_names, register_architecture, resolve, unregister_architecture

__all__ = ["Architecture", "architecture_names", "register_architecture", "resolve", "unregister_architecture"]
