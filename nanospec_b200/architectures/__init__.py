from . import debuvik, dezolorn, fubolix, llama, rasezen, sorizen  # registers Debuvik, Dezolorn, Fubolix, LlamaForCausalLM, Rasezen and Sorizen

__all__ = ["debuvik", "dezolorn", "fubolix", "llama", "rasezen", "sorizen"]
