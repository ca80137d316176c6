from . import debuvik, dezolorn, fubolix, llama, rasezen, sorizen, tafesun  # registers Debuvik, Dezolorn, Fubolix, LlamaForCausalLM, Rasezen, Sorizen and Tafesun

__all__ = ["debuvik", "dezolorn", "fubolix", "llama", "rasezen", "sorizen", "tafesun"]
