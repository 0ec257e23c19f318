from . import fevosun, llama, mivorax, nufasun, risizen, samulorn, vibunex  # noqa: F401  (register "Fevosun", "LlamaForCausalLM", "Mivorax", "Nufasun", "Risizen", "Samulorn", "Vibunex")
from .model import Model
