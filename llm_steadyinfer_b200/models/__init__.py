from . import fevosun, llama, mivorax, nufasun, risizen, vibunex  # noqa: F401  (register "Fevosun", "LlamaForCausalLM", "Mivorax", "Nufasun", "Risizen", "Vibunex")
from .model import Model
