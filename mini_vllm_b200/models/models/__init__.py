from .fupupel import FupupelForCausalLM
from .gemma3 import Gemma3ForCausalLM
from .qwen3 import Qwen3ForCausalLM
from .rasezen import RasezenForCausalLM
from .sunulorn import SunulornForCausalLM
from .vebonex import VebonexForCausalLM

_MODELS = {"Qwen3ForCausalLM": Qwen3ForCausalLM, "Gemma3ForCausalLM": Gemma3ForCausalLM, "Fupupel": FupupelForCausalLM,
           "Vebonex": VebonexForCausalLM, "Sunulorn": SunulornForCausalLM, "Rasezen": RasezenForCausalLM}


def get_model_class(architecture: str):
    return _MODELS.get(architecture)
