from . import diforax, fobatar, futezen, gukosun, kemitar, lfm2, vugipel  # noqa: F401  (register the architectures)
from .diforax import DiforaxForCausalLM
from .fobatar import FobatarForCausalLM
from .futezen import FutezenForCausalLM
from .gukosun import GukosunForCausalLM
from .kemitar import KemitarForCausalLM
from .lfm2 import Lfm2ForCausalLM
from .vugipel import VugipelForCausalLM

__all__ = ["DiforaxForCausalLM", "FobatarForCausalLM", "FutezenForCausalLM", "GukosunForCausalLM", "KemitarForCausalLM", "Lfm2ForCausalLM",
           "VugipelForCausalLM"]
