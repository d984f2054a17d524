from .decoder import DecoderModel, ScaledResidualDecoderModel, StreamDecoderModel
from .fezozen import FezozenForCausalLM
from .gulisun import GulisunForCausalLM
from .qwen3 import Qwen3ForCausalLM
from .ravutar import RavutarForCausalLM
from .sinulix import SinulixForCausalLM
from .tarupel import TarupelForCausalLM
from .zetonex import ZetonexForCausalLM

__all__ = ["DecoderModel", "ScaledResidualDecoderModel", "StreamDecoderModel", "FezozenForCausalLM", "GulisunForCausalLM",
           "Qwen3ForCausalLM", "RavutarForCausalLM", "SinulixForCausalLM", "TarupelForCausalLM",
           "ZetonexForCausalLM"]
