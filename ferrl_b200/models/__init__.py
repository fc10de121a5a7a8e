"""Policy model families: dense Qwen3 / Llama-3.x, Qwen3.5/3.6 hybrid
(GatedDeltaNet + gated GQA, dense and MoE), dense Gemma, Galodra (latent
attention, gated post-norm layers) and Mifutar (Mamba-2 and distance-biased
attention, hyper-connections)."""
from .dense import DenseCachedDecoder, DenseGradModel, DenseSpec  # noqa: F401
from .lora import BaseQuantization, DenseLoraTargets, FusedLoraLinear, LoraSpec  # noqa: F401
from .llama import llama_spec  # noqa: F401
from .qwen3 import qwen3_8b_spec, qwen3_spec  # noqa: F401
from .galodra import GalodraGradModel, GalodraSpec, galodra_spec  # noqa: F401
from .bias_attention import BiasAttention, BiasAttentionDims  # noqa: F401
from .latent import LatentAttention, LatentDims  # noqa: F401
from .mamba2 import Mamba2, Mamba2Dims  # noqa: F401
from .mifutar import MifutarGradModel, MifutarSpec, mifutar_spec  # noqa: F401
