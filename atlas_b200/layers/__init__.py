"""Decoder building blocks: attention, Gated DeltaNet, dense FFN, MoE, MTP head."""
from .common import ParallelCtx, make_weight, randn_weight  # noqa: F401
from .attention import Attention  # noqa: F401
from .mla import MLAttention  # noqa: F401
from .mlp import DenseMLP  # noqa: F401
from .moe import MoE  # noqa: F401
from .gdn import GatedDeltaNet  # noqa: F401
from .mamba2 import Mamba2Mixer  # noqa: F401
from .wkv import WKVMixer  # noqa: F401
from .mlstm import MLSTMMixer  # noqa: F401
from .latent import LatentAttention  # noqa: F401
from .rglru import RGLRUMixer  # noqa: F401
from .differential import DifferentialAttention  # noqa: F401
from .convolution import InputConvolution  # noqa: F401
from .side import TokenSide  # noqa: F401
from .gating import SublayerGate  # noqa: F401
from .parallel import ParallelMixer  # noqa: F401
from .hyper import HyperConnection  # noqa: F401

# mixers a layer listed in ``ModelConfig.layer_specs`` can have
MIXERS = {"attention": Attention, "mamba2": Mamba2Mixer, "wkv": WKVMixer, "parallel": ParallelMixer, "mlstm": MLSTMMixer,
          "latent_attention": LatentAttention, "rglru": RGLRUMixer, "differential": DifferentialAttention}
