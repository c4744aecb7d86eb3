"""A small B200-native inference library for the Qwen3 dense decoder, the Taredra hybrid decoder,
the Disorax latent-attention mixture-of-experts decoder, the Zadunex state-space hybrid decoder, the
Fogizen decoder (chunked attention with mixed head scores beside time mixing, routed experts), the Zefapel decoder
(matrix memories, gated linear attention and latent attention with rotated keys, routed experts with identity experts)
and the Givizen decoder (windowed attention with distance biases, norms on the sublayers' outputs, routed experts whose
weights multiply their inputs).

From a model folder (config.json + safetensors) or seeded random weights to
generated tokens on one GPU: typed configuration and registry, weights by
tensor name, layers put together from parts, a paged cache with slots, one step
function, a generation loop with greedy and temperature sampling, and trace
replay. All arithmetic of the model runs in this package's own CUDA kernels.
"""

from .config import ConfigError, DisoraxConfig, FogizenConfig, GivizenConfig, Qwen3Config, TaredraConfig, ZadunexConfig, ZefapelConfig, read_config, register_architecture
from .engine import Engine, StepEntry
from .sampling import SamplingParams
from .weights import WeightError, write_model_folder

__version__ = "0.1.0"
__all__ = ["ConfigError", "DisoraxConfig", "FogizenConfig", "GivizenConfig", "Qwen3Config", "TaredraConfig", "ZadunexConfig", "ZefapelConfig", "read_config",
           "register_architecture", "Engine", "StepEntry",
           "SamplingParams", "WeightError", "write_model_folder"]
