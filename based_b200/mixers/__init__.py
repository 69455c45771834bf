"""Drop-in mixer modules (same constructor / forward signatures and state layout as
based/models/mixers/linear_attention.py, slide_attention.py and convolution.py of the reference), and the mixers of hybrid
stacks (gated delta rule, real-gated linear recurrent unit, latent attention, grouped attention with keys as values,
linear attention with a constant decay)."""
from .linear_attention import FeatureMap, LinearAttention, TaylorExp  # noqa: F401
from .slide_attention import RotaryEmbedding, SlidingAttention  # noqa: F401
from .convolution import BaseConv, ShortConvolution  # noqa: F401
from .stateful import PackedLinear, StatefulMixer  # noqa: F401
from .gated_delta import GatedDelta  # noqa: F401
from .rglru import RGLRU  # noqa: F401
from .latent_attention import LatentAttention  # noqa: F401
from .grouped_attention import GroupedAttention  # noqa: F401
from .lightning import LightningAttention  # noqa: F401
