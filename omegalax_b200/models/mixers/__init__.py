"""Token mixers and feed-forwards of decoders with an fp32 residual stream.

A mixer's config has ``cache_spec()`` (what it keeps per token or per sequence, see
``paged_sequences``), its module ``forward(h, batch, store, x)``: h are the normed rows, ``batch`` the ``TokenBatch`` of the call,
``store`` the layer's cache tensor, and the result is added into the fp32 rows x.
"""
from .batch import TokenBatch
from .feed_forward import DenseMLPConfig, GatedMLP, GatedMLPConfig, MixtureOfExperts, MixtureOfExpertsConfig, SquaredReluMLP
from .gated_linear_attention import GatedLinearAttention, GatedLinearAttentionConfig
from .latent_attention import LatentAttention, LatentAttentionConfig
from .layers import LayerNorm, Projection, RMSNorm
from .window_attention import WindowAttention, WindowAttentionConfig

__all__ = ["TokenBatch", "DenseMLPConfig", "GatedMLP", "GatedMLPConfig", "MixtureOfExperts", "MixtureOfExpertsConfig",
           "SquaredReluMLP", "GatedLinearAttention", "GatedLinearAttentionConfig", "LatentAttention", "LatentAttentionConfig",
           "LayerNorm", "Projection", "RMSNorm", "WindowAttention", "WindowAttentionConfig"]
