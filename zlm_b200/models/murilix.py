"""Registers the Murilix architecture: ``Murilix`` -> ``MurilixConfig``.  As for every architecture the model is the
generic ``DecoderModel`` built from the specification the configuration lowers to: one norm for two sublayers side by
side, a convolution over time on what the mixer reads, latent attention with latent queries and latents shared between
layers, a gated recurrence, a feed-forward with a polynomial of normed powers or routed experts, and per-layer rows of
the tokens behind the sublayers, all of them registered parts that another design may name too."""
from ..config.murilix import ARCHITECTURE, MurilixConfig
from ..registry import register_architecture

register_architecture(ARCHITECTURE)(MurilixConfig)
