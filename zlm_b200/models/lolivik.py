"""Registers the Lolivik architecture: ``Lolivik`` -> ``LolivikConfig``.  As for every architecture the model is the
generic ``DecoderModel`` built from the specification the configuration lowers to: attention with a bias by distance and a
temperature, attention over a window and the first tokens, values shared between layers, a matrix memory, clamped gated
experts beside a shared one, norms on the sublayers' outputs times a constant, all of them registered parts that another
design may name too."""
from ..config.lolivik import ARCHITECTURE, LolivikConfig
from ..registry import register_architecture

register_architecture(ARCHITECTURE)(LolivikConfig)
