"""Typed configuration of the Murilix architecture, read from its own ``config.json`` keys, and its lowering to a
``ModelSpec``.

A Murilix config.json names the design with a string and lists its layers one by one; layers of one model may differ
in kind and in every size:

    {"architecture": "Murilix", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
     "canon": {"taps": n}, "token_side": {"dim": d},
     "layers": [{"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "mask": {"size": window},
                           "rot": {"base", "dims"}, "kv_from": an earlier layer (or absent)},
                 "mlp": null | {"kind": "dense", "ff": F}
                      | {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": k}}},
                {"type": "mingru", "mixer": {"width": w}, "mlp": ...}, ...]}

The design.  A layer has one norm, a layer norm without a bias, and both sublayers read its rows h: x += mixer(m) + ff(h).
The mixer's input is m = h + conv(h), a causal convolution of ``canon.taps`` taps over time on every channel.  A
``latent_attention`` mixer keeps one small normed latent and one rotated key part per token, its queries go through a
latent of their own, and it sees a sliding window; with ``kv_from`` it makes no latents but reads those of an earlier
layer, everything else its own.  A ``mingru`` mixer is a gated recurrence whose gates read the current token alone.  The
feed-forward is dense without a gate, its activation a polynomial of normed powers, or a mixture of gated silu experts
weighted by the softmax over the chosen experts' logits.  Every layer ends with the tokens' own rows of a side table
(``token_side.dim`` columns a layer), gated by the stream, projected, normed and added.  The embedding is scaled; a last
layer norm and the embedding table itself, unscaled, give the logits.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple, Union

from .spec import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry, coerce, require

ARCHITECTURE = "Murilix"
NO_POSITION_LIMIT = 1 << 24          # the design sets no longest sequence; the cache an engine is built with does


def _mapping(d: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    v = d.get(key)
    if not isinstance(v, Mapping):
        raise ConfigError(f"config.json: {where}'{key}' must be an object")
    return v


def _req(m: Mapping[str, Any], key: str, typ, where: str):
    if key not in m or m[key] is None:
        raise ConfigError(f"config.json: {where}missing key '{key}'")
    return coerce(m[key], where + key, typ)


def _opt(m: Mapping[str, Any], key: str, typ, where: str, default):
    return default if m.get(key) is None else coerce(m[key], where + key, typ)


@dataclass(frozen=True)
class LatentMixerConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int                       # 0: no rotation
    window: int = 0                     # 0: every earlier token
    kv_from: Optional[int] = None       # the layer whose latents and rotated keys this one reads

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "LatentMixerConfig":
        rot_dim = _req(d, "rot_dim", int, where)
        base, dims = 10000.0, 0
        if d.get("rot") is not None:
            rot = _mapping(d, "rot", where)
            base, dims = _req(rot, "base", float, where + "rot."), _req(rot, "dims", int, where + "rot.")
        if dims % 2 or not 0 <= dims <= rot_dim:
            raise ConfigError(f"config.json: {where}rot.dims={dims} must be even and at most rot_dim={rot_dim}")
        if base <= 0:
            raise ConfigError(f"config.json: {where}rot.base must be positive")
        window = 0
        if d.get("mask") is not None:
            window = _req(_mapping(d, "mask", where), "size", int, where + "mask.")
            if window <= 0:
                raise ConfigError(f"config.json: {where}mask.size must be positive")
        c = cls(_req(d, "heads", int, where), _req(d, "dim", int, where), rot_dim, _req(d, "vdim", int, where),
                _req(d, "q_rank", int, where), _req(d, "kv_rank", int, where), _req(d, "scale", float, where), base, dims,
                window, _opt(d, "kv_from", int, where, None))
        if min(c.heads, c.vdim, c.q_rank, c.kv_rank) <= 0 or c.dim < 0 or c.rot_dim < 0 or c.dim + c.rot_dim <= 0:
            raise ConfigError(f"config.json: {where}sizes must be positive")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim,
                             "q_rank": self.q_rank, "kv_rank": self.kv_rank, "scale": self.scale}
        if self.rot_dims:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        if self.window:
            d["mask"] = {"size": self.window}
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        return d

    @property
    def record(self) -> Tuple:
        """What a layer and the layer whose latents it reads must agree on."""
        return (self.kv_rank, self.rot_dim, self.rot_dims, self.rot_base if self.rot_dims else None)


@dataclass(frozen=True)
class MinGRUConfig:
    width: int

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "MinGRUConfig":
        c = cls(_req(d, "width", int, where))
        if c.width <= 0:
            raise ConfigError(f"config.json: {where}width must be positive")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"width": self.width}


@dataclass(frozen=True)
class FeedForwardConfig:
    ff: int
    experts: int = 0                    # 0: dense
    top: int = 0

    @classmethod
    def from_dict(cls, d: Any, where: str) -> Optional["FeedForwardConfig"]:
        if d is None:
            return None
        if not isinstance(d, Mapping):
            raise ConfigError(f"config.json: {where[:-1]} must be an object or null")
        kind = d.get("kind")
        if kind == "dense":
            c = cls(_req(d, "ff", int, where))
        elif kind == "moe":
            r = _mapping(d, "router", where)
            c = cls(_req(_mapping(d, "expert", where), "ff", int, where + "expert."),
                    _req(r, "experts", int, where + "router."), _req(r, "top", int, where + "router."))
            if not 0 < c.top <= c.experts:
                raise ConfigError(f"config.json: {where}router.top={c.top} of {c.experts} experts")
        else:
            raise ConfigError(f"config.json: {where}kind={kind!r} is not known (dense, moe)")
        if c.ff <= 0:
            raise ConfigError(f"config.json: {where}ff must be positive")
        return c

    def to_dict(self) -> Dict[str, Any]:
        if not self.experts:
            return {"kind": "dense", "ff": self.ff}
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class MurilixLayer:
    mixer: Union[LatentMixerConfig, MinGRUConfig]
    mlp: Optional[FeedForwardConfig]

    @property
    def type(self) -> str:
        return "latent_attention" if isinstance(self.mixer, LatentMixerConfig) else "mingru"


@dataclass(frozen=True)
class MurilixConfig:
    vocab_size: int
    width: int
    norm_eps: float
    taps: int
    side_dim: int
    layers: Tuple[MurilixLayer, ...]
    embedding_scale: float = 1.0
    eos_token_ids: Tuple[int, ...] = ()

    # ---- reading -----------------------------------------------------------
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "MurilixConfig":
        vocab, width = require(d, "vocab", int), require(d, "width", int)
        eps = _req(_mapping(d, "norm", ""), "eps", float, "norm.")
        taps = _req(_mapping(d, "canon", ""), "taps", int, "canon.")
        dim = _req(_mapping(d, "token_side", ""), "dim", int, "token_side.")
        if min(vocab, width, taps, dim) <= 0 or eps <= 0:
            raise ConfigError("config.json: vocab, width, norm.eps, canon.taps and token_side.dim must be positive")
        scale = 1.0
        if d.get("embedding") is not None:
            scale = _opt(_mapping(d, "embedding", ""), "scale", float, "embedding.", 1.0)
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, l in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(l, Mapping):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = l.get("type")
            m = _mapping(l, "mixer", where)
            if kind == "latent_attention":
                mixer: Union[LatentMixerConfig, MinGRUConfig] = LatentMixerConfig.from_dict(m, where + "mixer.")
                j = mixer.kv_from
                if j is not None:
                    if not 0 <= j < i or not isinstance(layers[j].mixer, LatentMixerConfig) or layers[j].mixer.kv_from is not None:
                        raise ConfigError(f"config.json: {where}mixer.kv_from={j} must name an earlier latent_attention layer "
                                          f"with latents of its own")
                    if layers[j].mixer.record != mixer.record:
                        raise ConfigError(f"config.json: {where}mixer.kv_from={j}: kv_rank, rot_dim and rot must be that layer's")
            elif kind == "mingru":
                mixer = MinGRUConfig.from_dict(m, where + "mixer.")
            else:
                raise ConfigError(f"config.json: {where}type={kind!r} is not known (latent_attention, mingru)")
            layers.append(MurilixLayer(mixer, FeedForwardConfig.from_dict(l.get("mlp"), where + "mlp.")))
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(eos))
        return cls(vocab, width, eps, taps, dim, tuple(layers), scale, eos_ids)

    # ---- writing -----------------------------------------------------------
    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {
            "architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.width, "norm": {"eps": self.norm_eps},
            "embedding": {"scale": self.embedding_scale}, "canon": {"taps": self.taps}, "token_side": {"dim": self.side_dim},
            "layers": [{"type": l.type, "mixer": l.mixer.to_dict(), "mlp": l.mlp.to_dict() if l.mlp else None}
                       for l in self.layers],
        }
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ---- lowering ----------------------------------------------------------
    def _mixer_spec(self, m: Union[LatentMixerConfig, MinGRUConfig], prefix: str) -> PartSpec:
        if isinstance(m, MinGRUConfig):
            return PartSpec("mingru", {"width": m.width}, prefix=prefix, rename={
                "z_proj.weight": "z", "z_proj.bias": "z.b", "x_proj.weight": "x", "x_proj.bias": "x.b", "g_proj.weight": "g",
                "o_proj.weight": "o"})
        position = ({"kind": "rope_interleaved", "base": m.rot_base, "dims": m.rot_dims} if m.rot_dims else {"kind": "none"})
        return PartSpec("latent_attention", {
            "num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "v_dim": m.vdim, "kv_rank": m.kv_rank,
            "q_rank": m.q_rank, "scale": m.scale, "norm_eps": self.norm_eps, "window": m.window, "position": position,
            "kv_proj": m.kv_from is None}, prefix=prefix)

    def _feed_forward_spec(self, f: Optional[FeedForwardConfig], prefix: str) -> PartSpec:
        if f is None:
            return PartSpec("none", {})
        if f.experts:
            return PartSpec("routed_experts", {
                "num_experts": f.experts, "top_k": f.top, "expert_ff": f.ff, "score": "softmax", "renormalize": True,
                "weight_on": "output", "activation": "swiglu"}, prefix=prefix)
        return PartSpec("poly_norm", {"intermediate_size": f.ff, "norm_eps": self.norm_eps}, prefix=prefix,
                        rename={"up_proj.weight": "up", "down_proj.weight": "down"})

    def to_model_spec(self) -> ModelSpec:
        def norm(prefix: str, name: str) -> PartSpec:
            return PartSpec("layer_norm", {"eps": self.norm_eps}, prefix=prefix, rename={"weight": name})
        layers, n = [], len(self.layers)
        for i, l in enumerate(self.layers):
            p = f"l{i}."
            side = PartSpec("gated_token_input", {
                "vocab_size": self.vocab_size, "dim": self.side_dim, "offset": i * self.side_dim,
                "table_width": n * self.side_dim, "norm": {"kind": "rms_norm", "eps": self.norm_eps}},
                rename={"table": "side.embed", "gate": p + "side.gate", "proj": p + "side.proj", "norm.weight": p + "side.norm"})
            layers.append(LayerSpec(
                "parallel_sublayers", self._mixer_spec(l.mixer, p + "mix."), self._feed_forward_spec(l.mlp, p + "mlp."),
                norm(p, "norm1"), PartSpec("none", {}),
                mixer_input=PartSpec("causal_conv", {"taps": self.taps}, prefix=p, rename={"weight": "canon1"}),
                layer_input=side))
        spec = ModelSpec(
            architecture=ARCHITECTURE, hidden_size=self.width, vocab_size=self.vocab_size,
            max_position=NO_POSITION_LIMIT, layers=tuple(layers),
            schedule=tuple(ScheduleEntry(i, cache_of=getattr(l.mixer, "kv_from", None)) for i, l in enumerate(self.layers)),
            embedding=PartSpec("token_embedding", {"scale": self.embedding_scale}, rename={"weight": "embed"}),
            final_norm=norm("final.", "norm"),
            head=PartSpec("lm_head", {"tied": True}, rename={"weight": "head"}),
        )
        spec.validate()
        return spec
