"""Typed configuration of the Lolivik architecture, read from its own ``config.json`` keys, and its lowering to a
``ModelSpec``.

A Lolivik config.json names the design with a string and lists its layers one by one; layers of one model may differ
in kind and in every size:

    {"architecture": "Lolivik", "vocab": V, "width": W, "norm": {"eps": e}, "residual_mult": m,
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "softcap", "bias_max",
                           "q_temp": {"coef", "every"}, "v_mix": true | false},
                 "mlp": null | {"kind": "dense", "ff": F}},
                {"type": "attention_2",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size", "keep_first"},
                           "rot": {"base", "dims", "scaling": {"factor", "original", "low", "high"}}, "v_mix"},
                 "mlp": {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top"},
                         "shared": {"ff", "limit"}}},
                {"type": "mlstm", "mixer": {"heads", "dim", "vdim", "gate_cap"}, "mlp": ...}]}

The design.  Sublayers read the stream as it is, and what they give is normed, multiplied by one constant and added:
x += m * norm1(mixer(x)), x += m * norm2(ff(x)).  An ``attention`` mixer sees every earlier token without rotation: q and
k normed over the whole projection, q multiplied by a temperature that grows with the logarithm of the position, capped
scores, a learned bias by distance and a learned sink per head.  An ``attention_2`` mixer sees a sliding window and the
sequence's first tokens: norms per head, rotation of neighbouring pairs with frequencies scaled for long contexts,
ordinary softmax.  In both, layers that say ``v_mix`` blend the values of the first such layer into their own.  An
``mlstm`` mixer is a matrix memory with exponential gates.  The feed-forward is dense (tanh gelu of the gate) or a mixture
of clamped gated experts, chosen by softmax scores that are then divided by their sum, beside a shared expert.  A last
norm and an untied head give the logits.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple, Union

from .spec import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry, coerce, require

ARCHITECTURE = "Lolivik"
NO_POSITION_LIMIT = 1 << 24          # the design sets no longest sequence; the cache an engine is built with does
SWISH_ALPHA = 1.702                  # g sigmoid(1.702 g)


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


SCALING_KEYS = ("factor", "original", "low", "high")


@dataclass(frozen=True)
class RotaryConfig:
    base: float
    dims: int
    scaling: Optional[Tuple[float, float, float, float]] = None      # SCALING_KEYS

    @classmethod
    def from_dict(cls, d: Any, where: str, dim: int) -> Optional["RotaryConfig"]:
        if d is None:
            return None
        if not isinstance(d, Mapping):
            raise ConfigError(f"config.json: {where[:-1]} must be an object")
        scaling = None
        if d.get("scaling") is not None:
            sc = _mapping(d, "scaling", where)
            scaling = tuple(_req(sc, k, float, where + "scaling.") for k in SCALING_KEYS)
            if min(scaling) <= 0:
                raise ConfigError(f"config.json: {where}scaling: {', '.join(SCALING_KEYS)} must be positive")
        c = cls(_req(d, "base", float, where), _req(d, "dims", int, where), scaling)
        if c.dims % 2 or not 0 <= c.dims <= dim:
            raise ConfigError(f"config.json: {where}dims={c.dims} must be even and at most dim={dim}")
        if c.base <= 0:
            raise ConfigError(f"config.json: {where}base={c.base}")
        return c if c.dims else None

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = dict(zip(SCALING_KEYS, self.scaling))
        return d

    def position(self) -> Dict[str, Any]:
        p: Dict[str, Any] = {"kind": "rope_interleaved", "base": self.base, "dims": self.dims}
        if self.scaling is not None:
            p["scaling"] = dict(zip(SCALING_KEYS, self.scaling))
        return p


def _head_sizes(d: Mapping[str, Any], where: str) -> Dict[str, Any]:
    heads = _req(d, "heads", int, where)
    s = {"heads": heads, "kv_heads": _opt(d, "kv_heads", int, where, heads), "dim": _req(d, "dim", int, where),
         "vdim": _req(d, "vdim", int, where), "scale": _req(d, "scale", float, where),
         "v_mix": _opt(d, "v_mix", bool, where, False)}
    if min(s["heads"], s["kv_heads"], s["dim"], s["vdim"]) <= 0:
        raise ConfigError(f"config.json: {where}sizes must be positive")
    if heads % s["kv_heads"]:
        raise ConfigError(f"config.json: {where}heads={heads} is not a multiple of kv_heads={s['kv_heads']}")
    return s


@dataclass(frozen=True)
class BiasedAttentionConfig:
    """``attention``: every earlier token, positions through a temperature and a bias by distance."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    v_mix: bool
    bias_max: int
    softcap: float = 0.0                              # 0: none
    q_temp: Optional[Tuple[float, int]] = None        # coef, every

    type = "attention"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "BiasedAttentionConfig":
        temp = None
        if d.get("q_temp") is not None:
            t = _mapping(d, "q_temp", where)
            temp = (_req(t, "coef", float, where + "q_temp."), _req(t, "every", int, where + "q_temp."))
            if temp[1] <= 0:
                raise ConfigError(f"config.json: {where}q_temp.every must be positive")
        c = cls(**_head_sizes(d, where), bias_max=_req(d, "bias_max", int, where),
                softcap=_opt(d, "softcap", float, where, 0.0), q_temp=temp)
        if c.bias_max <= 0 or c.softcap < 0:
            raise ConfigError(f"config.json: {where}bias_max={c.bias_max}, softcap={c.softcap}")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "scale": self.scale, "bias_max": self.bias_max, "v_mix": self.v_mix}
        if self.softcap:
            d["softcap"] = self.softcap
        if self.q_temp is not None:
            d["q_temp"] = dict(zip(("coef", "every"), self.q_temp))
        return d

    def params(self) -> Dict[str, Any]:
        return {"qk_norm": "row", "sink": True, "learned_sink": True, "softcap": self.softcap,
                "distance_bias": {"far": self.bias_max},
                "q_temp": None if self.q_temp is None else dict(zip(("coef", "every"), self.q_temp))}


@dataclass(frozen=True)
class WindowAttentionConfig:
    """``attention_2``: a sliding window beside the first tokens; ``window`` 0: every earlier token."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    v_mix: bool
    window: int = 0
    keep_first: int = 0
    rot: Optional[RotaryConfig] = None

    type = "attention_2"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "WindowAttentionConfig":
        sizes = _head_sizes(d, where)
        window = keep = 0
        if d.get("mask") is not None:
            m = _mapping(d, "mask", where)
            window, keep = _req(m, "size", int, where + "mask."), _opt(m, "keep_first", int, where + "mask.", 0)
            if window <= 0 or keep < 0:
                raise ConfigError(f"config.json: {where}mask: size={window}, keep_first={keep}")
        return cls(**sizes, window=window, keep_first=keep, rot=RotaryConfig.from_dict(d.get("rot"), where + "rot.", sizes["dim"]))

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "scale": self.scale, "v_mix": self.v_mix}
        if self.window:
            d["mask"] = {"size": self.window, "keep_first": self.keep_first}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d

    def params(self) -> Dict[str, Any]:
        return {"qk_norm": "head", "sink": False, "window": self.window, "keep": self.keep_first,
                "position": self.rot.position() if self.rot is not None else {"kind": "none"}}


@dataclass(frozen=True)
class MatrixMemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    type = "mlstm"
    v_mix = False

    @classmethod
    def from_dict(cls, d: Mapping[str, Any], where: str) -> "MatrixMemoryConfig":
        c = cls(_req(d, "heads", int, where), _req(d, "dim", int, where), _req(d, "vdim", int, where),
                _req(d, "gate_cap", float, where))
        if min(c.heads, c.dim, c.vdim) <= 0 or c.gate_cap <= 0:
            raise ConfigError(f"config.json: {where}sizes and gate_cap must be positive")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "gate_cap": self.gate_cap}


MIXER_TYPES = {c.type: c for c in (BiasedAttentionConfig, WindowAttentionConfig, MatrixMemoryConfig)}
MixerConfig = Union[BiasedAttentionConfig, WindowAttentionConfig, MatrixMemoryConfig]


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class ExpertsConfig:
    ff: int
    limit: float
    experts: int
    top: int
    shared: Optional[Tuple[int, float]] = None          # ff, limit

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit},
                             "router": {"experts": self.experts, "top": self.top}}
        if self.shared is not None:
            d["shared"] = dict(zip(("ff", "limit"), self.shared))
        return d


def _feed_forward(d: Any, where: str) -> Union[None, DenseConfig, ExpertsConfig]:
    if d is None:
        return None
    if not isinstance(d, Mapping):
        raise ConfigError(f"config.json: {where[:-1]} must be an object or null")
    kind = d.get("kind")
    if kind == "dense":
        c = DenseConfig(_req(d, "ff", int, where))
        if c.ff <= 0:
            raise ConfigError(f"config.json: {where}ff must be positive")
        return c
    if kind == "moe":
        def expert(key: str) -> Tuple[int, float]:
            m = _mapping(d, key, where)
            e = (_req(m, "ff", int, f"{where}{key}."), _req(m, "limit", float, f"{where}{key}."))
            if min(e) <= 0:
                raise ConfigError(f"config.json: {where}{key}: ff and limit must be positive")
            return e
        router = _mapping(d, "router", where)
        ff, limit = expert("expert")
        e = ExpertsConfig(ff, limit, _req(router, "experts", int, where + "router."), _req(router, "top", int, where + "router."),
                          expert("shared") if d.get("shared") is not None else None)
        if e.experts <= 0 or not 0 < e.top <= e.experts:
            raise ConfigError(f"config.json: {where}router.top={e.top} of {e.experts} experts")
        return e
    raise ConfigError(f"config.json: {where}kind={kind!r} is not known (dense, moe)")


@dataclass(frozen=True)
class LolivikLayer:
    mixer: MixerConfig
    mlp: Union[None, DenseConfig, ExpertsConfig]

    @property
    def type(self) -> str:
        return self.mixer.type


@dataclass(frozen=True)
class LolivikConfig:
    vocab_size: int
    width: int
    norm_eps: float
    layers: Tuple[LolivikLayer, ...]
    residual_mult: float = 1.0
    eos_token_ids: Tuple[int, ...] = ()

    # ---- reading -----------------------------------------------------------
    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "LolivikConfig":
        vocab, width = require(d, "vocab", int), require(d, "width", int)
        eps = require(_mapping(d, "norm", ""), "eps", float)
        if vocab <= 0 or width <= 0 or eps <= 0:
            raise ConfigError("config.json: vocab, width and norm.eps must be positive")
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers, first = [], None
        for i, l in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(l, Mapping):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = l.get("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}type={kind!r} is not known ({', '.join(MIXER_TYPES)})")
            m = MIXER_TYPES[kind].from_dict(_mapping(l, "mixer", where), where + "mixer.")
            if m.v_mix:
                first = first or (i, m.kv_heads * m.vdim)
                if m.kv_heads * m.vdim != first[1]:
                    raise ConfigError(f"config.json: {where}mixer: kv_heads * vdim = {m.kv_heads * m.vdim} values a token, but the "
                                      f"first layer with v_mix (layers[{first[0]}]) has {first[1]}")
            layers.append(LolivikLayer(m, _feed_forward(l.get("mlp"), where + "mlp.")))
        eos = d.get("eos_token_id")
        eos_ids = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(eos))
        return cls(vocab, width, eps, tuple(layers), _opt(d, "residual_mult", float, "", 1.0), eos_ids)

    # ---- writing -----------------------------------------------------------
    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {
            "architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.width, "norm": {"eps": self.norm_eps},
            "residual_mult": self.residual_mult,
            "layers": [{"type": l.type, "mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict()}
                       for l in self.layers],
        }
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d

    # ---- lowering ----------------------------------------------------------
    def _mixer(self, m: MixerConfig, prefix: str, role: Optional[str]) -> PartSpec:
        if isinstance(m, MatrixMemoryConfig):
            return PartSpec("mlstm", {"num_heads": m.heads, "head_dim": m.dim, "v_dim": m.vdim, "gate_cap": m.gate_cap,
                                      "norm_eps": self.norm_eps}, prefix=prefix,
                            rename={"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "g_proj.weight": "g",
                                    "o_proj.weight": "o", "norm.weight": "norm", "i_gate.weight": "i", "i_gate.bias": "i.b",
                                    "f_gate.weight": "f", "f_gate.bias": "f.b"})
        return PartSpec("conv_attention", {
            "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_dim": m.vdim, "conv_taps": 1, "conv": False,
            "gate": "none", "scale": m.scale, "norm_eps": self.norm_eps, "v_mix": role, **m.params()}, prefix=prefix,
            rename={"q_proj.weight": "q", "k_proj.weight": "k", "v_proj.weight": "v", "o_proj.weight": "o",
                    "q_norm.weight": "q.norm", "k_norm.weight": "k.norm", "bias": "rel", "sinks": "sink", "v_mix": "vmix"})

    def _ffn(self, f: Union[DenseConfig, ExpertsConfig], prefix: str) -> PartSpec:
        if isinstance(f, DenseConfig):
            return PartSpec("swiglu", {"intermediate_size": f.ff, "activation": "gelu_tanh"}, prefix=prefix,
                            rename={"gate_proj.weight": "gate", "up_proj.weight": "up", "down_proj.weight": "down"})
        shared = None if f.shared is None else {"intermediate_size": f.shared[0], "activation": "swish_limit",
                                                "limit": f.shared[1], "alpha": SWISH_ALPHA}
        return PartSpec("routed_experts", {
            "num_experts": f.experts, "top_k": f.top, "expert_ff": f.ff, "score": "softmax", "renormalize": True,
            "weight_on": "output", "activation": "swish_limit", "limit": f.limit, "alpha": SWISH_ALPHA, "shared": shared},
            prefix=prefix)

    def to_model_spec(self) -> ModelSpec:
        def norm(prefix: str, name: str, multiplier: float = 1.0) -> PartSpec:
            return PartSpec("rms_norm", {"eps": self.norm_eps, "multiplier": multiplier}, prefix=prefix, rename={"weight": name})
        layers, mixed = [], False
        for i, l in enumerate(self.layers):
            p, role = f"l{i}.", None
            if l.mixer.v_mix:
                role, mixed = ("reader" if mixed else "source"), True
            mixer = self._mixer(l.mixer, p + "mix.", role)
            if l.mlp is None:
                ffn, norm_f = PartSpec("none", {}), PartSpec("none", {})
            else:
                ffn, norm_f = self._ffn(l.mlp, p + "mlp."), norm(p, "norm2", self.residual_mult)
            layers.append(LayerSpec("sublayer_norm", mixer, ffn, norm(p, "norm1", self.residual_mult), norm_f))
        spec = ModelSpec(
            architecture=ARCHITECTURE, hidden_size=self.width, vocab_size=self.vocab_size,
            max_position=NO_POSITION_LIMIT, layers=tuple(layers),
            schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
            embedding=PartSpec("token_embedding", {}, rename={"weight": "embed"}),
            final_norm=norm("final.", "norm"),
            head=PartSpec("lm_head", {"tied": False}, rename={"weight": "head"}),
        )
        spec.validate()
        return spec
