"""Small Lolivik configurations and weights for the tests, and the oracle's inputs.

The configurations differ from each other, and from layer to layer, in every size and option: head counts (1, 2, 3, 5, 18)
over one, some or all key heads, key and value sizes that differ and are no multiples of 16 (and that are, 128 among them),
bias tables of 6 to 32 rows up to distances of 20 to 300, windows below a page, a little above one and above two, none,
kept first tokens of none, a few, a page, a little more than a page, rotation of a part of a head, all of it and none, with
scaled frequencies and without, caps on the scores and none, temperatures and none, values mixed from an attention layer of
either kind, or not at all, matrix memories of odd and even sizes, dense and routed feed-forwards and a layer without one,
one to all experts a token, with a shared expert and without.

Weights are drawn so that activations are of order one (matrices N(0, 1/in)) and attention is peaked: routing, gates and
attention then depend visibly on single keys and experts, which N(0, 0.02) would hide."""
from __future__ import annotations

import copy
import json
import os
from typing import Dict, List, Sequence

import torch

import plain_lolivik as P


def att(heads, kv_heads, dim, vdim, scale, bias_max, softcap=0.0, temp=None, v_mix=False):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max, "v_mix": v_mix}
    if softcap:
        m["softcap"] = softcap
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return m


def win(heads, kv_heads, dim, vdim, scale, window=0, keep=0, rot=None, v_mix=False):
    """rot: (base, dims) or (base, dims, factor, original, low, high)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "low", "high"), rot[2:]))
    return m


def mem(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, limit=0.8, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        d["shared"] = {"ff": shared[0], "limit": shared[1]}
    return d


def layer(mixer, mlp):
    kind = "mlstm" if "gate_cap" in mixer else ("attention" if "bias_max" in mixer else "attention_2")
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def model(layers, vocab, width, mult=0.6, eps=1e-5):
    return {"architecture": "Lolivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult,
            "layers": layers}


LOLI_A = model([
    layer(att(6, 2, 24, 20, 0.3, 40, softcap=5.0, temp=(0.3, 16), v_mix=True), dense(40)),
    layer(mem(3, 24, 20, 6.0), moe(24, 8, 3, 0.8, (40, 1.2))),
    layer(win(4, 2, 40, 20, 0.25, 70, 5, rot=(10000.0, 16, 8.0, 60, 1.0, 4.0), v_mix=True), moe(16, 6, 1, 1.1, (24, 0.7))),
    layer(att(5, 1, 16, 40, 0.4, 300, temp=(0.2, 50), v_mix=True), None),
    layer(mem(2, 40, 48, 15.0), dense(72)),
    layer(win(2, 1, 16, 24, 0.4, 9, 2, rot=(500.0, 16)), dense(24)),
], vocab=160, width=64)
# wider; the sizes that the tensor-core kernels take; 18 heads over one; kept tokens over more than a page; values mixed from
# a window layer; all experts of a router chosen; no shared expert
LOLI_B = model([
    layer(mem(2, 128, 64, 10.0), moe(48, 4, 4, 1.5)),
    layer(win(4, 2, 128, 128, 0.09, 130, 70, rot=(1e5, 32)), dense(96)),
    layer(win(2, 1, 64, 32, 0.12, 40, 64, v_mix=True), moe(8, 12, 4, 0.6, (64, 2.0))),
    layer(att(18, 1, 32, 32, 0.2, 60, softcap=8.0, v_mix=True), None),
    layer(att(4, 2, 128, 128, 0.09, 128, softcap=10.0, temp=(0.4, 32)), moe(64, 7, 2, 1.0, (32, 1.0))),
], vocab=200, width=128, mult=0.5, eps=1e-6)
# sizes that no kernel likes: odd heads, dims, feed-forwards and memories
LOLI_C = model([
    layer(att(3, 3, 7, 5, 0.4, 20, softcap=3.0, temp=(0.5, 7)), dense(37)),
    layer(mem(3, 9, 13, 4.0), moe(11, 3, 2, 0.7, (13, 0.9))),
    layer(win(5, 1, 9, 3, 0.4, 33, 1, rot=(300.0, 6, 4.0, 30, 1.0, 2.0)), None),
    layer(mem(1, 37, 6, 8.0), moe(9, 4, 4, 0.9)),
], vocab=77, width=40, mult=0.8, eps=1e-4)
# every layer mixes or none of the later ones does; a window layer without a window
LOLI_D = model([
    layer(win(2, 2, 16, 16, 0.4, 20, 3, rot=(1000.0, 8), v_mix=True), moe(32, 5, 4, 0.9, (16, 1.0))),
    layer(att(4, 4, 16, 8, 0.4, 25, temp=(0.6, 5), v_mix=True), moe(16, 4, 1, 1.0, (24, 0.8))),
    layer(win(3, 1, 32, 16, 0.3, rot=(1000.0, 32)), dense(24)),
], vocab=96, width=48, mult=0.7)
LOLI = {"A": LOLI_A, "B": LOLI_B, "C": LOLI_C, "D": LOLI_D}


def bias_rows(cfg) -> int:
    """Rows of a model's bias tables (a checkpoint's affair, not the configuration's)."""
    return {160: 16, 200: 32, 77: 6, 96: 12}.get(cfg["vocab"], 10)


def make_tensors(cfg_dict, seed: int) -> Dict[str, torch.Tensor]:
    """fp32 tensors by checkpoint name, every one rounded to bfloat16 values (so that both engine dtypes and the
    oracle compute on the same numbers)."""
    from zlm_b200.parts.model import DecoderModel
    from zlm_b200.registry import config_from_dict
    specs = DecoderModel(config_from_dict(cfg_dict).to_model_spec()).param_specs()
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name in sorted(specs):
        shape = tuple(bias_rows(cfg_dict) if s == -1 else s for s in specs[name].shape)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif last == "b":
            t = torch.randn(shape, generator=g) + (2.5 if name.endswith("f.b") else 0.0)      # memories that last
        elif last == "vmix":
            t = 0.3 + 0.4 * torch.rand(shape, generator=g)
        elif last in ("rel", "sink"):
            t = 1.2 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / shape[-1] ** 0.5
            if last == "router":
                t = t * ROUTER_GAIN
        out[name] = t.to(torch.bfloat16).float()
    return out


def write_model(tmp_path, cfg, tensors, tag: str):
    from zlm_b200.weights import write_safetensors
    folder = os.path.join(str(tmp_path), f"loli_{tag}")
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {n: t.to(torch.bfloat16) for n, t in tensors.items()})
    return folder


def make_model(tmp_path, name: str, seed: int = 0):
    """Writes the model to a folder; returns (folder, config mapping, float64 tensors for the oracle)."""
    cfg = LOLI[name]
    tensors = make_tensors(cfg, seed)
    return write_model(tmp_path, cfg, tensors, f"{name}_{seed}"), cfg, {n: t.double() for n, t in tensors.items()}


def one_layer(mixer, mlp=None, width=64, vocab=100, mult=0.8):
    """A model of one layer around the mechanism under test."""
    return model([layer(mixer, mlp)], vocab, width, mult)


def engine_for(tmp_path, cfg, tensors, dtype, tag, **kw):
    from zlm_b200 import Engine
    kw.setdefault("max_tokens", 2048)
    return Engine.from_pretrained(write_model(tmp_path, cfg, tensors, tag), dtype=dtype, **kw)


# how far a bfloat16 run's router logits may be from the oracle's
CLOSE_CALL = 0.08
# how little may be left of a memory's read-out after cancellation: the heads' norm brings the rest back to order one
CANCELLED = 0.03
ROUTER_GAIN = 2.0


class Oracle:
    """The oracle's logits of one sequence, and which positions do not hang on a router's close call (all of them in
    32-bit).  A bfloat16 run may choose another expert where two logits nearly tie; it then computes another function at
    that position and, through attention and memories, at later ones.  So the oracle runs twice more with the choice pushed
    by CLOSE_CALL one way and the other; positions whose logits move, and positions with a close call of their own, are not
    compared; nor are positions where nearly all of a memory's read-out cancels, or that a rounding of the embeddings alone moves by 4 % and more."""

    def __init__(self, tensors, cfg, ids: Sequence[int], dtype: str):
        logits, _, margin, left = P.forward(cfg, tensors, ids)
        self.logits = logits.float()
        self.safe = torch.ones(len(ids), dtype=torch.bool)
        if dtype == "float32":
            return
        self.safe &= left >= CANCELLED
        if any((l.get("mlp") or {}).get("kind") == "moe" for l in cfg["layers"]):
            self.safe &= margin >= CLOSE_CALL
            other = P.forward(cfg, tensors, ids, tilt=CLOSE_CALL)[0]
            self.safe &= (other - logits).norm(dim=-1) <= 0.035 * logits.norm(dim=-1)
        g = torch.Generator().manual_seed(77)
        moved = dict(tensors)
        moved["embed"] = tensors["embed"] * (1.0 + 2.0 ** -8 * (2.0 * torch.rand(tensors["embed"].shape, generator=g,
                                                                                  dtype=torch.float64) - 1.0))
        other = P.forward(cfg, moved, ids)[0]
        self.safe &= (other - logits).norm(dim=-1) <= 0.04 * logits.norm(dim=-1)

    def check(self, got: torch.Tensor, places, dtype: str, what: str = "", tol=None) -> None:
        places = list(places)
        keep = [i for i, p in enumerate(places) if bool(self.safe[p])]
        assert len(keep) * 10 >= len(places) or len(places) < 32, f"{what}: too many close calls to test anything"
        if keep:
            assert_rows_close(got.float().cpu().reshape(len(places), -1)[keep], self.logits[[places[i] for i in keep]],
                              dtype, what, tol, few=True)


def oracle(tensors, cfg, ids, dtype) -> Oracle:
    return Oracle(tensors, cfg, ids, dtype)


# rows are compared as vectors: |got - want|_2 <= row * |want|_2.  bfloat16: activations are rounded to 8 bits of mantissa
# between kernels while the oracle keeps 64-bit ones; every row has a loose bound and the median of many rows a tight one.
# A wrong key, expert, state or position shows as tens of per cent (and to four digits in the 32-bit runs of the same
# kernels).  In bfloat16 one row in twenty-five may pass the loose bound, up to OUTLIER_TOL: single positions where a
# peaked softmax multiplies a rounding, or where it turns a router's choice (the same rows however the prompt is cut).
ROW_TOL = {"float32": 1e-4, "bfloat16": 6e-2}
MEDIAN_TOL = {"float32": 2e-5, "bfloat16": 2.5e-2}
OUTLIER_TOL = 0.6


def assert_rows_close(got: torch.Tensor, want: torch.Tensor, dtype: str, what: str = "", tol=None, few=False):
    """``tol``: another bound for every row; no row may pass it unless ``few``."""
    got, want = got.float().cpu(), want.float().cpu()
    assert got.shape == want.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(want.shape)}"
    if got.dim() == 1:
        got, want = got[None], want[None]
    assert bool(torch.isfinite(got).all()), f"{what}: not finite"
    rel = (got - want).norm(dim=-1) / want.norm(dim=-1).clamp_min(1e-9)
    outliers = 0 if (dtype == "float32" or (tol is not None and not few)) else max(1, len(rel) // 25)
    tol = tol or ROW_TOL[dtype]
    over = (rel > tol).nonzero().flatten().tolist()
    assert len(over) <= outliers and (not over or float(rel.max()) <= OUTLIER_TOL), (
        f"{what}: row {int(rel.argmax())} differs by {rel.max():.3e} of its norm; rows over {tol}: {over[:12]}")
    if len(rel) >= 8:
        assert float(rel.median()) <= MEDIAN_TOL[dtype], f"{what}: the median row differs by {rel.median():.3e} of its norm"


def prompts(vocab: int, lengths: Sequence[int], seed: int) -> List[List[int]]:
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, vocab, (n,), generator=g).tolist() for n in lengths]


def greedy_generate(tensors, cfg, prompt: Sequence[int], n: int) -> List[int]:
    """The oracle's greedy continuation (the whole sequence is run anew for every token: the oracle keeps no state)."""
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(torch.argmax(P.forward(cfg, tensors, ids)[0][-1])))
    return ids[len(prompt):]


def changed(cfg, path: Sequence, value):
    """A copy of the configuration with one value replaced (path: keys and indices from the top)."""
    c = copy.deepcopy(cfg)
    at = c
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    return c
