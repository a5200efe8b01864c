"""Small Murilix configurations and weights for the tests, and the oracle's inputs.

The configurations differ from each other, and from layer to layer, in every size and option: head counts (1, 2, 3, 18),
plain, rotated and value sizes that differ and are no multiples of 16 (and that are), rotation of a part of the rotated
slice, of all of it and none, query latents narrower and wider than the key latents and of odd sizes, windows below a
page, of exactly a page, a little above two pages, and none, layers that read an earlier layer's latents with a window
wider and narrower than that layer's, recurrences of odd and even widths, dense and routed feed-forwards and a layer
without one, one to four experts a token (also all of them), convolutions of 1 to 5 taps, side tables of 3 to 16 columns
a layer.

Weights are drawn so that activations are of order one (matrices N(0, 1/in)): attention and routing then depend
visibly on single keys and experts, which N(0, 0.02) would hide."""
from __future__ import annotations

import copy
import json
import os
from typing import Dict, List, Sequence

import torch

import plain_murilix as P


def lat(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot=None, window=0, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(mixer, mlp):
    return {"type": "mingru" if set(mixer) == {"width"} else "latent_attention", "mixer": mixer, "mlp": mlp}


def model(layers, vocab, width, taps, side, eps=1e-5, scale=None):
    cfg = {"architecture": "Murilix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps},
           "token_side": {"dim": side}, "layers": layers, "embedding": {"scale": 1.0 if scale is None else scale}}
    if scale is None:
        del cfg["embedding"]
    return cfg


MURI_A = model([
    layer(lat(3, 24, 8, 20, 40, 48, 0.4, rot=(10000.0, 8), window=70), dense(40)),
    layer({"width": 48}, moe(24, 8, 3)),
    # reads layer 0's latents through a window wider than that layer's own: the pages must stay for it
    layer(lat(2, 40, 8, 16, 24, 48, 0.3, rot=(10000.0, 8), window=150, kv_from=0), moe(16, 6, 1)),
    layer(lat(1, 16, 4, 12, 20, 28, 0.6, rot=(500.0, 2), window=9), None),
    layer({"width": 40}, dense(72)),
    layer(lat(4, 8, 4, 8, 16, 28, 0.5, rot=(500.0, 2), kv_from=3), moe(32, 5, 4)),
], vocab=160, width=64, taps=4, side=12, scale=6.0)
# wider; 18 heads; sizes the tensor-core kernels take; a window of exactly a page and one read through a narrower window;
# no rotation; two taps; all experts of a router chosen
MURI_B = model([
    layer({"width": 96}, moe(48, 4, 4)),
    layer(lat(18, 32, 16, 32, 64, 64, 0.25, rot=(1e5, 16), window=130), dense(96)),
    layer(lat(4, 16, 16, 24, 32, 64, 0.35, rot=(1e5, 16), window=64, kv_from=1), moe(8, 12, 4)),
    layer(lat(2, 48, 16, 40, 96, 32, 0.3), moe(64, 7, 2)),
], vocab=200, width=128, taps=2, side=16, eps=1e-6)
# sizes that no kernel likes: one tap, odd side columns, recurrence, latents and feed-forward of odd widths, heads whose
# outputs do not fill a piece of 8
MURI_C = model([
    layer(lat(3, 7, 6, 5, 13, 19, 0.7, rot=(300.0, 4), window=33), dense(37)),
    layer({"width": 27}, moe(11, 3, 2)),
    layer(lat(5, 9, 6, 3, 22, 19, 0.5, rot=(300.0, 4), kv_from=0), None),
    layer({"width": 50}, dense(18)),
], vocab=77, width=40, taps=1, side=3, eps=1e-4, scale=3.0)
# a convolution longer than short portions
MURI_D = model([
    layer({"width": 32}, dense(32)),
    layer(lat(2, 16, 16, 16, 32, 32, 0.5, rot=(1000.0, 16), window=20), moe(16, 4, 1)),
], vocab=96, width=48, taps=5, side=8, scale=2.0)
MURI = {"A": MURI_A, "B": MURI_B, "C": MURI_C, "D": MURI_D}
# the same with a small embedding scale: with a tied head a model whose stream is mostly its token's row only ever repeats
# that token, and says little about greedy generation
TALKATIVE = {n: dict(copy.deepcopy(c), embedding={"scale": 0.1 if n == "C" else 0.2}) for n, c in MURI.items()}


def make_tensors(cfg_dict, seed: int) -> Dict[str, torch.Tensor]:
    """fp32 tensors by checkpoint name, every one rounded to bfloat16 values (so that both engine dtypes and the
    oracle compute on the same numbers)."""
    from zlm_b200.parts.model import DecoderModel
    from zlm_b200.registry import config_from_dict
    specs = DecoderModel(config_from_dict(cfg_dict).to_model_spec()).param_specs()
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name in sorted(specs):
        if specs[name].ignorable:
            continue
        shape = specs[name].shape
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif last == "b":
            t = torch.randn(shape, generator=g) - (1.0 if name.endswith("z.b") else 0.0)      # gates mostly below one half
        elif last == "act":
            t = torch.tensor([0.7, -0.5, 0.4, 0.3]) + 0.3 * torch.randn(shape, generator=g)
        elif last == "canon1":
            t = 0.5 * torch.randn(shape, generator=g)
        elif name in ("embed", "side.embed"):
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / shape[-1] ** 0.5
            if last == "router":
                t = t * ROUTER_GAIN
        out[name] = t.to(torch.bfloat16).float()
    return out


def write_model(tmp_path, cfg, tensors, tag: str):
    from zlm_b200.weights import write_safetensors
    folder = os.path.join(str(tmp_path), f"muri_{tag}")
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), {n: t.to(torch.bfloat16) for n, t in tensors.items()})
    return folder


def make_model(tmp_path, name: str, seed: int = 0, talkative: bool = False):
    """Writes the model to a folder; returns (folder, config mapping, float64 tensors for the oracle)."""
    cfg = (TALKATIVE if talkative else MURI)[name]
    tensors = make_tensors(cfg, seed)
    return write_model(tmp_path, cfg, tensors, f"{name}_{seed}"), cfg, {n: t.double() for n, t in tensors.items()}


def one_layer(mixer, mlp=None, width=64, vocab=96, taps=2, side=8, **top):
    """A model of one layer around the mechanism under test."""
    cfg = model([layer(mixer, mlp)], vocab, width, taps, side)
    cfg.update(top)
    return cfg


def engine_for(tmp_path, cfg, tensors, dtype, tag, **kw):
    from zlm_b200 import Engine
    kw.setdefault("max_tokens", 2048)
    return Engine.from_pretrained(write_model(tmp_path, cfg, tensors, tag), dtype=dtype, **kw)


# how far a bfloat16 run's router logits may be from the oracle's
CLOSE_CALL = 0.06
ROUTER_GAIN = 2.0


class Oracle:
    """The oracle's logits of one sequence, and which positions do not hang on a router's close call (all of them in
    32-bit).  A bfloat16 run may choose another expert where two logits nearly tie; it then computes another function at
    that position and, through windows, convolutions and states, at later ones.  So the oracle runs twice more with the
    choice pushed by CLOSE_CALL one way and the other; positions whose logits move, and positions with a close call of
    their own, are not compared; nor are positions that a rounding of the embeddings alone moves by 4 % and more."""

    def __init__(self, tensors, cfg, ids: Sequence[int], dtype: str):
        logits, _, margin = P.forward(cfg, tensors, ids)
        self.logits = logits.float()
        self.safe = torch.ones(len(ids), dtype=torch.bool)
        if dtype == "float32":
            return
        if any((l.get("mlp") or {}).get("kind") == "moe" for l in cfg["layers"]):
            self.safe &= margin >= CLOSE_CALL
            for tilt in (CLOSE_CALL, -CLOSE_CALL):
                other = P.forward(cfg, tensors, ids, tilt=tilt)[0]
                self.safe &= (other - logits).norm(dim=-1) <= 0.02 * logits.norm(dim=-1)
        for seed in (77, 78):
            g = torch.Generator().manual_seed(seed)
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
# peaked softmax multiplies a rounding (the same rows however the prompt is cut).
ROW_TOL = {"float32": 1e-4, "bfloat16": 6e-2}
MEDIAN_TOL = {"float32": 2e-5, "bfloat16": 2.5e-2}
OUTLIER_TOL = 0.3


def assert_rows_close(got: torch.Tensor, want: torch.Tensor, dtype: str, what: str = "", tol=None, few=False):
    """``tol``: another bound for every row; no row may pass it unless ``few``."""
    got, want = got.float().cpu(), want.float().cpu()
    assert got.shape == want.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(want.shape)}"
    if got.dim() == 1:
        got, want = got[None], want[None]
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
