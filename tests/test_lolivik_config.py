"""Lolivik without a GPU: the configuration reader (defaults, refusals, round trip, tensor names), the cache's part in kept
first tokens and nested states, the bias table's rows, and the plain implementation checked by hand on tiny inputs and
against itself."""
import copy
import math

import pytest
import torch

import plain_lolivik as P
from lolivik_helpers import LOLI, changed, make_tensors

F64 = torch.float64


def test_the_reader_round_trips_and_lowers_every_layer():
    from zlm_b200.registry import config_from_dict
    from zlm_b200.parts.model import DecoderModel
    for name, d in LOLI.items():
        cfg = config_from_dict(d)
        assert config_from_dict(cfg.to_dict()) == cfg, name
        spec = cfg.to_model_spec()
        assert [l.arrangement for l in spec.layers] == ["sublayer_norm"] * len(d["layers"])
        assert [l.mixer.kind for l in spec.layers] == ["mlstm" if l["type"] == "mlstm" else "conv_attention" for l in d["layers"]]
        names = DecoderModel(spec).param_specs()
        mixing = [i for i, l in enumerate(d["layers"]) if l["mixer"].get("v_mix")]
        for i, l in enumerate(d["layers"]):
            m, p = l["mixer"], f"l{i}.mix."
            assert names[f"l{i}.norm1"].shape == (d["width"],) and (f"l{i}.norm2" in names) == (l["mlp"] is not None)
            assert names[p + "q"].shape == (m["heads"] * m["dim"], d["width"])
            assert (p + "rel" in names) == (p + "sink" in names) == (l["type"] == "attention")
            assert (p + "vmix" in names) == (i in mixing) and (i not in mixing or names[p + "vmix"].ignorable == (i == mixing[0]))
            if l["type"] == "mlstm":
                assert names[p + "norm"].shape == (m["heads"] * m["vdim"],) and names[p + "i.b"].shape == (m["heads"],)
                assert names[p + "f"].shape == (m["heads"], d["width"]) and names[p + "g"].shape == names[p + "v"].shape
            elif l["type"] == "attention":
                assert names[p + "q.norm"].shape == (m["heads"] * m["dim"],) and names[p + "k.norm"].shape == (m["kv_heads"] * m["dim"],)
            else:
                assert names[p + "q.norm"].shape == names[p + "k.norm"].shape == (m["dim"],)
            ff = l["mlp"] or {}
            assert (f"l{i}.mlp.router" in names) == (ff.get("kind") == "moe") and (f"l{i}.mlp.gate" in names) == (ff.get("kind") == "dense")
            assert (f"l{i}.mlp.shared.gate" in names) == ("shared" in ff)
        assert "embed" in names and "final.norm" in names and not names["head"].ignorable


def test_defaults_and_refusals():
    from zlm_b200 import ConfigError
    from zlm_b200.registry import config_from_dict
    d = copy.deepcopy(LOLI["A"])
    del d["residual_mult"], d["layers"][0]["mixer"]["softcap"], d["layers"][0]["mixer"]["q_temp"], d["layers"][5]["mixer"]["mask"]
    del d["layers"][5]["mixer"]["kv_heads"], d["layers"][2]["mixer"]["mask"]["keep_first"]
    cfg = config_from_dict(d)
    assert cfg.residual_mult == 1.0 and cfg.layers[0].mixer.softcap == 0.0 and cfg.layers[0].mixer.q_temp is None
    assert cfg.layers[5].mixer.window == 0 and cfg.layers[5].mixer.kv_heads == 2 and cfg.layers[2].mixer.keep_first == 0
    bad = [(("layers", 0, "type"), "latent_attention", "type"), (("layers", 0, "mixer", "kv_heads"), 4, "kv_heads"),
           (("layers", 0, "mixer", "bias_max"), 0, "bias_max"), (("layers", 0, "mixer", "q_temp", "every"), 0, "every"),
           (("layers", 3, "mixer", "vdim"), 24, "v_mix"), (("layers", 2, "mixer", "rot", "dims"), 7, "dims"),
           (("layers", 2, "mixer", "rot", "dims"), 42, "dims"), (("layers", 2, "mixer", "rot", "scaling", "high"), 0, "scaling"),
           (("layers", 2, "mixer", "mask", "size"), 0, "mask"), (("layers", 2, "mixer", "mask", "keep_first"), -1, "mask"),
           (("layers", 1, "mixer", "gate_cap"), 0, "gate_cap"), (("layers", 1, "mlp", "router", "top"), 9, "top"),
           (("layers", 1, "mlp", "expert", "limit"), 0, "limit"), (("layers", 1, "mlp", "shared", "ff"), 0, "ff"),
           (("layers", 0, "mlp", "kind"), "sparse", "kind"), (("norm", "eps"), 0, "eps")]
    for path, value, word in bad:
        with pytest.raises(ConfigError, match=word):
            config_from_dict(changed(LOLI["A"], path, value))
    for path in (("layers", 0, "mixer", "scale"), ("layers", 0, "mixer", "bias_max"), ("layers", 1, "mixer", "gate_cap"),
                 ("layers", 1, "mlp", "expert", "limit"), ("layers", 2, "mixer", "rot", "scaling", "low"), ("norm",), ("width",)):
        d = copy.deepcopy(LOLI["A"])
        at = d
        for k in path[:-1]:
            at = at[k]
        del at[path[-1]]
        with pytest.raises(ConfigError, match=path[-1]):
            config_from_dict(d)


@pytest.mark.parametrize("rows,far", [(16, 40), (32, 128), (6, 20), (12, 7), (2, 40), (10, 4000), (64, 33)])
def test_the_bias_tables_rows_by_distance(rows, far):
    """The product's table of rows against the formula; monotonic, and constant from the largest distance on."""
    from zlm_b200.parts.conv_attention import distance_rows
    got = distance_rows(rows, far)
    assert got == [P.distance_bucket(n, rows, far) for n in range(far + 1)] and got == sorted(got)
    assert got[-1] == rows - 1 == P.distance_bucket(10 * far, rows, far)


def test_first_tokens_stay_in_the_cache_beside_a_window():
    from zlm_b200.cache.kv_cache import KVCache
    from zlm_b200.config.spec import ScheduleEntry
    from zlm_b200.parts.base import CacheRequest

    def held_after(keep, n, window=70):
        c = KVCache([ScheduleEntry(0)], [CacheRequest(1, 16, window, keep=keep)], [None], 64 * 40, 2, 4096, torch.float32, "cpu")
        s = c.alloc_slot()
        for at in range(0, n, 100):                        # page by page, as a long decode gives them back
            c.reserve([(s, min(100, n - at))])
            c.commit([(s, min(100, n - at))])
        c.check()
        held = [p >= 0 for p in c.groups[0].slot_pages[s]]
        pages = c.groups[0].pages.held
        c.free_slot(s)
        assert c.tokens_held() == 0 and pages == sum(held)
        return held
    # the next query sits at 1000: 70 keys reach back to 931, in page 14
    assert held_after(0, 1000) == [i >= 14 for i in range(16)]
    assert held_after(1, 1000) == [i >= 14 or i < 1 for i in range(16)]
    assert held_after(64, 1000) == [i >= 14 or i < 1 for i in range(16)]
    assert held_after(65, 1000) == [i >= 14 or i < 2 for i in range(16)]
    assert held_after(5000, 1000) == [True] * 16


def test_layers_that_keep_different_first_tokens_are_groups_of_their_own():
    from zlm_b200.cache.kv_cache import KVCache
    from zlm_b200.config.spec import ScheduleEntry
    from zlm_b200.parts.base import CacheRequest
    reqs = [CacheRequest(1, 16, 20, keep=3), CacheRequest(1, 16, 20), CacheRequest(1, 16, 20, keep=3)]
    c = KVCache([ScheduleEntry(i) for i in range(3)], reqs, [None] * 3, 640, 2, 640, torch.float32, "cpu")
    assert sorted(g.entries for g in c.groups) == [[0, 2], [1]] and {g.keep for g in c.groups} == {0, 3}


# ------------------------------------------------------------------------------------------ the plain functions by hand
def test_window_and_first_tokens_by_hand():
    seen = P.window_with_first_tokens(6, {"size": 2, "keep_first": 1})
    want = [[1, 0, 0, 0, 0, 0], [1, 1, 0, 0, 0, 0], [1, 1, 1, 0, 0, 0], [1, 0, 1, 1, 0, 0], [1, 0, 0, 1, 1, 0], [1, 0, 0, 0, 1, 1]]
    assert seen.int().tolist() == want
    assert P.window_with_first_tokens(3, None).int().tolist() == [[1, 0, 0], [1, 1, 0], [1, 1, 1]]
    assert P.window_with_first_tokens(2, {"size": 1, "keep_first": 9}).int().tolist() == [[1, 0], [1, 1]]


def test_buckets_by_hand():
    # 8 rows up to 64: 4 rows for 0 .. 3, then 4 + floor(ln(n / 4) / ln(16) * 4) = 4 + floor(log2(n / 4)), at most 7
    assert [P.distance_bucket(n, 8, 64) for n in (0, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 999)] == [0, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    b = P.distance_bias(3, torch.tensor([[1.0], [2.0], [3.0], [4.0]], dtype=F64), 8)[..., 0]
    assert b[2].tolist() == [3.0, 2.0, 1.0]


def test_attention_with_cap_bias_and_sink_by_hand():
    q = torch.tensor([[[1.0]], [[3.0]]], dtype=F64)
    k = torch.tensor([[[2.0]], [[-1.0]]], dtype=F64)
    v = torch.tensor([[[1.0]], [[10.0]]], dtype=F64)
    bias = torch.zeros(2, 2, 1, dtype=F64)
    bias[1, 0], bias[1, 1] = 0.5, -0.25
    o = P.attend(q, k, v, 0.5, P.window_with_first_tokens(2, None), 2.0, bias, torch.tensor([0.3], dtype=F64))
    a, b, s = math.exp(2 * math.tanh(3.0 / 2) + 0.5), math.exp(2 * math.tanh(-1.5 / 2) - 0.25), math.exp(0.3)
    assert float(o[1]) == pytest.approx((a + 10 * b) / (a + b + s))
    assert float(o[0]) == pytest.approx(math.exp(2 * math.tanh(0.5)) / (math.exp(2 * math.tanh(0.5)) + s))


def test_temperature_rotation_and_frequencies_by_hand():
    t = P.query_temperature(9, {"coef": 0.5, "every": 4})
    want = [1 + 0.5 * math.log(1 + x) for x in (0, 0, 0, 1, 1, 1, 1, 2, 2)]
    assert torch.allclose(t, torch.tensor(want, dtype=F64))
    x = torch.zeros(4, 1, 5, dtype=F64)
    x[3, 0] = torch.tensor([1.0, 2.0, 3.0, 4.0, 5.0])
    y = P.rotate_neighbours(x, {"base": 100.0, "dims": 4})[3, 0]
    a0, a1 = 3.0, 0.3                                                          # pairs (0, 1) and (2, 3)
    want = [math.cos(a0) - 2 * math.sin(a0), 2 * math.cos(a0) + math.sin(a0), 3 * math.cos(a1) - 4 * math.sin(a1),
            4 * math.cos(a1) + 3 * math.sin(a1), 5.0]
    assert torch.allclose(y, torch.tensor(want, dtype=F64))
    # wavelengths 2 pi * (1, 10, 100, 1000); original 100: kept below 25, divided above 100, a mixture between
    f = P.rotary_frequencies({"base": 1e4, "dims": 8, "scaling": {"factor": 8.0, "original": 100, "low": 1.0, "high": 4.0}})
    s = (100 / (20 * math.pi) - 1) / 3
    assert torch.allclose(f, torch.tensor([1.0, (1 - s) * 0.1 / 8 + s * 0.1, 0.01 / 8, 0.001 / 8], dtype=F64))


def test_matrix_memory_by_hand():
    """Two tokens, one head of 1 x 1: the running maximum from 0, both kinds of denominator."""
    t = lambda *v: torch.tensor(v, dtype=F64).view(-1, 1, 1)
    g = lambda *v: torch.tensor(v, dtype=F64).view(-1, 1)
    o, (S, n, m) = P.matrix_memory(t(2.0, 0.1), t(3.0, -1.0), t(5.0, 7.0), g(-1.0, 2.0), g(-0.5, -0.25))
    # token 0: m = max(-0.5 + 0, -1) = -0.5; S = e^(-0.5) 15; n = e^(-0.5) 3; |n q| = 3.64 > e^0.5
    a = math.exp(-0.5)
    assert float(o[0]) == pytest.approx(a * 15 * 2 / (a * 3 * 2 + 1e-6), rel=1e-9)
    # token 1: m = max(-0.75, 2) = 2; S = e^(-2.75) S0 - 7; n = e^(-2.75) n0 - 1; |n q| = 0.09 < e^-2 = 0.135
    b = math.exp(-0.25 - 0.5 - 2.0)
    assert float(S) == pytest.approx(b * a * 15 - 7) and float(n) == pytest.approx(b * a * 3 - 1) and float(m) == 2.0
    assert float(o[1]) == pytest.approx((b * a * 15 - 7) * 0.1 / (math.exp(-2.0) + 1e-6))


def test_expert_and_routing_by_hand():
    one = torch.ones(1, 1, dtype=F64)
    t = {"gate": 2.0 * one, "up": -3.0 * one, "down": 5.0 * one}
    got = float(P.expert(torch.tensor([[1.0]], dtype=F64), "", 1.5, t))
    assert got == pytest.approx(5 * 1.5 / (1 + math.exp(-1.702 * 1.5)) * (-1.5 + 1))
    got = float(P.expert(torch.tensor([[-4.0]], dtype=F64), "", 1.5, t))             # a gate far below zero is not clamped
    assert got == pytest.approx(5 * -8 / (1 + math.exp(1.702 * 8)) * 2.5)
    picked, margin = P.choose(torch.tensor([1.0, 3.0, -2.0, 2.0], dtype=F64), 2)
    e = math.exp(-1.0)
    assert [x for x, _ in picked] == [1, 3] and margin == 1.0
    assert picked[0][1] == pytest.approx(1 / (1 + e)) and picked[1][1] == pytest.approx(e / (1 + e))


@pytest.mark.parametrize("name", sorted(LOLI))
def test_the_whole_model_is_causal(name):
    cfg = LOLI[name]
    ref = {n: t.double() for n, t in make_tensors(cfg, 3).items()}
    ids = torch.randint(0, cfg["vocab"], (40,), generator=torch.Generator().manual_seed(1)).tolist()
    full = P.forward(cfg, ref, ids)[0]
    assert torch.allclose(full[:25], P.forward(cfg, ref, ids[:25])[0], atol=1e-9)


def test_frequencies_of_the_product_are_those_of_the_formula():
    from types import SimpleNamespace
    from zlm_b200.parts.rope import RotaryInterleaved
    for base, dims, sc in ((1e4, 8, (8.0, 100, 1.0, 4.0)), (5e5, 64, (4.0, 8192, 1.0, 4.0)), (300.0, 6, (4.0, 30, 1.0, 2.0)), (1e4, 16, None)):
        sc = dict(zip(("factor", "original", "low", "high"), sc)) if sc else None
        r = RotaryInterleaved(base, dims, scaling=sc)
        r.attach(SimpleNamespace(device="cpu"))
        want = P.rotary_frequencies({"base": base, "dims": dims, "scaling": sc})
        assert torch.allclose(r.inv_freq.double(), want, rtol=1e-6)
