"""Murilix without a GPU: the configuration reader (defaults, refusals, round trip, tensor names), the cache's part in
shared latents and block states, and the plain implementation checked by hand on tiny inputs and against itself."""
import copy
import math

import pytest
import torch

import plain_murilix as P
from murilix_helpers import MURI, changed, make_tensors

F64 = torch.float64


def test_the_reader_round_trips_and_lowers_every_layer():
    from zlm_b200.registry import config_from_dict
    from zlm_b200.parts.model import DecoderModel
    for name, d in MURI.items():
        cfg = config_from_dict(d)
        assert config_from_dict(cfg.to_dict()) == cfg, name
        spec = cfg.to_model_spec()
        assert [l.arrangement for l in spec.layers] == ["parallel_sublayers"] * len(d["layers"])
        assert [l.mixer.kind for l in spec.layers] == [l["type"] for l in d["layers"]]
        assert [e.cache_of for e in spec.schedule] == [l["mixer"].get("kv_from") for l in d["layers"]]
        names = DecoderModel(spec).param_specs()
        assert names["side.embed"].shape == (d["vocab"], d["token_side"]["dim"] * len(d["layers"]))
        for i, l in enumerate(d["layers"]):
            m = l["mixer"]
            assert names[f"l{i}.norm1"].shape == (d["width"],) and f"l{i}.norm2" not in names
            assert names[f"l{i}.canon1"].shape == (d["width"], d["canon"]["taps"])
            assert names[f"l{i}.side.gate"].shape == (d["token_side"]["dim"], d["width"])
            assert names[f"l{i}.side.norm"].shape == (d["width"],)
            if l["type"] == "mingru":
                assert names[f"l{i}.mix.z.b"].shape == (m["width"],) and names[f"l{i}.mix.o"].shape == (d["width"], m["width"])
            else:
                assert names[f"l{i}.mix.uq"].shape == (m["heads"] * (m["dim"] + m["rot_dim"]), m["q_rank"])
                assert names[f"l{i}.mix.dq.norm"].shape == (m["q_rank"],) and f"l{i}.mix.q" not in names
                assert (f"l{i}.mix.dkv" in names) == (f"l{i}.mix.dkv.norm" in names) == ("kv_from" not in m)
            kind = (l["mlp"] or {}).get("kind")
            assert (f"l{i}.mlp.act" in names) == (kind == "dense") and (f"l{i}.mlp.router" in names) == (kind == "moe")
            assert f"l{i}.mlp.gate" not in names
        assert "embed" in names and "final.norm" in names and names["head"].ignorable


def test_every_layer_reads_its_own_columns_of_one_side_table():
    from zlm_b200.registry import config_from_dict
    spec = config_from_dict(MURI["A"]).to_model_spec()
    assert [l.layer_input.params["offset"] for l in spec.layers] == [12 * i for i in range(6)]
    assert {l.layer_input.tensor_name("table") for l in spec.layers} == {"side.embed"}


def test_defaults_and_refusals():
    from zlm_b200 import ConfigError
    from zlm_b200.registry import config_from_dict
    cfg = config_from_dict(MURI["B"])
    assert cfg.embedding_scale == 1.0 and cfg.layers[3].mixer.window == 0 and cfg.layers[3].mixer.rot_dims == 0
    bad = [(("layers", 0, "type"), "attention", "type"), (("layers", 2, "mixer", "kv_from"), 1, "kv_from"),
           (("layers", 2, "mixer", "kv_from"), 2, "kv_from"), (("layers", 5, "mixer", "kv_from"), 2, "kv_from"),
           (("layers", 2, "mixer", "kv_rank"), 32, "kv_from"), (("layers", 2, "mixer", "rot", "base"), 1.0, "kv_from"),
           (("layers", 0, "mixer", "rot", "dims"), 7, "dims"), (("layers", 0, "mixer", "rot", "dims"), 10, "dims"),
           (("layers", 0, "mixer", "mask", "size"), 0, "mask"), (("layers", 0, "mixer", "q_rank"), 0, "sizes"),
           (("layers", 1, "mixer", "width"), 0, "width"), (("layers", 1, "mlp", "router", "top"), 9, "top"),
           (("layers", 0, "mlp", "kind"), "sparse", "kind"), (("canon", "taps"), 0, "taps"), (("token_side", "dim"), 0, "dim")]
    for path, value, word in bad:
        with pytest.raises(ConfigError, match=word):
            config_from_dict(changed(MURI["A"], path, value))
    for path in (("layers", 0, "mixer", "scale"), ("layers", 0, "mixer", "q_rank"), ("canon",), ("token_side",), ("norm",)):
        d = copy.deepcopy(MURI["A"])
        at = d
        for k in path[:-1]:
            at = at[k]
        del at[path[-1]]
        with pytest.raises(ConfigError, match=path[-1]):
            config_from_dict(d)


def test_pages_stay_as_long_as_any_reader_needs_them():
    """A window group gives a page back when no entry that reads it can see it, and not before: the reader's window may
    be wider than the window of the entry that wrote the page, or there may be none."""
    from zlm_b200.cache.kv_cache import KVCache
    from zlm_b200.config.spec import ScheduleEntry
    from zlm_b200.parts.base import CacheRequest

    def held_after(windows, n):
        sched = [ScheduleEntry(0)] + [ScheduleEntry(i + 1, cache_of=0) for i in range(len(windows) - 1)]
        reqs = [CacheRequest(1, 8, w, token_shape=(8,)) for w in windows]
        c = KVCache(sched, reqs, [None] * len(sched), 64 * 32, 2, 2048, torch.float32, "cpu")
        s = c.alloc_slot()
        c.reserve([(s, n)])
        c.commit([(s, n)])
        c.check()
        return c.groups[0].slot_pages[s]
    # the next query sits at position 1000: 70 keys reach back to 931 (page 14), 300 to 701 (page 10)
    assert held_after([70], 1000).index(next(p for p in held_after([70], 1000) if p >= 0)) == 14
    for order in ([70, 300], [300, 70]):
        pages = held_after(order, 1000)
        assert [p >= 0 for p in pages] == [i >= 10 for i in range(16)]
    assert all(p >= 0 for p in held_after([70, 0], 1000))


def test_groups_differ_by_their_readers_and_states_may_nest():
    from zlm_b200.cache.kv_cache import KVCache
    from zlm_b200.config.spec import ScheduleEntry
    from zlm_b200.parts.base import CacheRequest, StateRequest
    reqs = [CacheRequest(1, 8, 9, token_shape=(8,))] * 2 + [CacheRequest(1, 8, 100, token_shape=(8,))]
    state = (StateRequest((4,)), None), StateRequest((3, 2), torch.bfloat16)
    c = KVCache([ScheduleEntry(0), ScheduleEntry(1), ScheduleEntry(2, cache_of=1)], reqs, [None, state, None], 640, 2, 640,
                torch.float32, "cpu")
    assert len(c.groups) == 2 and {g.reach for g in c.groups} == {((9, 0),), ((9, 0), (100, 0))}
    inner, conv = c.ios[1].state
    assert inner[0].shape == (2, 4) and inner[1] is None and conv.shape == (2, 3, 2) and conv.dtype == torch.bfloat16
    s = c.alloc_slot()
    inner[0][s] = 1.0
    conv[s] = 1.0
    c.free_slot(s)
    s = c.alloc_slot()
    assert float(inner[0][s].abs().max()) == 0.0 and float(conv[s].float().abs().max()) == 0.0


# ------------------------------------------------------------------------------------------ the plain functions by hand
def test_layer_norm_and_unit_rms_by_hand():
    x = torch.tensor([[1.0, 3.0, 5.0, 7.0]], dtype=F64)
    w = torch.tensor([1.0, 2.0, 1.0, 0.5], dtype=F64)
    want = [v / math.sqrt(5.0 + 0.25) for v in (-3.0, -1.0 * 2, 1.0, 3.0 * 0.5)]
    assert torch.allclose(P.layer_norm(x, w, 0.25)[0], torch.tensor(want, dtype=F64))
    assert torch.allclose(P.rms_unit(torch.tensor([3.0, 4.0], dtype=F64), 0.5), torch.tensor([3.0, 4.0], dtype=F64) / math.sqrt(13.0))


def test_convolution_and_rotation_by_hand():
    h = torch.tensor([[1.0], [2.0], [3.0]], dtype=F64)
    y = P.causal_conv(h, torch.tensor([[100.0, 10.0, 1.0]], dtype=F64))        # the last column is the current token's
    assert y.flatten().tolist() == [1.0, 12.0, 123.0]
    x = torch.tensor([[[1.0, 2.0, 3.0, 4.0, 5.0]]], dtype=F64)
    y = P.rotate_pairs(x, torch.tensor([3]), 100.0, 4)[0, 0]
    a0, a1 = 3.0, 0.3                                                          # pairs (0, 1) and (2, 3)
    want = [math.cos(a0) - 2 * math.sin(a0), 2 * math.cos(a0) + math.sin(a0), 3 * math.cos(a1) - 4 * math.sin(a1),
            4 * math.cos(a1) + 3 * math.sin(a1), 5.0]
    assert torch.allclose(y, torch.tensor(want, dtype=F64))


def test_window_recurrence_and_candidate_by_hand():
    w = P.windowed_softmax(torch.zeros(1, 4, 4, dtype=F64), 2)[0]              # itself and one token before it
    assert torch.allclose(w, torch.tensor([[1, 0, 0, 0], [.5, .5, 0, 0], [0, .5, .5, 0], [0, 0, .5, .5]], dtype=F64))
    assert torch.allclose(P.windowed_softmax(torch.zeros(1, 3, 3, dtype=F64), 0)[0, 2], torch.full((3,), 1 / 3, dtype=F64))
    z = torch.tensor([[0.5], [0.25], [1.0]], dtype=F64)
    c = torch.tensor([[4.0], [8.0], [1.0]], dtype=F64)
    assert P.gated_recurrence(z, c).flatten().tolist() == [2.0, 0.75 * 2.0 + 2.0, 1.0]
    u = torch.tensor([0.0, 2.0, -1.0], dtype=F64)
    assert torch.allclose(P.candidate(u), torch.tensor([0.5, 2.5, 1 / (1 + math.e)], dtype=F64))


def test_polynomial_of_normed_powers_by_hand():
    z = torch.tensor([[1.0, -2.0]], dtype=F64)
    got = P.poly_norm(z, torch.tensor([2.0, 3.0, 5.0, 7.0], dtype=F64), 0.5)[0]
    n1, n2, n3 = math.sqrt(2.5 + 0.5), math.sqrt(8.5 + 0.5), math.sqrt(32.5 + 0.5)
    want = [2 / n1 + 3 / n2 + 5 / n3 + 7, -4 / n1 + 12 / n2 - 40 / n3 + 7]
    assert torch.allclose(got, torch.tensor(want, dtype=F64))


def test_routing_by_hand():
    z = torch.tensor([[1.0, 3.0, -2.0, 2.0]], dtype=F64)
    idx, wgt, margin = P.route(z, 2)
    e = math.exp(-1.0)
    assert idx.tolist() == [[1, 3]] and torch.allclose(wgt[0], torch.tensor([1 / (1 + e), e / (1 + e)], dtype=F64))
    assert float(margin) == 1.0
    idx, wgt, margin = P.route(z, 4)                            # all of them: no one is left out
    assert sorted(idx.tolist()[0]) == [0, 1, 2, 3] and float(wgt.sum()) == pytest.approx(1.0) and math.isinf(float(margin))


def test_token_input_by_hand():
    t = {"gate": torch.tensor([[1.0, 0.0]], dtype=F64), "proj": torch.tensor([[3.0], [4.0]], dtype=F64),
         "norm": torch.tensor([1.0, 2.0], dtype=F64)}
    x = torch.tensor([[2.0, 9.0]], dtype=F64)
    g = 0.5 * 2.0 * (1 + math.tanh(math.sqrt(2 / math.pi) * (2.0 + 0.044715 * 8.0))) * -1.5
    ms = (9 * g * g + 16 * g * g) / 2
    want = [3 * g / math.sqrt(ms + 0.1), 2 * 4 * g / math.sqrt(ms + 0.1)]
    assert torch.allclose(P.token_input(x, torch.tensor([[-1.5]], dtype=F64), "", t, 0.1)[0], torch.tensor(want, dtype=F64))


@pytest.mark.parametrize("name", sorted(MURI))
def test_the_whole_model_is_causal(name):
    cfg = MURI[name]
    ref = {n: t.double() for n, t in make_tensors(cfg, 3).items()}
    g = torch.Generator().manual_seed(1)
    ids = torch.randint(0, cfg["vocab"], (40,), generator=g).tolist()
    full = P.forward(cfg, ref, ids)[0]
    assert torch.allclose(full[:25], P.forward(cfg, ref, ids[:25])[0], atol=1e-9)


def test_a_reader_attends_over_the_named_layers_latents():
    """Other rotated keys in layer 0's records move what layer 2, which reads them, gives: it makes none of its own."""
    cfg = MURI["A"]
    ref = {n: t.double() for n, t in make_tensors(cfg, 4).items()}
    m = torch.randn(12, cfg["width"], dtype=F64, generator=torch.Generator().manual_seed(2))
    pos = torch.arange(12)
    recs = {}
    P.latent_attention(m, pos, "l0.mix.", cfg["layers"][0]["mixer"], ref, 1e-5, recs, 0)
    a = P.latent_attention(m, pos, "l2.mix.", cfg["layers"][2]["mixer"], ref, 1e-5, recs, 2)
    assert set(recs) == {0}
    moved = {0: (recs[0][0], recs[0][1].flip(1))}
    b = P.latent_attention(m, pos, "l2.mix.", cfg["layers"][2]["mixer"], ref, 1e-5, moved, 2)
    assert torch.allclose(a[0], b[0]) and float((a - b)[1:].norm()) > 1e-2      # (a first token sees itself alone)
