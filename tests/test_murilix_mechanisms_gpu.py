"""Murilix's mechanisms one at a time on the GPU, each as a small model run through the engine (or as the kernel alone)
against the function of the plain implementation, with weights and inputs made so that a fault shows: attention so
peaked that single keys carry a query's weight (the plain implementation is first asked whether a window that is one
token off, or a reader's window taken from the layer it reads, would change the answer: it must), gates so small that a
state from hundreds of tokens back still counts, convolutions whose weights are as large as what they are added to."""
import copy
from types import SimpleNamespace

import pytest
import torch

import plain_murilix as P
from murilix_helpers import (assert_rows_close, changed, dense, engine_for, lat, layer, make_tensors, model, moe, one_layer,
                             oracle, prompts)

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
F64 = torch.float64


def run_cut(eng, ids, cuts, then_single=0):
    """The sequence in portions of the given sizes, then ``then_single`` tokens one by one; logits at every place."""
    from zlm_b200 import StepEntry
    s = eng.new_sequence()
    at, got = 0, []
    for c in list(cuts) + [1] * then_single:
        got.append(eng.step([StepEntry(s, ids[at:at + c], list(range(c)))]).clone())
        at += c
    eng.release(s)
    return torch.cat(got)


def scaled(tensors, by):
    """A copy of the weights with some of them multiplied (name -> factor)."""
    out = dict(tensors)
    for n, f in by.items():
        out[n] = (out[n] * f).to(torch.bfloat16).float()
    return out


def moves(cfg, path, value, ref, ids, want, after, by=0.02, at_least=2):
    """Whether the plain implementation gives other logits with one value of the configuration replaced."""
    other = P.forward(changed(cfg, path, value), ref, ids)[0]
    rel = (other - want)[after:].norm(dim=-1) / want[after:].norm(dim=-1)
    assert int((rel > by).sum()) >= at_least, f"{path}={value} would not show"


def plan_for(lens, starts, slots):
    """The step arrays a kernel reads, for sequences of ``lens`` new tokens after ``starts`` earlier ones."""
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    seq = [r for r, n in enumerate(lens) for _ in range(n)]
    pos = [starts[r] + i for r, n in enumerate(lens) for i in range(n)]
    t = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    scratch = lambda name, shape, dtype: torch.full(shape, float("nan"), dtype=dtype, device="cuda")
    return SimpleNamespace(T=cu[-1], R=len(lens), token_pos=t(pos), token_seq=t(seq), token_slot=t([slots[r] for r in seq]),
                           seq_slot=t(slots), seq_start=t(starts), seq_new=t(lens), cu_seqlens=t(cu), max_new=max(lens),
                           is_decode=all(n == 1 for n in lens), scratch=scratch)


# ------------------------------------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,sizes", [(9, (2, 16, 8, 24, 20, 16)), (64, (3, 48, 16, 32, 40, 32)), (70, (1, 24, 4, 8, 12, 20)),
                                          (130, (18, 32, 32, 48, 64, 64))])
def test_latent_attention_sees_exactly_its_window(tmp_path, dtype, window, sizes):
    """Peaked attention: the plain implementation with a window one token longer or shorter gives other logits, the
    engine gives those of the right one, in prompts (both forms of latent attention), in portions that start inside a
    window, and token by token across page borders."""
    H, dn, dr, dv, qr, r = sizes
    cfg = one_layer(lat(H, dn, dr, dv, qr, r, 0.6, rot=(300.0, dr), window=window))
    t = scaled(make_tensors(cfg, 11), {"l0.mix.dq.norm": 2.5, "l0.mix.o": 2.0})
    ref = {n: x.double() for n, x in t.items()}
    n = window + 75
    (ids,) = prompts(cfg["vocab"], [n], seed=window)
    want = P.forward(cfg, ref, ids)[0]
    for other in (window + 1, window - 1):
        moves(cfg, ("layers", 0, "mixer", "mask", "size"), other, ref, ids, want, window)
    eng = engine_for(tmp_path, cfg, t, dtype, f"win{window}")
    tol = None if dtype == "float32" else 0.12          # (peaked attention multiplies bfloat16's rounding of q and k)
    assert_rows_close(run_cut(eng, ids, [n]), want, dtype, "whole", tol)
    assert_rows_close(run_cut(eng, ids, [window - 1, 2, 3, n - window - 4]), want, dtype, "portions", tol)
    assert_rows_close(run_cut(eng, ids, [window - 3], then_single=n - window + 3), want, dtype, "token by token", tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(2, 16, 8, 24, 20, 16), (4, 48, 16, 64, 40, 32), (3, 7, 6, 5, 13, 19)])
def test_far_keys_count_where_there_is_no_window(tmp_path, dtype, sizes):
    """400 tokens and one key that stands out: the value of an early token reaches every later query."""
    H, dn, dr, dv, qr, r = sizes
    cfg = one_layer(lat(H, dn, dr, dv, qr, r, 0.8, rot=(10000.0, dr // 2 * 2)))
    t = scaled(make_tensors(cfg, 12), {"l0.mix.dq.norm": 3.0, "l0.mix.o": 2.0})
    ref = {n: x.double() for n, x in t.items()}
    (ids,) = prompts(cfg["vocab"], [400], seed=5)
    want = P.forward(cfg, ref, ids)[0]
    other = P.forward(cfg, ref, prompts(cfg["vocab"], [150], seed=6)[0] + ids[150:])[0]
    assert int(((other - want)[250:].norm(dim=-1) / want[250:].norm(dim=-1) > 0.05).sum()) >= 10, "far keys do not show"
    eng = engine_for(tmp_path, cfg, t, dtype, f"far{H}")
    tol = None if dtype == "float32" else 0.15
    held = oracle(ref, cfg, ids, dtype)
    held.check(run_cut(eng, ids, [400]), range(400), dtype, "whole", tol)
    held.check(run_cut(eng, ids, [190, 2, 140], then_single=68), range(400), dtype, "portions and single tokens", tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("own,reader", [(9, 150), (150, 9), (70, 0), (64, 65)])
def test_a_reader_of_another_layers_latents_has_a_window_of_its_own(tmp_path, dtype, own, reader):
    """Two layers over one set of latents, with windows that differ either way: the wider one decides which pages stay
    (300 tokens, five pages; another sequence takes up pages that are given back)."""
    from zlm_b200 import StepEntry
    a = lat(2, 16, 8, 16, 24, 32, 0.7, rot=(1000.0, 8), window=own)
    b = lat(3, 24, 8, 16, 20, 32, 0.6, rot=(1000.0, 8), window=reader, kv_from=0)
    cfg = model([layer(a, None), layer(b, None)], 96, 64, 2, 8)
    t = scaled(make_tensors(cfg, 13), {"l0.mix.dq.norm": 2.0, "l1.mix.dq.norm": 2.5, "l1.mix.o": 2.0})
    ref = {n: x.double() for n, x in t.items()}
    ids, other = prompts(cfg["vocab"], [300, 200], seed=7)
    held, held_o = oracle(ref, cfg, ids, dtype), oracle(ref, cfg, other, dtype)
    want = P.forward(cfg, ref, ids)[0]
    moves(cfg, ("layers", 1, "mixer", "mask"), {"size": own}, ref, ids, want, 160, at_least=5 if reader > own + 1 or not reader else 1)
    eng = engine_for(tmp_path, cfg, t, dtype, f"share{own}_{reader}", max_tokens=640)
    tol = None if dtype == "float32" else 0.12
    held.check(run_cut(eng, ids, [300]), range(300), dtype, "whole", tol)
    s, s2 = eng.new_sequence(), eng.new_sequence()
    got, got2 = [eng.step([StepEntry(s, ids[:150], list(range(150)))]).clone()], []
    for i in range(150):
        e = [StepEntry(s, [ids[150 + i]], [0])] + ([StepEntry(s2, other[i:i + 1], [0])] if i % 3 else [StepEntry(s2, other[i:i + 1], [])])
        out = eng.step(e).clone()
        got.append(out[:1])
        if i % 3:
            got2.append((i, out[1]))
    held.check(torch.cat(got), range(300), dtype, "token by token beside another sequence", tol)
    held_o.check(torch.stack([x for _, x in got2]), [i for i, _ in got2], dtype, "the other sequence", tol)
    eng.cache.check()
    eng.release(s)
    eng.release(s2)
    assert eng.cache.tokens_held() == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_query_latents_and_records_from_one_kernel(dtype):
    """latent_down alone: the query latent's norm, its padding, the record with its rotation at far positions, the second
    place of the records; and without records."""
    from zlm_b200.kernels import PAGE_TOKENS, get_kernels
    k = get_kernels()
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(3)
    T, qr, r, dr, n_rot, eps = 5, 21, 12, 10, 8, 1e-3
    down = (0.05 * torch.randn(T, qr + r + dr + 3, generator=g)).to(dt).cuda()
    qw, cw = (1 + torch.randn(qr, generator=g)).to(dt), (1 + torch.randn(r, generator=g)).to(dt)
    inv = torch.tensor([50.0 ** (-2 * i / n_rot) for i in range(n_rot // 2)], dtype=torch.float32)
    plan = plan_for([3, 2], [62, 1000], [1, 0])
    table = torch.arange(40, dtype=torch.int32).flip(0).view(2, 20).contiguous().cuda()
    pool = torch.zeros(40, PAGE_TOKENS, r + dr, dtype=dt, device="cuda")
    cq = torch.full((T, 24), 7.0, dtype=dt, device="cuda")
    rec = torch.empty(T, r + dr, dtype=dt, device="cuda")
    k.latent_down(cq, down[:, :qr], qw.cuda(), eps, down[:, qr:qr + r + dr], cw.cuda(), inv.cuda(), n_rot, plan.token_pos,
                  plan.token_slot, table, pool, dr, r, rec_out=rec)
    d = down.cpu().to(F64)
    want_q = P.rms_unit(d[:, :qr], eps) * qw.to(F64)
    pos = plan.token_pos.cpu().long()
    want_r = torch.cat([P.rms_unit(d[:, qr:qr + r], eps) * cw.to(F64), P.rotate_pairs(d[:, qr + r:qr + r + dr], pos, 50.0, n_rot)], 1)
    tol = 1e-5 if dtype == "float32" else 6e-3
    assert_rows_close(cq[:, :qr], want_q, dtype, "query latent", tol)
    assert float(cq[:, qr:].float().abs().max()) == 0.0
    assert_rows_close(rec, want_r, dtype, "record", tol)
    slot = plan.token_slot.cpu().long()
    pages = table.cpu().long()[slot, pos // PAGE_TOKENS]
    assert torch.equal(pool.cpu()[pages, pos % PAGE_TOKENS], rec.cpu())
    assert int((pool.float().abs().sum(-1) > 0).sum()) == T                    # and nowhere else
    before = pool.clone()
    cq2 = torch.empty_like(cq)
    k.latent_down(cq2, down[:, :qr], qw.cuda(), eps)
    assert torch.equal(cq2, cq) and torch.equal(pool, before)


# ------------------------------------------------------------------------------------------------ the recurrence
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [27, 48, 300])
def test_gated_recurrence_remembers_from_far_back(tmp_path, dtype, width):
    """Gates near 0.01: 500 tokens whole (a cluster's warps side by side), in portions, then token by token; two sequences side
    by side; a slot used again starts from zero."""
    from zlm_b200 import StepEntry
    cfg = one_layer({"width": width}, dense(32))
    t = make_tensors(cfg, 21)
    t["l0.mix.z.b"] = (t["l0.mix.z.b"] * 0.5 - 3.5).to(torch.bfloat16).float()
    t = scaled(t, {"l0.mix.o": 3.0})
    ref = {n: x.double() for n, x in t.items()}
    a, b = prompts(cfg["vocab"], [500, 37], seed=9)
    want = P.forward(cfg, ref, a)[0]
    other = P.forward(cfg, ref, prompts(cfg["vocab"], [150], seed=4)[0] + a[150:])[0]
    assert float(((other - want)[160:200].norm(dim=-1) / want[160:200].norm(dim=-1)).median()) > 0.02, "the state does not show"
    eng = engine_for(tmp_path, cfg, t, dtype, f"gru{width}")
    assert_rows_close(run_cut(eng, a, [500]), want, dtype, "whole")
    assert_rows_close(run_cut(eng, a, [1, 2, 1, 3, 250, 2, 200], then_single=41), want, dtype, "portions, then single tokens")
    s1, s2 = eng.new_sequence(), eng.new_sequence()
    got = eng.step([StepEntry(s1, b, [36]), StepEntry(s2, a[:200], [99, 199])]).clone()          # (clusters, unequal sequences)
    assert_rows_close(got, torch.stack([P.forward(cfg, ref, b)[0][36], want[99], want[199]]), dtype, "side by side")
    got = eng.step([StepEntry(s1, a[:5], []), StepEntry(s2, a[200:210], [9])]).clone()
    assert_rows_close(got, want[209:210], dtype, "going on from the cluster's state")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cluster", [False, True])
@pytest.mark.parametrize("W,lens", [(5, [1, 1]), (64, [200, 1, 33]), (130, [31, 32, 65, 700]), (128, [1100]), (66, [2100, 7, 1024])])
def test_gated_recurrence_kernel(dtype, cluster, W, lens):
    """The kernel alone from states that are not zero: candidates on both sides of u = 0 (and at it), gates saturated
    either way, columns in any order inside wider rows, slots not in order."""
    from zlm_b200.kernels import get_kernels
    k = get_kernels()
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(W)
    R, T = len(lens), sum(lens)
    off = {"g": 2, "z": 2 + W, "x": 2 + 2 * W}
    proj = (2.0 * torch.randn(T, 3 * W + 4, generator=g)).to(dt)
    proj[:, off["x"]] = 0.0
    proj[::3, off["z"]] = 60.0
    proj[1::3, off["z"]] = -60.0
    bz, bx = torch.randn(W, generator=g).to(dt), torch.randn(W, generator=g).to(dt)
    bx[0] = 0.0
    slots = list(range(R))[::-1]
    state = torch.randn(R, W, generator=g)
    st = state.cuda().clone()
    out = torch.empty(T, W + 2, dtype=dt, device="cuda")[:, :W]
    k.mingru(out, proj.cuda(), off["z"], off["x"], off["g"], bz.cuda(), bx.cuda(), st, plan_for(lens, [3] * R, slots), cluster=cluster)
    p, at = proj.to(F64), 0
    tol = 2e-5 if dtype == "float32" else 8e-3
    for r, n in enumerate(lens):
        cut = lambda name: p[at:at + n, off[name]:off[name] + W]
        z, cand = torch.sigmoid(cut("z") + bz.to(F64)), P.candidate(cut("x") + bx.to(F64))
        S, S0 = [], state[slots[r]].to(F64)
        for i in range(n):
            S0 = (1 - z[i]) * S0 + z[i] * cand[i]
            S.append(S0)
        assert_rows_close(out[at:at + n], torch.stack(S) * P.silu(cut("g")), dtype, f"sequence {r}", tol)
        assert_rows_close(st[slots[r]], S0, "float32", f"state {r}", 2e-5)
        at += n


# ------------------------------------------------------------------------------------------------ the mixer's input
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
@pytest.mark.parametrize("C", [40, 37])
def test_input_convolution_kernel(dtype, taps, C):
    """Sequences shorter and longer than the convolution side by side, from states that are not zero; the state after
    portions of one, two and many tokens; a long run of single tokens."""
    from zlm_b200.kernels import get_kernels
    k = get_kernels()
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(taps)
    w = (torch.randn(C, taps, generator=g) * 0.8).to(dt)
    wt = w.t().contiguous().cuda()
    total = [60, 9, 31]
    hs = [torch.randn(n, C, generator=g).to(dt) for n in total]
    want = [h.to(F64) + P.causal_conv(h.to(F64), w.to(F64)) for h in hs]
    state = torch.zeros(3, max(taps - 1, 1), C, dtype=dt, device="cuda") if taps > 1 else None
    at, got = [0, 0, 0], [[], [], []]
    for cut in ([1, 2, 8], [2, 0, 1], [17, 3, 0], [1, 1, 1], [1, 1, 1], [38, 2, 20]):
        live = [r for r in (2, 0, 1) if cut[r]]
        lens = [cut[r] for r in live]
        h = torch.cat([hs[r][at[r]:at[r] + cut[r]] for r in live]).cuda()
        out = torch.empty_like(h)
        k.input_conv(out, h, wt, state, plan_for(lens, [at[r] for r in live], live))
        for r, o in zip(live, out.cpu().split(lens)):
            got[r].append(o)
            at[r] += cut[r]
        for r in range(3):
            for m in range(taps - 1):
                p = at[r] - (taps - 1) + m
                have = state[r, m].cpu()
                assert torch.equal(have, hs[r][p] if p >= 0 else torch.zeros(C, dtype=dt)), f"state of {r} after {at[r]}"
    assert at == total or at == [60, 9, 31]
    for r in range(3):
        assert_rows_close(torch.cat(got[r]), want[r], dtype, f"sequence {r}", 1e-5 if dtype == "float32" else 6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [2, 3, 4, 6])
def test_input_convolution_of_many_tokens(dtype, taps):
    """700 tokens of five sequences (runs of tokens that cross from one into the next, sequences shorter than the
    convolution among them), from states that are not zero."""
    from zlm_b200.kernels import get_kernels
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(taps)
    C, lens, slots = 136, [301, 1, 2, 390, 6], [3, 0, 4, 1, 2]
    w = (torch.randn(C, taps, generator=g) * 0.8).to(dt)
    st0 = torch.randn(5, taps - 1, C, generator=g).to(dt)
    h, st = torch.randn(sum(lens), C, generator=g).to(dt), st0.cuda()
    out = torch.empty(sum(lens), C, dtype=dt, device="cuda")
    get_kernels().input_conv(out, h.cuda(), w.t().contiguous().cuda(), st, plan_for(lens, [9] * 5, slots))
    for r, (x, o) in enumerate(zip(h.split(lens), out.cpu().split(lens))):
        ext = torch.cat([st0[slots[r]], x])
        want = x.to(F64) + P.causal_conv(ext.to(F64), w.to(F64))[taps - 1:]
        assert_rows_close(o, want, dtype, f"sequence {r}", 1e-5 if dtype == "float32" else 6e-3)
        assert torch.equal(st[slots[r]].cpu(), ext[len(ext) - (taps - 1):])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("center", [False, True])
@pytest.mark.parametrize("H", [40, 1000, 4096, 6001])
@pytest.mark.parametrize("taps", [0, 1, 2, 4, 6])
def test_closing_norm_opening_norm_and_convolution_in_one_kernel(dtype, center, H, taps):
    """The fused kernel against its parts: the residual add, both kinds of opening norm (on rows far from zero mean), the
    convolution and its state."""
    from zlm_b200.kernels import get_kernels
    k = get_kernels()
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(H + taps)
    R = 3
    x = torch.randn(R, H, generator=g) + 5.0
    y = torch.randn(R, H, generator=g) * 0.1
    w1, w2 = 1 + 0.3 * torch.randn(H, generator=g), 1 + 0.3 * torch.randn(H, generator=g)
    stream, out = x.cuda(), torch.empty(R, H, dtype=dt, device="cuda")
    conv = None
    if taps:
        cw = (torch.randn(taps, H, generator=g)).to(dt)
        st0 = torch.randn(5, taps - 1, H, generator=g).to(dt) if taps > 1 else None
        st = st0.cuda() if taps > 1 else None
        mixed = torch.empty_like(out)
        slots = [4, 0, 2]
        conv = (mixed, cw.cuda(), st, plan_for([1] * R, [7] * R, slots))
    k.norm_add_norm(stream, y.cuda(), w1.cuda(), 1e-5, out, w2.cuda(), 1e-4, center=center, conv=conv)
    want_x = x.to(F64) + P.rms_unit(y.to(F64), 1e-5) * w1.to(F64)
    want = P.layer_norm(want_x, w2.to(F64), 1e-4) if center else P.rms_unit(want_x, 1e-4) * w2.to(F64)
    tol = 1e-5 if dtype == "float32" else 5e-3
    assert_rows_close(stream, want_x, "float32", "stream", 1e-6)
    assert_rows_close(out, want, dtype, "opening norm", tol)
    if taps:
        h = out.cpu().to(F64)
        want_m = h * (1.0 + cw[taps - 1].to(F64))
        for j in range(taps - 1):
            want_m = want_m + cw[j].to(F64) * st0[slots, j].to(F64)
        assert_rows_close(mixed, want_m, dtype, "mixed", tol)
        if taps > 1:
            want_st = st0.clone()
            for r, s in enumerate(slots):
                want_st[s] = torch.cat([st0[s, 1:], out[r:r + 1].cpu()])
            assert torch.equal(st.cpu(), want_st)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H", [37, 64, 4096, 9000])
def test_layer_norm_kernel(dtype, H):
    """Rows whose mean is a hundred times their spread (a variance from squares would lose it), chosen rows."""
    from zlm_b200.kernels import get_kernels
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(H)
    x = (100.0 + torch.randn(6, H, generator=g)).float()
    w = (1 + 0.3 * torch.randn(H, generator=g)).to(dt)
    out = torch.empty(3, H, dtype=dt, device="cuda")
    rows = torch.tensor([5, 0, 3], dtype=torch.int32, device="cuda")
    get_kernels().layernorm(out, x.cuda(), w.cuda(), 1e-5, rows)
    want = P.layer_norm(x.to(F64)[[5, 0, 3]], w.to(F64), 1e-5)
    assert_rows_close(out, want, dtype, "rows", 2e-5 if dtype == "float32" else 5e-3)


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_mixer_reads_the_convolved_rows_and_the_feed_forward_the_plain_ones(tmp_path, dtype):
    """Large taps; the plain implementation with the convolution on neither or on both sublayers gives other logits."""
    cfg = one_layer({"width": 32}, dense(48), taps=3)
    t = scaled(make_tensors(cfg, 31), {"l0.canon1": 2.5, "l0.mix.o": 2.0, "l0.mlp.down": 2.0})
    ref = {n: x.double() for n, x in t.items()}
    (ids,) = prompts(cfg["vocab"], [80], seed=3)
    want = P.forward(cfg, ref, ids)[0]
    off = dict(ref)
    off["l0.canon1"] = torch.zeros_like(ref["l0.canon1"])
    assert float(((P.forward(cfg, off, ids)[0] - want).norm(dim=-1) / want.norm(dim=-1)).median()) > 0.05
    eng = engine_for(tmp_path, cfg, t, dtype, "canon")
    assert_rows_close(run_cut(eng, ids, [80]), want, dtype, "whole")
    assert_rows_close(run_cut(eng, ids, [2, 2, 1, 2, 30, 3], then_single=40), want, dtype, "portions, then single tokens")


# ------------------------------------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("F,cols", [(37, 40), (40, 40), (512, 512), (6000, 6000), (18000, 18000)])
@pytest.mark.parametrize("coef", [(0.7, -0.5, 0.4, 0.3), (0.0, 0.0, 1.0, 0.0), (0.0, 1.0, 0.0, 0.0), (0.0, 0.0, 0.0, 2.0)])
def test_polynomial_of_normed_powers_kernel(dtype, F, cols, coef):
    """Each power by itself too; rows large, ordinary and so small that eps decides; the padding columns become zeros."""
    from zlm_b200.kernels import get_kernels
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(F)
    z = (torch.randn(4, F, generator=g) * torch.tensor([[30.0], [1.0], [0.05], [1e-3]])).to(dt)
    c = torch.tensor(coef)
    out = torch.full((4, cols), 9.0, dtype=dt, device="cuda")
    get_kernels().poly_norm(out, z.cuda(), c.to(dt).cuda(), 1e-6)
    want = P.poly_norm(z.to(F64), c.to(dt).to(F64), 1e-6)
    assert_rows_close(out[:, :F], want, dtype, "rows", 1e-5 if dtype == "float32" else 6e-3)
    if cols > F:
        assert float(out[:, F:].float().abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [37, 96])
def test_dense_feed_forward(tmp_path, dtype, ff):
    cfg = one_layer({"width": 16}, dense(ff))
    t = scaled(make_tensors(cfg, 41), {"l0.mlp.down": 3.0, "l0.mix.o": 0.3})
    ref = {n: x.double() for n, x in t.items()}
    (ids,) = prompts(cfg["vocab"], [90], seed=3)
    want = P.forward(cfg, ref, ids)[0]
    for i in range(4):                                   # each of the four numbers counts
        moved = dict(ref)
        moved["l0.mlp.act"] = ref["l0.mlp.act"].clone()
        moved["l0.mlp.act"][i] += 0.5
        assert float(((P.forward(cfg, moved, ids)[0] - want).norm(dim=-1) / want.norm(dim=-1)).median()) > 0.02
    eng = engine_for(tmp_path, cfg, t, dtype, f"dense{ff}")
    assert_rows_close(run_cut(eng, ids, [90]), want, dtype, "whole")
    assert_rows_close(run_cut(eng, ids, [5], then_single=85), want, dtype, "single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("r", [(8, 3, 24), (6, 1, 32), (4, 4, 16), (5, 2, 11)])
def test_routed_layer_against_the_plain_one(tmp_path, dtype, r):
    """Few tokens and many (the grouped product), an expert width that only the plain kernels take, all experts chosen."""
    experts, top, ff = r
    cfg = one_layer({"width": 16}, moe(ff, experts, top))
    t = scaled(make_tensors(cfg, 51), {f"l0.mlp.e{e}.down": 2.0 for e in range(experts)})
    ref = {n: x.double() for n, x in t.items()}
    eng = engine_for(tmp_path, cfg, t, dtype, f"moe{experts}")
    for n in (3, 150):
        (a,) = prompts(cfg["vocab"], [n], seed=n)
        oracle(ref, cfg, a, dtype).check(run_cut(eng, a, [n]), range(n), dtype, f"{n} tokens")


def test_weights_are_the_softmax_over_the_chosen_alone():
    """Both router kernels, logits far apart and far from zero: the chosen weights sum to one."""
    from zlm_b200.kernels import get_kernels
    k = get_kernels()
    g = torch.Generator().manual_seed(2)
    T, E, top = 40, 11, 3
    z = 8.0 * torch.randn(T, E, generator=g) + 50.0
    z[0] = torch.arange(E).float() * 20.0
    idx = torch.empty(T, top, dtype=torch.int32, device="cuda")
    wgt = torch.empty(T, top, dtype=torch.float32, device="cuda")
    k.moe_choose(idx, wgt, z.cuda().contiguous(), E, top, None, "softmax", True)
    want_i, want_w, _ = P.route(z.to(F64), top)
    assert torch.equal(idx.cpu().long(), want_i) and torch.allclose(wgt.cpu().to(F64), want_w, atol=1e-6)
    x, w = torch.randn(T, 32, generator=g), torch.randn(E, 32, generator=g)
    k.moe_route(idx, wgt, x.cuda(), w.cuda(), top, None, None, "softmax", True)
    want_i, want_w, _ = P.route(x.to(F64) @ w.to(F64).T, top)
    assert torch.equal(idx.cpu().long(), want_i) and torch.allclose(wgt.cpu().to(F64), want_w, atol=1e-5)


# ------------------------------------------------------------------------------------------------ the tokens' side rows
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [1, 3, 8, 16, 17, 200])
@pytest.mark.parametrize("K,dim", [(64, 3), (40, 12), (2560, 24), (4096, 256)])
def test_side_rows_gated(dtype, T, K, dim):
    """Both forms of the gate (few tokens: product, gelu and row in one kernel) against the plain formula, layer columns
    from the middle of the table, padding columns zero."""
    from zlm_b200.kernels import get_kernels
    k = get_kernels()
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    g = torch.Generator().manual_seed(T + K)
    V, L = 50, 3
    x = torch.randn(T, K, generator=g)
    w = (torch.randn(dim, K, generator=g) * 1.5 / K ** 0.5).to(dt)
    side = torch.randn(V, L * dim, generator=g).to(dt)
    ids = torch.randint(0, V, (T,), generator=g)
    cols = (dim + 7) // 8 * 8 if dtype == "bfloat16" else dim
    xin = x.to(F64)
    out = torch.full((T, cols), 9.0, dtype=dt, device="cuda")
    if k.token_gate_few_supported(T, w):
        assert dtype == "bfloat16" and T <= 16
        k.token_gate_few(out, x.cuda(), w.cuda(), side.cuda(), dim, ids.int().cuda())
    else:
        xc = x.to(dt).cuda()
        xin = xc.cpu().to(F64)
        z = torch.empty(T, dim, dtype=dt, device="cuda")
        k.linear(z, xc, w.cuda())
        k.token_gate(out, z, side.cuda(), dim, ids.int().cuda())
    want = P.gelu_tanh(xin @ w.to(F64).T) * side.to(F64)[ids, dim:2 * dim]
    assert_rows_close(out[:, :dim].reshape(1, -1), want.reshape(1, -1), dtype, "g", 1e-5 if dtype == "float32" else 8e-3)
    if cols > dim:
        assert float(out[:, dim:].float().abs().max()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("side", [3, 16])
def test_every_layer_reads_its_own_side_columns(tmp_path, dtype, side):
    """Two layers whose side rows count: exchanging the two halves of the table moves the logits, the engine gives those
    of the right order, prompts and single tokens."""
    cfg = model([layer({"width": 16}, None), layer({"width": 24}, dense(16))], 60, 48, 2, side)
    t = scaled(make_tensors(cfg, 61), {"l0.side.norm": 2.0, "l1.side.norm": 2.0})
    ref = {n: x.double() for n, x in t.items()}
    (ids,) = prompts(cfg["vocab"], [50], seed=3)
    want = P.forward(cfg, ref, ids)[0]
    moved = dict(ref)
    moved["side.embed"] = ref["side.embed"].roll(side, dims=1)
    assert float(((P.forward(cfg, moved, ids)[0] - want).norm(dim=-1) / want.norm(dim=-1)).median()) > 0.2
    eng = engine_for(tmp_path, cfg, t, dtype, f"side{side}")
    assert_rows_close(run_cut(eng, ids, [50]), want, dtype, "whole")
    assert_rows_close(run_cut(eng, ids, [3, 2], then_single=45), want, dtype, "single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_layer_run_twice_keeps_two_states(tmp_path, dtype):
    """A schedule that names a layer twice keeps two states and two caches for it."""
    import dataclasses
    from zlm_b200 import Engine
    from zlm_b200.config.spec import ScheduleEntry
    from zlm_b200.registry import config_from_dict
    cfg = model([layer({"width": 24}, dense(32)), layer(lat(2, 16, 8, 16, 24, 16, 0.5, rot=(100.0, 8), window=20), None)], 90, 64, 3, 8)
    t = make_tensors(cfg, 71)
    ids = prompts(90, [70], seed=8)[0]
    config = config_from_dict(cfg)
    spec = config.to_model_spec()
    twice = dataclasses.replace(spec, schedule=(ScheduleEntry(0), ScheduleEntry(1), ScheduleEntry(0), ScheduleEntry(1)))
    holder = SimpleNamespace(to_model_spec=lambda: twice)
    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    tensors = {n: (x.to(dt)).cuda() for n, x in t.items()}
    eng = Engine(holder, tensors, dt, "cuda:0", 1024)
    # the plain model with the layers copied (and with them their columns of the side table)
    big = copy.deepcopy(cfg)
    big["layers"] = big["layers"] + copy.deepcopy(big["layers"])
    ref = {n: x.double() for n, x in t.items()}
    for n in list(ref):
        for i in (0, 1):
            if n.startswith(f"l{i}."):
                ref[f"l{i + 2}." + n[3:]] = ref[n]
    ref["side.embed"] = torch.cat([ref["side.embed"], ref["side.embed"]], 1)
    want = P.forward(big, ref, ids)[0]
    assert_rows_close(run_cut(eng, ids, [70]), want, dtype, "whole")
    assert_rows_close(run_cut(eng, ids, [30, 2], then_single=38), want, dtype, "portions, then single tokens")
