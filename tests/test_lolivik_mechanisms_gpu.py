"""Lolivik's mechanisms one at a time on the GPU, each as a small model run through the engine (or as the kernel alone)
against the function of the plain implementation, with weights and inputs made so that a fault shows: attention so peaked
that single keys carry a query's weight (the plain implementation is first asked whether a window that is one token off, a
first token more or less, another constant, would change the answer: it must), memories whose gates keep hundreds of tokens,
or forget at once."""
import dataclasses
from types import SimpleNamespace

import pytest
import torch

import plain_lolivik as P
from lolivik_helpers import (assert_rows_close, att, changed, dense, engine_for, layer, make_tensors, mem, model, moe, one_layer,
                             oracle, prompts, win)

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
F64 = torch.float64


def torch_dtype(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


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


def doubles(tensors):
    return {n: x.double() for n, x in tensors.items()}


def rel(other, want):
    return (other - want).norm(dim=-1) / want.norm(dim=-1)


def moves(cfg, path, value, ref, ids, want, after=0, by=0.02, at_least=2):
    """Asks the plain implementation whether it gives other logits with one value of the configuration replaced."""
    other = P.forward(changed(cfg, path, value), ref, ids)[0]
    assert int((rel(other, want)[after:] > by).sum()) >= at_least, f"{path}={value} would not show"


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
                           max_len=max(s + n for s, n in zip(starts, lens)), is_decode=all(n == 1 for n in lens), scratch=scratch)


# ------------------------------------------------------------------------------------------------ the attention kernels
def attend_in_pages(dtype, H, G, hd, vd, lens, starts, impl=None, **opt):
    """The attention kernel on sequences whose keys and values lie in shuffled pages (whatever a query must not read is
    there too, and pages that no query may touch hold NaN), against the plain attention; -> (got, want) per sequence."""
    from zlm_b200.kernels import PAGE_TOKENS, get_kernels, pad_bias
    k = get_kernels()
    dt = torch_dtype(dtype)
    g = torch.Generator().manual_seed(H * 1000 + hd + sum(lens))
    R = len(lens)
    pages = [-(-(s + n) // PAGE_TOKENS) for s, n in zip(starts, lens)]
    order = torch.randperm(sum(pages) + 3, generator=g).tolist()
    table = torch.zeros(R, max(pages) + 1, dtype=torch.int32)
    pool = torch.zeros(sum(pages) + 3, 2, G, PAGE_TOKENS, hd)
    qs, seqs, at = [], [], 0
    window, keep = opt.get("window", 0), opt.get("keep", 0)
    for r in range(R):
        n = starts[r] + lens[r]
        kk = (torch.randn(n, G, hd, generator=g) * 1.3).to(dt)
        vv = torch.zeros(n, G, hd).to(dt)
        vv[..., :vd] = torch.randn(n, G, vd, generator=g).to(dt)
        q = (torch.randn(n, H, hd, generator=g) * 1.3).to(dt)
        first_seen = max(0, starts[r] + 1 - window) if window else 0
        for p in range(pages[r]):
            page = order[at + p]
            table[r, p] = page
            m = min(PAGE_TOKENS, n - p * PAGE_TOKENS)
            pool[page, 0, :, :m] = kk[p * 64:p * 64 + m].float().transpose(0, 1)
            pool[page, 1, :, :m] = vv[p * 64:p * 64 + m].float().transpose(0, 1)
            if (p + 1) * PAGE_TOKENS <= first_seen and p * PAGE_TOKENS >= keep:
                pool[page] = float("nan")                         # a page that has been given back
        at += pages[r]
        qs.append(q)
        seqs.append((q, kk, vv))
    plan = plan_for(lens, starts, list(range(R)))
    plan.attention_impl = impl
    q_new = torch.cat([q[s:] for q, s in zip(qs, starts)]).reshape(plan.T, H * hd).cuda()
    out = torch.full((plan.T, H * hd), 7.0, dtype=dt, device="cuda")
    scale = 0.7 * hd ** -0.5
    sinks, bias = opt.get("sinks"), opt.get("bias")
    k.attention(out, q_new, pool.to(dt).cuda(), table.cuda(), plan.token_pos, plan.token_slot, H, G, hd, scale, window, plan,
                v_dim=vd if vd < hd else None, softcap=opt.get("softcap", 0.0), keep=keep,
                sinks=None if sinks is None else sinks.cuda(), bias=None if bias is None else pad_bias(bias).cuda())
    got = out.cpu().view(plan.T, H, hd)
    assert vd == hd or float(got[..., vd:].float().abs().max()) == 0.0
    pairs, at = [], 0
    for r, (q, kk, vv) in enumerate(seqs):
        n = starts[r] + lens[r]
        b = None
        if bias is not None:
            far = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).clamp(0, bias.shape[1] - 1)
            b = bias.to(F64).t()[far]
        want = P.attend(q.to(F64), kk.to(F64), vv[..., :vd].to(F64), scale,
                        P.window_with_first_tokens(n, {"size": window, "keep_first": keep} if window else None),
                        opt.get("softcap", 0.0), b, None if sinks is None else sinks.to(F64))
        pairs.append((got[at:at + lens[r], :, :vd].reshape(lens[r], H * vd), want[starts[r]:]))
        at += lens[r]
    return pairs


# (heads, key heads, key width, value width): the widths pick the form of the kernel
FORMS = {"plain": (3, 3, 16, 16), "odd": (5, 1, 32, 32), "narrow values": (4, 2, 48, 32), "two heads a block": (4, 1, 128, 128),
         "one head a block": (3, 1, 128, 128), "many heads": (18, 1, 64, 64), "wide": (2, 1, 192, 192)}
STEPS = {"prompts": ([200, 1, 333, 64], [0, 0, 0, 0]), "portions": ([2, 150, 70, 129], [300, 61, 64, 250]),
         "decode": ([1, 1, 1, 1, 1], [0, 5, 63, 64, 700])}


def check_pairs(pairs, dtype, what):
    for r, (got, want) in enumerate(pairs):
        assert_rows_close(got, want, dtype, f"{what}, sequence {r}", 2e-5 if dtype == "float32" else 2e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("form", sorted(FORMS))
@pytest.mark.parametrize("step", sorted(STEPS))
@pytest.mark.parametrize("far,softcap", [(20, 5.0), (300, 0.0), (64, 8.0), (150, 40.0), (1, 0.0)])
def test_bias_by_distance_in_every_form(dtype, form, step, far, softcap):
    """A bias of order 2 that differs from distance to distance, alone and with a cap and sinks (which it must not pass
    through; caps that most scores reach half of, and one that none does), tables that end inside a tile, beyond the sequences, and after one entry."""
    H, G, hd, vd = FORMS[form]
    g = torch.Generator().manual_seed(far)
    bias = 2.0 * torch.randn(H, far + 1, generator=g)
    sinks = 2.0 * torch.randn(H, generator=g) if softcap else None
    check_pairs(attend_in_pages(dtype, H, G, hd, vd, *STEPS[step], bias=bias, softcap=softcap, sinks=sinks), dtype, "bias")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("form", sorted(FORMS))
@pytest.mark.parametrize("step", sorted(STEPS))
@pytest.mark.parametrize("window,keep", [(1, 1), (9, 2), (64, 64), (70, 5), (130, 70), (20, 200), (33, 0)])
def test_window_beside_first_tokens_in_every_form(dtype, form, step, window, keep):
    """Kept tokens of a few, a page, a little more than a page and more than some sequences have; pages between them and
    the window hold NaN."""
    H, G, hd, vd = FORMS[form]
    check_pairs(attend_in_pages(dtype, H, G, hd, vd, *STEPS[step], window=window, keep=keep), dtype, "window and first tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("step", sorted(STEPS))
@pytest.mark.parametrize("form", ["odd", "two heads a block"])
def test_bias_cap_sinks_window_and_first_tokens_together(dtype, step, form):
    H, G, hd, vd = FORMS[form]
    g = torch.Generator().manual_seed(4)
    check_pairs(attend_in_pages(dtype, H, G, hd, vd, *STEPS[step], window=70, keep=9, bias=2.0 * torch.randn(H, 51, generator=g),
                                softcap=6.0, sinks=torch.randn(H, generator=g)), dtype, "all of them")


@pytest.mark.parametrize("extra", ["bias", "keep", "both"])
def test_two_prefill_forms_agree(extra):
    """Heads of 128 through the tcgen05 form and the mma.sync form, one and two heads a block."""
    from zlm_b200.kernels import get_kernels
    g = torch.Generator().manual_seed(6)
    opt = {}
    if extra != "keep":
        opt.update(bias=2.0 * torch.randn(4, 140, generator=g), softcap=7.0)
    if extra != "bias":
        opt.update(window=100, keep=67)
    k = get_kernels()
    try:
        for heads in (1, 2):
            k.set_prefill_attention_heads(heads)
            for impl in (None, "mma"):
                check_pairs(attend_in_pages("bfloat16", 4, 2, 128, 128, [500, 3, 129], [0, 640, 77], impl=impl, **opt), "bfloat16",
                            f"{impl} {heads}")
    finally:
        k.set_prefill_attention_heads(0)


# ------------------------------------------------------------------------------------------------ attention layers
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep,sizes", [(9, 2, (2, 1, 24, 16)), (64, 1, (3, 3, 16, 24)), (70, 6, (4, 2, 40, 20)), (130, 66, (4, 2, 128, 128))])
def test_a_layer_sees_exactly_its_window_and_first_tokens(tmp_path, dtype, window, keep, sizes):
    """The plain implementation with a window or a number of first tokens that is one off gives other logits, the engine
    gives those of the right ones, in prompts, portions that start inside a window, and token by token while pages are
    given back."""
    H, G, D, V = sizes
    cfg = one_layer(win(H, G, D, V, 1.0 * D ** -0.5, window, keep, rot=(300.0, D // 4 * 2)))
    t = scaled(make_tensors(cfg, 11), {"l0.mix.q.norm": 3.0, "l0.norm1": 2.0})
    ref = doubles(t)
    n = window + keep + 75
    (ids,) = prompts(cfg["vocab"], [n], seed=window)
    want = P.forward(cfg, ref, ids)[0]
    for path, value in ((("size",), window + 1), (("size",), window - 1), (("keep_first",), keep + 1), (("keep_first",), keep - 1)):
        moves(cfg, ("layers", 0, "mixer", "mask") + path, value, ref, ids, want)
    eng = engine_for(tmp_path, cfg, t, dtype, f"win{window}")
    held = oracle(ref, cfg, ids, dtype)
    tol = None if dtype == "float32" else 0.12          # (peaked attention multiplies bfloat16's rounding of q and k)
    held.check(run_cut(eng, ids, [n]), range(n), dtype, "whole", tol)
    held.check(run_cut(eng, ids, [window - 1, 2, 3, n - window - 4]), range(n), dtype, "portions", tol)
    held.check(run_cut(eng, ids, [max(1, window - 3)], then_single=n - max(1, window - 3)), range(n), dtype, "token by token", tol)
    eng.cache.check()
    assert eng.cache.tokens_held() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(2, 1, 24, 16), (5, 5, 16, 40), (4, 2, 128, 128), (3, 3, 7, 5)])
def test_every_constant_of_the_biased_attention_shows(tmp_path, dtype, sizes):
    """Temperature, cap, largest distance and scale one by one in the plain implementation, then the table, the sinks and
    the norms over the whole projection: each moves the logits, the engine gives those of the right ones."""
    H, G, D, V = sizes
    cfg = one_layer(att(H, G, D, V, 1.5 * D ** -0.5, 50, softcap=4.0, temp=(0.5, 16)))
    t = scaled(make_tensors(cfg, 12), {"l0.mix.q.norm": 2.0, "l0.mix.rel": 1.5, "l0.norm1": 2.0})
    ref = doubles(t)
    (ids,) = prompts(cfg["vocab"], [210], seed=5)
    want = P.forward(cfg, ref, ids)[0]
    for path, value in ((("q_temp", "coef"), 0.3), (("q_temp", "every"), 20), (("softcap",), 6.0), (("bias_max",), 70),
                        (("scale",), 1.2 * D ** -0.5)):
        moves(cfg, ("layers", 0, "mixer") + path, value, ref, ids, want, at_least=20)
    for name, change in (("rel", lambda x: x.flip(0)), ("sink", lambda x: x + 2.0), ("k.norm", lambda x: x.flip(0))):
        moved = dict(ref, **{"l0.mix." + name: change(ref["l0.mix." + name])})
        assert int((rel(P.forward(cfg, moved, ids)[0], want) > 0.02).sum()) >= 20, name
    eng = engine_for(tmp_path, cfg, t, dtype, f"bias{H}")
    held = oracle(ref, cfg, ids, dtype)
    tol = None if dtype == "float32" else 0.12
    held.check(run_cut(eng, ids, [210]), range(210), dtype, "whole", tol)
    held.check(run_cut(eng, ids, [63, 2, 1, 62], then_single=82), range(210), dtype, "portions, then single tokens", tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(2, 1, 24, 16), (4, 2, 128, 128)])
def test_far_keys_count_without_a_window(tmp_path, dtype, sizes):
    """400 tokens: the values of early tokens reach the last queries, far beyond the bias table's largest distance."""
    H, G, D, V = sizes
    cfg = one_layer(att(H, G, D, V, 2.0 * D ** -0.5, 40, softcap=12.0, temp=(0.3, 64)))
    t = scaled(make_tensors(cfg, 13), {"l0.mix.q.norm": 2.0, "l0.norm1": 2.0})
    ref = doubles(t)
    (ids,) = prompts(cfg["vocab"], [400], seed=5)
    want = P.forward(cfg, ref, ids)[0]
    other = P.forward(cfg, ref, prompts(cfg["vocab"], [150], seed=6)[0] + ids[150:])[0]
    assert int((rel(other, want)[250:] > 0.05).sum()) >= 10, "far keys do not show"
    eng = engine_for(tmp_path, cfg, t, dtype, f"far{H}")
    held = oracle(ref, cfg, ids, dtype)
    tol = None if dtype == "float32" else 0.15
    held.check(run_cut(eng, ids, [400]), range(400), dtype, "whole", tol)
    held.check(run_cut(eng, ids, [190, 2, 140], then_single=68), range(400), dtype, "portions and single tokens", tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("order", ["aw", "wa", "mawa"])
def test_values_are_mixed_from_the_first_layer_that_mixes(tmp_path, dtype, order):
    """The first mixing layer of either kind, behind other layers too; every later layer's share of its values shows, also in
    decode steps, where what a layer hands on is made anew each step."""
    kinds = {"a": att(3, 1, 16, 24, 0.4, 30, v_mix=True), "w": win(2, 2, 24, 12, 0.3, 40, 3, v_mix=True), "m": mem(2, 16, 16, 5.0)}
    cfg = model([layer(kinds[c], None) for c in order], 90, 64, mult=0.8)
    t = make_tensors(cfg, 14)
    ref = doubles(t)
    (ids,) = prompts(90, [110], seed=8)
    want = P.forward(cfg, ref, ids)[0]
    mixing = [i for i, c in enumerate(order) if c != "m"]
    for i in mixing[1:]:
        moved = dict(ref, **{f"l{i}.mix.vmix": ref[f"l{i}.mix.vmix"] * 0.5})
        assert float(rel(P.forward(cfg, moved, ids)[0], want).median()) > 0.02
    moved = dict(ref, **{f"l{mixing[0]}.mix.vmix": ref[f"l{mixing[0]}.mix.vmix"] + 9.0})         # (the first one's is unused)
    assert torch.equal(P.forward(cfg, moved, ids)[0], want)
    eng = engine_for(tmp_path, cfg, t, dtype, f"vmix{order}")
    assert_rows_close(run_cut(eng, ids, [110]), want, dtype, "whole")
    assert_rows_close(run_cut(eng, ids, [2, 30, 3], then_single=75), want, dtype, "portions, then single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("norm", ["head", "row"])
@pytest.mark.parametrize("interleaved", [False, True])
def test_preparation_kernel(dtype, norm, interleaved):
    """attn_prep alone: norm, rotation either way at far positions, temperature, mixed values, what the next layers get,
    padding, and places in the cache."""
    from zlm_b200.kernels import PAGE_TOKENS, get_kernels
    k = get_kernels()
    dt = torch_dtype(dtype)
    g = torch.Generator().manual_seed(3)
    H, G, D, V, hdp, n_rot, eps, lam, temp = 4, 2, 12, 20, 32, 8, 1e-3, 0.375, (0.5, 16)
    plan = plan_for([3, 2], [62, 1000], [1, 0])
    T, C = plan.T, (H + G) * D + G * V
    proj = torch.randn(T, C + 3, generator=g).to(dt)
    qw, kw = (1 + torch.randn(D if norm == "head" else H * D, generator=g)), (1 + torch.randn(D if norm == "head" else G * D, generator=g))
    inv = torch.tensor([50.0 ** (-2 * i / n_rot) for i in range(n_rot // 2)], dtype=torch.float32)
    table = torch.arange(40, dtype=torch.int32).flip(0).view(2, 20).contiguous().cuda()
    pool = torch.zeros(40, 2, G, PAGE_TOKENS, hdp, dtype=dt, device="cuda")
    first, keep = torch.randn(T, G * V, generator=g).to(dt), torch.zeros(T, G * V, dtype=dt, device="cuda")
    q_out = torch.full((T, H * hdp), 9.0, dtype=dt, device="cuda")
    k.attn_prep(q_out, proj.cuda(), None, None, plan, table, pool, H, G, D, V, 1, norm, qw.cuda(), kw.cuda(), eps, inv.cuda(), n_rot,
                interleaved=interleaved, q_temp=temp, v_first=first.cuda(), v_lambda=lam, v_keep=keep)
    d, pos = proj.to(F64), plan.token_pos.cpu().long()

    def prepared(x, heads, w):
        x = P.rms_norm(x.view(T, heads, D), w.to(F64), eps) if norm == "head" else P.rms_norm(x, w.to(F64), eps).view(T, heads, D)
        a = pos.to(F64)[:, None, None] * inv.to(F64)
        u, v = (x[..., 0:n_rot:2], x[..., 1:n_rot:2]) if interleaved else (x[..., :n_rot // 2], x[..., n_rot // 2:n_rot])
        y = x.clone()
        ru, rv = u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)
        if interleaved:
            y[..., 0:n_rot:2], y[..., 1:n_rot:2] = ru, rv
        else:
            y[..., :n_rot // 2], y[..., n_rot // 2:n_rot] = ru, rv
        return y
    temps = P.query_temperature(1100, {"coef": temp[0], "every": temp[1]})[pos]
    tol = 2e-5 if dtype == "float32" else 6e-3
    got_q = q_out.cpu().view(T, H, hdp)
    assert_rows_close(got_q[..., :D].reshape(T, -1), (prepared(d[:, :H * D], H, qw) * temps[:, None, None]).reshape(T, -1), dtype, "q", tol)
    assert float(got_q[..., D:].float().abs().max()) == 0.0
    slot = plan.token_slot.cpu().long()
    at = table.cpu().long()[slot, pos // PAGE_TOKENS]
    rows = pool.cpu()[at, :, :, pos % PAGE_TOKENS]                           # [T, 2, G, hdp]
    assert_rows_close(rows[:, 0, :, :D].reshape(T, -1), prepared(d[:, H * D:(H + G) * D], G, kw).reshape(T, -1), dtype, "k", tol)
    v = d[:, (H + G) * D:C]
    assert_rows_close(rows[:, 1, :, :V].reshape(T, -1), (1 - lam) * v + lam * first.to(F64), dtype, "v", tol)
    assert torch.equal(keep.cpu(), proj[:, (H + G) * D:C])
    assert float(rows[:, 0, :, D:].float().abs().max()) == 0.0 and float(rows[:, 1, :, V:].float().abs().max()) == 0.0


# ------------------------------------------------------------------------------------------------ the matrix memory
MEMORIES = [(3, 24, 20), (1, 37, 6), (2, 128, 128), (4, 16, 300), (2, 200, 64), (1, 1, 1)]


def memory_case(dtype, H, D, V, lens, forget, big, seed=0):
    """A projection, gate logits, biases and states that are not zero, and what the plain recurrence makes of them."""
    dt = torch_dtype(dtype)
    g = torch.Generator().manual_seed(seed + D + len(lens))
    T, R = sum(lens), len(lens)
    off = {"q": 8, "k": 8 + H * D, "v": 8 + 2 * H * D, "g": 8 + 2 * H * D + H * V}
    proj = torch.randn(T, off["g"] + H * V, generator=g).to(dt)
    z = torch.randn(T, 2 * H + 1, generator=g) * big
    bi, bf = torch.randn(H, generator=g).to(dt), (torch.randn(H, generator=g) + forget).to(dt)
    slots = list(range(R))[::-1]
    state = (torch.randn(R, H, D, V, generator=g), torch.randn(R, H, D, generator=g), torch.randn(R, H, generator=g))
    cap = 6.0
    want, ends, at = [], {}, 0
    d = proj.to(F64)
    for r, n in enumerate(lens):
        row = slice(at, at + n)
        i = P.softcap(z[row, :H].to(F64) + bi.to(F64), cap)
        f = torch.nn.functional.logsigmoid(P.softcap(z[row, H + 1:].to(F64) + bf.to(F64), cap))
        cut = lambda name, w: d[row, off[name]:off[name] + H * w].reshape(n, H, w)
        o, end = P.matrix_memory(cut("q", D) * D ** -0.5, cut("k", D), cut("v", V), i, f, tuple(s[slots[r]].to(F64) for s in state))
        want.append(o.reshape(n, H * V))
        ends[slots[r]] = end
        at += n
    dev = tuple(s.cuda().clone() for s in state)
    args = (z.cuda(), 0, H + 1, bi.cuda(), bf.cuda(), cap, dev, plan_for(lens, [7] * R, slots), H, D, V, D ** -0.5)
    return proj, off, args, torch.cat(want), ends, dev


def check_states(dev, ends, tol=2e-5):
    for slot, end in ends.items():
        for name, got, want in zip("Snm", dev, end):
            assert_rows_close(got[slot].reshape(1, -1), want.reshape(1, -1), "float32", f"{name} of slot {slot}", tol)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,V", MEMORIES)
@pytest.mark.parametrize("lens", [[1, 2], [64, 65, 63], [300, 1, 17, 129]])
@pytest.mark.parametrize("forget,big", [(4.0, 1.0), (0.0, 3.0), (-6.0, 5.0)])
def test_matrix_memory_in_pieces(dtype, H, D, V, lens, forget, big):
    """The kernels alone from states that are not zero: memories that last, gates all over their range, and memories that
    forget a token at once (their logarithms add up to hundreds inside a piece)."""
    from zlm_b200.kernels import get_kernels
    proj, off, args, want, ends, dev = memory_case(dtype, H, D, V, lens, forget, big)
    o = torch.full((sum(lens), H * V), float("nan"), device="cuda")
    get_kernels().mlstm(o, proj.cuda(), off["q"], off["k"], off["v"], *args)
    # (whatever the element type, all that follows the projection is fp32; a denominator near zero multiplies its rounding)
    assert_rows_close(o, want, "float32", "read-out", 2e-4 if D > 1 else 2e-3)
    check_states(dev, ends)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,V", MEMORIES)
@pytest.mark.parametrize("forget,big", [(4.0, 1.0), (0.0, 3.0), (-6.0, 5.0)])
@pytest.mark.parametrize("proj32", [False, True])
def test_matrix_memory_one_token_with_norm_and_gate(dtype, H, D, V, forget, big, proj32):
    """The decode kernel alone: the same recurrence, the heads' norm and the gate; the projection in fp32 too."""
    from zlm_b200.kernels import get_kernels
    R, eps = 5, 1e-5
    dt = torch_dtype(dtype)
    proj, off, args, want, ends, dev = memory_case(dtype, H, D, V, [1] * R, forget, big, seed=9)
    w = 1 + 0.3 * torch.randn(H * V, generator=torch.Generator().manual_seed(2))
    out = torch.full((R, H * V + 4), 9.0, dtype=dt, device="cuda")
    p = proj.float().cuda() if proj32 else proj.cuda()
    get_kernels().mlstm_step(out[:, :H * V], p, off["q"], off["k"], off["v"], off["g"], *args, w.cuda(), eps)
    gate = torch.sigmoid(proj.to(F64)[:, off["g"]:])
    want = P.rms_norm(want.view(R, H, V), None, eps).reshape(R, H * V) * w.to(F64) * gate
    assert_rows_close(out[:, :H * V], want, dtype, "out", 2e-4 if dtype == "float32" else 8e-3)
    assert float((out[:, H * V:].float() - 9.0).abs().max()) == 0.0
    check_states(dev, ends)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(3, 24, 20), (1, 37, 6), (2, 64, 64)])
def test_memories_reach_far_back(tmp_path, dtype, sizes):
    """Forget gates near one: 500 tokens whole (pieces side by side), in portions, then token by token; two sequences side by
    side; a slot used again starts from nothing."""
    from zlm_b200 import StepEntry
    cfg = one_layer(mem(*sizes, 9.0), dense(32))
    t = make_tensors(cfg, 21)
    t["l0.mix.f.b"] = (t["l0.mix.f.b"] + 4.0).to(torch.bfloat16).float()
    t = scaled(t, {"l0.norm1": 2.0})
    ref = doubles(t)
    a, b = prompts(cfg["vocab"], [500, 37], seed=9)
    want = P.forward(cfg, ref, a)[0]
    other = P.forward(cfg, ref, prompts(cfg["vocab"], [150], seed=4)[0] + a[150:])[0]
    assert float(rel(other, want)[160:250].median()) > 0.02, "the memory does not show"
    eng = engine_for(tmp_path, cfg, t, dtype, f"mem{sizes[0]}")
    assert_rows_close(run_cut(eng, a, [500]), want, dtype, "whole")
    assert_rows_close(run_cut(eng, a, [1, 2, 1, 3, 250, 2, 200], then_single=41), want, dtype, "portions, then single tokens")
    s1, s2 = eng.new_sequence(), eng.new_sequence()
    got = eng.step([StepEntry(s1, b, [36]), StepEntry(s2, a[:200], [99, 199])]).clone()
    assert_rows_close(got, torch.stack([P.forward(cfg, ref, b)[0][36], want[99], want[199]]), dtype, "side by side")
    got = eng.step([StepEntry(s1, a[:5], []), StepEntry(s2, a[200:210], [9])]).clone()
    assert_rows_close(got, want[209:210], dtype, "going on from the pieces' state")
    got = eng.step([StepEntry(s1, a[:1], []), StepEntry(s2, a[210:211], [0])]).clone()
    assert_rows_close(got, want[210:211], dtype, "and from a portion's")


@pytest.mark.parametrize("dtype", DTYPES)
def test_gates_far_below_zero(tmp_path, dtype):
    """Input gates so small that the denominator's floor exp(-m) holds and the heads' norm feels its eps: a constant on all
    input gates then counts (where the floor does not hold it cancels); the cap of the gates shows too; from the very first
    token on, whose maximum starts from 0."""
    cfg = one_layer(mem(2, 16, 24, 6.0))
    t = make_tensors(cfg, 22)
    t["l0.mix.i.b"] = (t["l0.mix.i.b"] * 0.2 - 3.0).to(torch.bfloat16).float()
    t = scaled(t, {"l0.norm1": 2.0, "l0.mix.o": 0.02})
    cfg["norm"]["eps"] = 1e-3
    ref = doubles(t)
    (ids,) = prompts(cfg["vocab"], [80], seed=2)
    want = P.forward(cfg, ref, ids)[0]
    moves(cfg, ("layers", 0, "mixer", "gate_cap"), 9.0, ref, ids, want, at_least=5)
    other = P.forward(cfg, dict(ref, **{"l0.mix.i.b": ref["l0.mix.i.b"] - 1.0}), ids)[0]
    assert bool((rel(other, want)[:3] > 0.02).all())
    eng = engine_for(tmp_path, cfg, t, dtype, "low")
    assert_rows_close(run_cut(eng, ids, [80]), want, dtype, "whole")
    assert_rows_close(run_cut(eng, ids, [], then_single=80), want, dtype, "token by token")


# ------------------------------------------------------------------------------------------------ feed-forwards, norms
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("r", [(8, 3, 24, (40, 0.9)), (6, 1, 32, None), (4, 4, 16, (16, 2.0)), (5, 2, 11, (13, 0.5)), (12, 2, 128, (64, 1.0))])
def test_routed_layer_against_the_plain_one(tmp_path, dtype, r):
    """Few tokens and many (the grouped product), widths that are padded, all experts chosen; both clamps show, each alone."""
    experts, top, ff, shared = r
    cfg = one_layer(mem(2, 8, 8, 5.0), moe(ff, experts, top, 0.7, shared))
    t = scaled(make_tensors(cfg, 51), {"l0.norm2": 2.0})
    ref = doubles(t)
    (ids,) = prompts(cfg["vocab"], [150], seed=3)
    want = P.forward(cfg, ref, ids)[0]
    moves(cfg, ("layers", 0, "mlp", "expert", "limit"), 1.0, ref, ids, want, at_least=20)
    if shared:
        moves(cfg, ("layers", 0, "mlp", "shared", "limit"), shared[1] * 1.5, ref, ids, want, at_least=20)
    eng = engine_for(tmp_path, cfg, t, dtype, f"moe{experts}")
    held = oracle(ref, cfg, ids, dtype)
    held.check(run_cut(eng, ids, [150]), range(150), dtype, "150 tokens")
    held.check(run_cut(eng, ids, [3, 16, 17], then_single=20), range(56), dtype, "few tokens")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("interleaved", [False, True])
@pytest.mark.parametrize("limit,alpha", [(0.5, 1.702), (3.0, 0.8)])
def test_clamped_experts_kernel(dtype, interleaved, limit, alpha):
    """moe_up alone: halves beyond both limits, weights on the output, both layouts."""
    from zlm_b200.kernels import get_kernels, interleave_gate_up
    dt = torch_dtype(dtype)
    g = torch.Generator().manual_seed(7)
    T, E, top, F, K = 5, 4, 2, 24, 40
    x = (2.0 * torch.randn(T, K, generator=g)).to(dt)
    gate, up = (torch.randn(E, F, K, generator=g).to(dt) / 4 for _ in range(2))
    w = torch.stack([interleave_gate_up(a, b) if interleaved else torch.cat([a, b]) for a, b in zip(gate, up)]).contiguous()
    idx = torch.randint(0, E, (T, top), generator=g).int()
    wgt = torch.rand(T, top, generator=g)
    act = torch.empty(T, top, F, dtype=dt, device="cuda")
    get_kernels().moe_up(act, x.cuda(), w.cuda(), idx.cuda(), wgt.cuda(), False, "swish_limit" + ("_interleaved" if interleaved else ""),
                         limit=limit, alpha=alpha)
    for t in range(T):
        for j in range(top):
            e = int(idx[t, j])
            a = (gate[e].to(F64) @ x[t].to(F64)).clamp_max(limit)
            b = (up[e].to(F64) @ x[t].to(F64)).clamp(-limit, limit)
            assert_rows_close(act[t, j], a * torch.sigmoid(alpha * a) * (b + 1) * float(wgt[t, j]), dtype, "act", 1e-5 if dtype == "float32" else 6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff", [37, 96])
def test_dense_feed_forward(tmp_path, dtype, ff):
    """Widths that are padded and that are not; the multiplier of the sublayers' norms shows."""
    cfg = one_layer(mem(2, 8, 8, 5.0), dense(ff))
    t = scaled(make_tensors(cfg, 41), {"l0.norm2": 2.0})
    ref = doubles(t)
    (ids,) = prompts(cfg["vocab"], [90], seed=3)
    want = P.forward(cfg, ref, ids)[0]
    moves(cfg, ("residual_mult",), 0.7, ref, ids, want, at_least=50)
    eng = engine_for(tmp_path, cfg, t, dtype, f"dense{ff}")
    assert_rows_close(run_cut(eng, ids, [90]), want, dtype, "whole")
    assert_rows_close(run_cut(eng, ids, [5], then_single=85), want, dtype, "single tokens")


@pytest.mark.parametrize("dtype", DTYPES)
def test_padded_weights_read_back_as_they_were(tmp_path, dtype):
    """Widths that the bfloat16 products pad, gates interleaved with up rows, norms with the multiplier folded in."""
    cfg = model([layer(mem(3, 9, 13, 4.0), moe(11, 3, 2, 0.7, (13, 0.9))), layer(att(3, 1, 7, 5, 0.4, 20), dense(37))], 70, 40)
    t = make_tensors(cfg, 61)
    eng = engine_for(tmp_path, cfg, t, dtype, "read")
    for n, x in t.items():
        assert torch.equal(eng.tensor(n).float().cpu().reshape(x.shape), x), n


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_layer_run_twice_keeps_two_memories_and_caches(tmp_path, dtype):
    """A schedule that names every layer twice keeps two states and two caches for each."""
    from zlm_b200 import Engine
    from zlm_b200.config.spec import ScheduleEntry
    from zlm_b200.registry import config_from_dict
    cfg = model([layer(mem(2, 16, 12, 5.0), dense(32)), layer(win(2, 1, 16, 16, 0.5, 20, 4, rot=(100.0, 8)), None)], 90, 64)
    t = make_tensors(cfg, 71)
    ids = prompts(90, [70], seed=8)[0]
    spec = config_from_dict(cfg).to_model_spec()
    twice = dataclasses.replace(spec, schedule=tuple(ScheduleEntry(i) for i in (0, 1, 0, 1)))
    dt = torch_dtype(dtype)
    eng = Engine(SimpleNamespace(to_model_spec=lambda: twice), {n: x.to(dt).cuda() for n, x in t.items()}, dt, "cuda:0", 1024)
    big = dict(cfg, layers=cfg["layers"] * 2)
    ref = doubles(t)
    for n in list(ref):
        if n[:3] in ("l0.", "l1."):
            ref[f"l{int(n[1]) + 2}." + n[3:]] = ref[n]
    want = P.forward(big, ref, ids)[0]
    assert_rows_close(run_cut(eng, ids, [70]), want, dtype, "whole")
    assert_rows_close(run_cut(eng, ids, [30, 2], then_single=38), want, dtype, "portions, then single tokens")
