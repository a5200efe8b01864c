"""Per-operation timing of a step, in the manner of the reference's ``run --profile``
(per-op nanoseconds, weight bytes per token and matvec GB/s:
src/cli/commands/run.zig:233-299, counters filled in src/runtime/executor.zig:104-128).

``ProfilingKernels`` stands in the kernel object's place (parts never launch anything
themselves, they call ``rt.k``): every call is bracketed by two CUDA events on the
launching stream and filed under the operation's name, with the bytes it has to move and
the floating-point operations it has to do, counted from its arguments.  Steps run
eagerly (no graph) while it is in place.  So that the times are the kernels' and not the
host's launch gaps, a profiled step begins with a short device-side wait that lets the
host queue the step's launches ahead.

Events around every launch are right for the long kernels of a prefill.  The kernels of a
decode step take a few microseconds each, as long as an event and the launch gap beside it;
for them ``mode="graph"`` only notes the calls of one step, and ``table`` then captures, for
each operation, all its calls of the step (one per layer, each with that layer's own
weights, which together are far larger than L2) as one CUDA graph, replays it, and divides
its time by the number of calls: the operation as it runs inside a captured step, weights
streaming from HBM.

``profile_engine`` runs one prefill and some decode steps this way and returns a table.
"""
from __future__ import annotations

from collections import OrderedDict
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from .parts.base import Part


@dataclass
class OpRecord:
    calls: int = 0
    bytes: float = 0.0
    flops: float = 0.0
    events: List[Tuple[torch.cuda.Event, torch.cuda.Event]] = field(default_factory=list)
    noted: List = field(default_factory=list)       # graph mode: the calls, to be replayed
    ms: float = 0.0

    def settle(self) -> None:
        for a, b in self.events:
            self.ms += a.elapsed_time(b)
        self.events = []


def _nbytes(t: Optional[torch.Tensor]) -> int:
    return 0 if t is None else t.numel() * t.element_size()


class ProfilingKernels:
    """Wraps a kernel object; same methods, timed."""

    name = "profiling"

    def __init__(self, kernels, weight_names: Optional[Dict[int, str]] = None, mode: str = "events",
                 pdl: bool = False):
        self.k = kernels
        self.weight_names = weight_names or {}
        self.mode = mode
        self.pdl = pdl          # graph mode: capture with programmatic dependent launch, as the decode runner does
        self.phase = "step"
        self.records: "OrderedDict[Tuple[str, str], OpRecord]" = OrderedDict()

    def __getattr__(self, name):
        # whatever is not timed here (status, scratch, settings) goes to the real object
        return getattr(self.k, name)

    # ------------------------------------------------------------------ bookkeeping
    def _timed(self, op: str, nbytes: float, flops: float, fn, *args, **kw):
        rec = self.records.setdefault((self.phase, op), OpRecord())
        if self.mode == "graph":
            rec.calls += 1
            rec.bytes += nbytes
            rec.flops += flops
            rec.noted.append((fn, args, kw))
            return fn(*args, **kw)
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        out = fn(*args, **kw)
        e1.record()
        rec.calls += 1
        rec.bytes += nbytes
        rec.flops += flops
        rec.events.append((e0, e1))
        return out

    def run_ahead(self, microseconds: int = 2000) -> None:
        """Keeps the device busy for a moment so that the host can queue launches ahead."""
        sleep = getattr(torch.cuda, "_sleep", None)
        if sleep is not None:
            sleep(int(microseconds * 1900))         # cycles at about 1.9 GHz

    def _replay_noted(self, rec: OpRecord, repeats: int = 5) -> None:
        """All noted calls of one operation as one graph; the best of a few replays."""
        import gc
        torch.cuda.synchronize()
        g = torch.cuda.CUDAGraph()
        gc.collect()
        if self.pdl:
            self.k.set_pdl(True)
        try:
            with torch.cuda.graph(g):
                for fn, args, kw in rec.noted:
                    fn(*args, **kw)
        finally:
            if self.pdl:
                self.k.set_pdl(False)
        best = None
        for _ in range(repeats + 1):
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            g.replay()
            e1.record()
            torch.cuda.synchronize()
            t = e0.elapsed_time(e1)
            best = t if best is None else min(best, t)
        rec.ms = best
        rec.noted = []

    def table(self) -> List[dict]:
        torch.cuda.synchronize()
        rows = []
        for (phase, op), r in self.records.items():
            if r.noted:
                self._replay_noted(r)
            r.settle()
            us = r.ms * 1e3 / max(1, r.calls)
            sec = r.ms * 1e-3
            rows.append({"phase": phase, "op": op, "calls": r.calls, "us_per_call": round(us, 2),
                         "total_ms": round(r.ms, 4), "mb_per_call": round(r.bytes / max(1, r.calls) / 1e6, 3),
                         "gb_s": round(r.bytes / sec / 1e9, 1) if sec > 0 else 0.0,
                         "tflop_s": round(r.flops / sec / 1e12, 2) if sec > 0 else 0.0})
        return rows

    # ------------------------------------------------------------------ the kernels
    def embed(self, out, table, ids):
        n = _nbytes(out) + out.shape[0] * out.shape[1] * table.element_size()
        return self._timed("embed", n, 0, self.k.embed, out, table, ids)

    def rmsnorm(self, out, x, w, eps, rows=None):
        R, H = out.shape
        return self._timed("rmsnorm", R * H * 4 + _nbytes(out) + _nbytes(w), 0, self.k.rmsnorm, out, x, w, eps, rows)

    def swiglu(self, out, gu):
        return self._timed("swiglu", _nbytes(out) + _nbytes(gu), 0, self.k.swiglu, out, gu)

    def _linear_name(self, w, kind: str) -> str:
        return f"{kind} {self.weight_names.get(w.data_ptr(), f'[{w.shape[0]}x{w.shape[1]}]')}"

    def linear(self, out, x, w, accumulate=False, impl=None, defer=False):
        T, K = x.shape
        N = w.shape[0]
        n = _nbytes(w) + T * K * x.element_size() + T * N * out.element_size() * (2 if accumulate else 1)
        # graph mode times every operation by itself, so a product is finished where it is issued
        return self._timed(self._linear_name(w, "linear"), n, 2.0 * T * N * K, self.k.linear, out, x, w,
                           accumulate=accumulate, impl=impl, defer=defer and self.mode != "graph")

    def linear_swiglu(self, out, x, w, impl=None, **kw):
        T, K = x.shape
        N = w.shape[0]
        n = _nbytes(w) + T * K * x.element_size() + _nbytes(out)
        return self._timed(self._linear_name(w, "linear+swiglu"), n, 2.0 * T * N * K, self.k.linear_swiglu, out, x, w,
                           impl=impl, **kw)

    def rope_table(self, out, inv_freq, n_rot, token_pos):
        return self._timed("rope_table", _nbytes(out), 0, self.k.rope_table, out, inv_freq, n_rot, token_pos)

    def linear_qkv_rope(self, q_out, x, w, *args, **kw):
        T, K = x.shape
        N = w.shape[0]
        n = _nbytes(w) + T * K * x.element_size() + T * N * q_out.element_size()
        return self._timed(self._linear_name(w, "linear+qk_norm+rope+cache_write"), n, 2.0 * T * N * K,
                           self.k.linear_qkv_rope, q_out, x, w, *args, **kw)

    def qk_norm_rope_write(self, qkv, q_w, k_w, eps, inv_freq, n_rot, token_pos, token_slot, block_table, pool,
                           nq, nkv, hd, write=True):
        T, el = qkv.shape[0], qkv.element_size()
        n = T * (nq + 2 * nkv) * hd * el + T * nq * hd * el + T * 2 * nkv * hd * el
        return self._timed("qk_norm+rope+cache_write", n, 0, self.k.qk_norm_rope_write, qkv, q_w, k_w, eps, inv_freq,
                           n_rot, token_pos, token_slot, block_table, pool, nq, nkv, hd, write)

    @staticmethod
    def _reach(plan, window: int, chunk: int, keep: int = 0):
        """(keys the step reads of the cache, query-key pairs it scores) from the step's host-side plan."""
        def first(p):
            lo = max(0, p + 1 - window) if window else 0
            return max(lo, p - p % chunk) if chunk else lo
        keys_read, pairs = 0, 0
        if plan is not None and getattr(plan, "h_seq_start", None):
            for start, new in zip(plan.h_seq_start, plan.h_seq_new):
                end = start + new
                keys_read += end - first(start) + min(keep, first(start))
                for p in range(start, end):                 # visible keys of each new token
                    pairs += (p + 1) - first(p) + min(keep, first(p))
        return keys_read, pairs

    def attention(self, out, q, pool, block_table, token_pos, token_slot, nq, nkv, hd, scale, window, plan=None,
                  len_bucket=None, v_dim=None, sink=False, chunk=0, v_share=1, keep=0, bias=None, **kw):
        T, el = q.shape[0], q.element_size()
        keys_read, pairs = self._reach(plan, window, chunk, keep)
        n = 2 * T * nq * hd * el + keys_read * (nkv + nkv // v_share) * hd * pool.element_size()
        kind = "attention decode" if (plan is not None and plan.is_decode) else "attention prefill"
        if v_share > 1:
            kind += ", %d maps on one value head" % v_share
        kind += (", bias by distance" if bias is not None else "") + (", first tokens kept" if keep else "")
        return self._timed(kind, n, 2.0 * nq * (hd + (v_dim or hd)) * pairs, self.k.attention, out, q, pool, block_table,
                           token_pos, token_slot, nq, nkv, hd, scale, window, plan, len_bucket=len_bucket, v_dim=v_dim,
                           sink=sink, chunk=chunk, v_share=v_share, keep=keep, bias=bias, **kw)

    # differential attention and the stream of designs that norm a sublayer's output
    def diff_prep(self, q_out, proj, *args, **kw):
        T, el = proj.shape[0], proj.element_size()
        n = T * proj.shape[1] * el + _nbytes(q_out) + T * (q_out.shape[1] // 2) * el
        return self._timed("maps' qk_norm+rope+cache_write", n, 0, self.k.diff_prep, q_out, proj, *args, **kw)

    def diff_combine(self, out, a, *args, **kw):
        return self._timed("maps' difference+head norm", _nbytes(out) + _nbytes(a), 0, self.k.diff_combine, out, a, *args, **kw)

    def norm_scale_add(self, stream, y, *args, **kw):
        extra = _nbytes(kw.get("cast_out"))
        return self._timed("sublayer norm+scale+add", 2 * _nbytes(stream) + _nbytes(y) + extra, 0, self.k.norm_scale_add,
                           stream, y, *args, **kw)

    def cast_rows(self, out, x):
        return self._timed("stream to bf16", _nbytes(out) + _nbytes(x), 0, self.k.cast_rows, out, x)

    def gated_act(self, out, gu, act="silu"):
        return self._timed("gated activation", _nbytes(out) + _nbytes(gu), 0, self.k.gated_act, out, gu, act)

    def head_scalar_gate(self, x, g):
        T, H, V = x.shape
        return self._timed("heads*gate", 2 * T * H * V * x.element_size(), 0, self.k.head_scalar_gate, x, g)

    def embed_scaled(self, out, table, ids, *args, **kw):
        return self._timed("embed", 2 * _nbytes(out), 0, self.k.embed_scaled, out, table, ids, *args, **kw)

    # short convolution, retention, gated heads
    def conv_norm_write(self, q_out, proj, conv_w, state, plan, block_table, pool, nq, nkv, dim, vdim, taps, norm, eps):
        T, el = proj.shape[0], proj.element_size()
        n = T * ((nq + nkv) * dim + nkv * vdim) * el + _nbytes(q_out) + T * 2 * nkv * pool.shape[-1] * el
        return self._timed("conv+qk_norm+cache_write", n, 0, self.k.conv_norm_write, q_out, proj, conv_w, state, plan,
                           block_table, pool, nq, nkv, dim, vdim, taps, norm, eps)

    def head_gate(self, out, o, g, heads, v_dim, norm, eps, act):
        T = out.shape[0]
        n = 2 * _nbytes(out) + T * heads * v_dim * o.element_size()
        return self._timed("heads norm*gate" if norm else "heads*gate", n, 0, self.k.head_gate, out, o, g, heads, v_dim,
                           norm, eps, act)

    def retention(self, o, proj, q_off, k_off, v_off, inv_freq, n_rot, decay, state, plan, heads, dim, v_dim, k_scale,
                  pieces=None, cos_sin=None):
        T, el = proj.shape[0], proj.element_size()
        n = T * heads * (2 * dim + v_dim) * el + _nbytes(o) + 2 * plan.R * heads * dim * v_dim * 4
        kind = "retention decode" if plan.is_decode else "retention prefill"
        # (fp32 multiply-adds on the ordinary cores, not the tensor cores: state update and read-out)
        return self._timed(kind, n, 4.0 * T * heads * dim * v_dim, self.k.retention, o, proj, q_off, k_off, v_off, inv_freq,
                           n_rot, decay, state, plan, heads, dim, v_dim, k_scale, pieces, cos_sin)

    # mixers side by side, recurrent mixers, the general q/k/v preparation
    def attn_prep(self, q_out, proj, conv_w, state, plan, block_table, pool, nq, nkv, dim, vdim, *args, **kw):
        T, el = proj.shape[0], proj.element_size()
        n = T * ((nq + nkv) * dim + nkv * vdim) * el + _nbytes(q_out) + T * 2 * nkv * pool.shape[-1] * el
        return self._timed("conv+qk_norm+rope+cache_write", n, 0, self.k.attn_prep, q_out, proj, conv_w, state, plan,
                           block_table, pool, nq, nkv, dim, vdim, *args, **kw)

    def norm_gate(self, out, o, g, *args, **kw):
        return self._timed("heads norm*gate", 2 * _nbytes(out) + _nbytes(o), 0, self.k.norm_gate, out, o, g, *args, **kw)

    def rglru(self, out, proj, *args, **kw):
        T, W = out.shape
        blocks = args[15] if len(args) > 15 else 1
        # x and y read, u / gate logits written and read (fp32), the gated output written; the gates' multiply-adds
        n = 3 * _nbytes(out) + 6 * T * W * 4
        return self._timed("recurrent gated unit", n, 4.0 * T * W * (W // max(1, int(blocks))), self.k.rglru, out, proj,
                           *args, **kw)

    def lowrank_decay(self, alpha, proj, lo_off, w2, *args, **kw):
        return self._timed("decays from a low rank", _nbytes(alpha) + _nbytes(w2), 2.0 * alpha.shape[0] * w2.numel(),
                           self.k.lowrank_decay, alpha, proj, lo_off, w2, *args, **kw)

    def linear_attention(self, o, proj, q_off, k_off, v_off, alpha, head_decay, state, plan, heads, dim, v_dim, *args, **kw):
        T, el = proj.shape[0], proj.element_size()
        n = (T * heads * (2 * dim + v_dim) * el + _nbytes(o) + (0 if alpha is None else _nbytes(alpha))
             + 2 * plan.R * heads * dim * v_dim * 4)
        kind = "gated linear attention decode" if plan.is_decode else "gated linear attention prefill"
        return self._timed(kind, n, 6.0 * T * heads * dim * v_dim, self.k.linear_attention, o, proj, q_off, k_off, v_off,
                           alpha, head_decay, state, plan, heads, dim, v_dim, *args, **kw)

    def mlstm(self, o, proj, q_off, k_off, v_off, z, i_off, f_off, b_i, b_f, cap, state, plan, heads, dim, v_dim, *args):
        T, el = proj.shape[0], proj.element_size()
        n = T * heads * (2 * dim + v_dim) * el + _nbytes(o) + 2 * plan.R * heads * dim * v_dim * 4
        # (fp32 multiply-adds on the ordinary cores: state update and read-out, as for the other recurrences)
        return self._timed("matrix memory prefill", n, 4.0 * T * heads * dim * v_dim, self.k.mlstm, o, proj, q_off, k_off, v_off, z,
                           i_off, f_off, b_i, b_f, cap, state, plan, heads, dim, v_dim, *args)

    def mlstm_step(self, out, proj, q_off, k_off, v_off, g_off, z, i_off, f_off, b_i, b_f, cap, state, plan, heads, dim, v_dim, *args):
        T, el = proj.shape[0], proj.element_size()
        n = T * heads * 2 * (dim + v_dim) * el + _nbytes(out) + 2 * plan.R * heads * dim * v_dim * 4
        return self._timed("matrix memory decode (norm and gate with it)", n, 4.0 * T * heads * dim * v_dim, self.k.mlstm_step, out,
                           proj, q_off, k_off, v_off, g_off, z, i_off, f_off, b_i, b_f, cap, state, plan, heads, dim, v_dim, *args)

    def norm_add_norm(self, stream, y, w1, eps1, out2, w2, eps2, center=False, conv=None):
        n, name = 3 * _nbytes(stream) + _nbytes(out2), "sublayer norm+add+next norm"
        if conv is not None:
            n, name = n + (2 * conv[1].shape[0] - 1) * _nbytes(out2) + _nbytes(conv[1]), name + "+conv"
        kw = {} if not center and conv is None else {"center": center, "conv": conv}
        return self._timed(name, n, 0, self.k.norm_add_norm, stream, y, w1, eps1, out2, w2, eps2, **kw)

    # a layer norm, the mixer's input convolved, a polynomial of normed powers, a gated recurrence, the tokens' side rows
    def layernorm(self, out, x, w, eps, rows=None):
        R, H = out.shape
        return self._timed("layernorm", R * H * 4 + _nbytes(out) + _nbytes(w), 0, self.k.layernorm, out, x, w, eps, rows)

    def input_conv(self, out, h, w, state, plan):
        n = 2 * _nbytes(h) + _nbytes(w) + 2 * plan.R * (w.shape[0] - 1) * h.shape[1] * h.element_size()
        return self._timed("mixer input convolved", n, 0, self.k.input_conv, out, h, w, state, plan)

    def poly_norm(self, out, z, coef, eps):
        return self._timed("polynomial of normed powers", _nbytes(out) + z.numel() * z.element_size(), 0, self.k.poly_norm,
                           out, z, coef, eps)

    def mingru(self, out, proj, *args, **kw):
        T, W = out.shape
        return self._timed("gated recurrence (mingru)", 4 * T * W * out.element_size(), 0, self.k.mingru, out, proj, *args, **kw)

    def token_gate(self, g, z, *args):
        return self._timed("tokens' side rows gated", 3 * _nbytes(g), 0, self.k.token_gate, g, z, *args)

    def token_gate_few(self, g, x, w, *args):
        return self._timed("side gate product+gelu+rows", _nbytes(w) + _nbytes(x) + 2 * _nbytes(g), 2.0 * x.shape[0] * w.numel(),
                           self.k.token_gate_few, g, x, w, *args)

    def latent_down(self, cq, down, q_weight, eps, dkv=None, *args, **kw):
        n = 2 * _nbytes(cq) + 2 * _nbytes(dkv)
        return self._timed("query latent norm" + ("+latent norm+rope+cache_write" if dkv is not None else ""), n, 0,
                           self.k.latent_down, cq, down, q_weight, eps, dkv, *args, **kw)

    def scaled_sum(self, out, a, alpha, b, beta, accumulate=True):
        return self._timed("two sides summed", 3 * _nbytes(out), 0, self.k.scaled_sum, out, a, alpha, b, beta, accumulate)

    def silu_rows(self, x, cols):
        return self._timed("silu on q, k, v", 2 * x.shape[0] * cols * x.element_size(), 0, self.k.silu_rows, x, cols)

    def gated_limit(self, out, gu, limit, alpha):
        return self._timed("gated activation", _nbytes(out) + _nbytes(gu), 0, self.k.gated_limit, out, gu, limit, alpha)

    def softcap_(self, x, cap):
        return self._timed("logit cap", 2 * _nbytes(x), 0, self.k.softcap_, x, cap)

    # latent attention and routed experts
    def latent_prep(self, q, q_rot, dkv, *args, **kw):
        # (only the rotated parts of q are read)
        n = 2 * _nbytes(q_rot) + 2 * _nbytes(dkv)
        return self._timed("latent norm+rope+cache_write", n, 0, self.k.latent_prep, q, q_rot, dkv, *args, **kw)

    def latent_gather(self, rec, *args):
        return self._timed("latent records gathered", 2 * _nbytes(rec), 0, self.k.latent_gather, rec, *args)

    def latent_unfold(self, spool, stable, kv, rec, *args):
        return self._timed("per-head keys and values written out", 3 * _nbytes(kv), 0, self.k.latent_unfold, spool, stable,
                           kv, rec, *args)

    def head_linear(self, out, x, w):
        T = x.shape[0]
        n = _nbytes(w) + T * x.shape[1] * x.shape[2] * x.element_size() + T * out.shape[1] * out.shape[2] * out.element_size()
        return self._timed(f"per-head linear [{w.shape[1]}x{w.shape[2]}]", n, 2.0 * T * w.numel(), self.k.head_linear, out, x, w)

    def latent_attention(self, out, q, pool, block_table, token_pos, token_slot, heads, kv_rank, rot_dim, scale,
                         window=0, plan=None, len_bucket=None, impl=None, chunk=0, **kw):
        keys_read, pairs = self._reach(plan, window, chunk)
        n = _nbytes(q) + _nbytes(out) + keys_read * (kv_rank + rot_dim) * pool.element_size()
        kind = "latent attention decode" if (plan is not None and plan.is_decode) else "latent attention prefill"
        return self._timed(kind, n, 2.0 * heads * (2 * kv_rank + rot_dim) * pairs, self.k.latent_attention, out, q, pool,
                           block_table, token_pos, token_slot, heads, kv_rank, rot_dim, scale, window, plan,
                           len_bucket=len_bucket, impl=impl, chunk=chunk, **kw)

    def moe_route(self, idx, wgt, x, w_router, top, *args, **kw):
        T, K = x.shape
        return self._timed("router", _nbytes(w_router) + T * K * x.element_size(), 2.0 * T * w_router.numel(),
                           self.k.moe_route, idx, wgt, x, w_router, top, *args, **kw)

    def moe_choose(self, idx, wgt, logits, *args, **kw):
        return self._timed("router choice", _nbytes(logits), 0, self.k.moe_choose, idx, wgt, logits, *args, **kw)

    def _experts_read(self, T, top, w):
        return min(T * top, w.shape[0]) * w.shape[1] * w.shape[2] * w.element_size()

    def moe_up(self, act, x, w_up, idx, wgt, scale_input=True, activation="relu2", **kw):
        T, top = idx.shape
        return self._timed("experts up", self._experts_read(T, top, w_up) + _nbytes(act), 2.0 * T * top * w_up.shape[1] * w_up.shape[2],
                           self.k.moe_up, act, x, w_up, idx, wgt, scale_input, activation, **kw)

    def moe_down(self, stream, act, w_down, idx, identity_input=None, wgt=None):
        T, top = idx.shape
        return self._timed("experts down", self._experts_read(T, top, w_down) + _nbytes(act) + 2 * _nbytes(stream),
                           2.0 * T * top * w_down.shape[1] * w_down.shape[2], self.k.moe_down, stream, act, w_down, idx,
                           identity_input, wgt)

    def moe_grouped(self, stream, x, w_up, w_down, idx, wgt, scale_input=True, impl=None, activation="relu2", identity=False,
                    **kw):
        T, top = idx.shape
        n = self._experts_read(T, top, w_up) + self._experts_read(T, top, w_down) + 2 * _nbytes(stream) + T * top * (
            4 * w_up.shape[1] + 8 * w_down.shape[1] + 2 * x.shape[1])
        # (both matrices of every chosen expert: 2 flops a weight and pair)
        return self._timed("experts (sorted, grouped up+down)", n,
                           2.0 * T * top * (w_up.shape[1] * w_up.shape[2] + w_down.shape[1] * w_down.shape[2]),
                           self.k.moe_grouped, stream, x, w_up, w_down, idx, wgt, scale_input, impl=impl,
                           activation=activation, identity=identity, **kw)

    def relu2_scale(self, out, u, row_scale=None):
        return self._timed("relu2*gate", _nbytes(out) + _nbytes(u), 0, self.k.relu2_scale, out, u, row_scale)

    def argmax(self, out, logits, fresh=False):
        return self._timed("argmax", _nbytes(logits), 0, self.k.argmax, out, logits, fresh=fresh)

    def sample(self, out, logits, *args, **kw):
        return self._timed("sample", _nbytes(logits), 0, self.k.sample, out, logits, *args, **kw)


def weight_names(model) -> Dict[int, str]:
    """Device address of every matrix a part holds -> "Part.attribute" (the same for all layers)."""
    names: Dict[int, str] = {}
    parts = [model.embedding, model.final_norm, model.head]
    for b in model.blocks:
        parts.append(b)
        children = getattr(b, "children", None)
        if children:
            parts += list(children().values())
    parts += [p.shared for p in parts if isinstance(getattr(p, "shared", None), Part)]        # (a part inside another)
    for p in parts:
        for attr, val in vars(p).items():
            if isinstance(val, torch.Tensor) and val.dim() == 2 and val.is_cuda:
                names.setdefault(val.data_ptr(), f"{type(p).__name__}.{attr}")
    return names


def profile_engine(engine, prompts: Sequence[Sequence[int]], decode_steps: int = 8, sampling=None,
                   decode_mode: str = "graph") -> List[dict]:
    """One prefill step with every prompt whole and ``decode_steps`` decode steps of all
    rows, each operation timed by CUDA events; returns ``ProfilingKernels.table()``.  The
    sequences are released again."""
    from .sampling import SamplingParams
    sampling = sampling or SamplingParams()
    real = engine.rt.k
    prof = ProfilingKernels(real, weight_names(engine.model))
    if decode_mode == "graph":
        decode_steps = min(decode_steps, 1)        # one step's calls are noted and replayed per operation
    graphs = engine.decoder.use_graphs
    slots = [engine.new_sequence() for _ in prompts]
    # as many prompts per prefill step as the engine's step takes
    per = max(1, engine.max_step_tokens // max(len(p) for p in prompts))

    def prefill():
        toks = []
        for i in range(0, len(prompts), per):
            prof.run_ahead()
            toks += engine.prefill_sample(slots[i:i + per], prompts[i:i + per], sampling,
                                          list(range(i, i + len(prompts[i:i + per]))))
        return toks

    try:
        # once unprofiled, so that no first-call set-up (scratch buffers, attributes) is timed
        toks = prefill()
        for s in slots:
            engine.release(s)
        slots = [engine.new_sequence() for _ in prompts]
        engine.rt.k = prof
        engine.decoder.use_graphs = False
        prof.phase = "prefill"
        toks = prefill()
        prof.phase = "decode"
        if decode_steps:
            toks = engine.decode_sample(slots, toks, sampling, list(range(len(prompts))))     # first-call set-up, untimed
            prof.records = OrderedDict((k, v) for k, v in prof.records.items() if k[0] != "decode")
            prof.mode = decode_mode
            prof.pdl = len(prompts) <= 16 and hasattr(real, "set_pdl")
        for _ in range(decode_steps):
            if any(engine.length(s) + 1 > engine.max_seq_len for s in slots):
                break
            prof.run_ahead()
            toks = engine.decode_sample(slots, toks, sampling, list(range(len(prompts))))
        rows = prof.table()          # graph mode replays the noted calls: the sequences must still be held
    finally:
        engine.rt.k = real
        engine.decoder.use_graphs = graphs
        for s in slots:
            engine.release(s)
    return rows


def format_table(rows: List[dict]) -> str:
    out = []
    for phase in OrderedDict((r["phase"], None) for r in rows):
        sel = [r for r in rows if r["phase"] == phase]
        total = sum(r["total_ms"] for r in sel) or 1.0
        out.append(f"{phase}: {total:.3f} ms in timed operations")
        out.append(f"  {'operation':<44}{'calls':>6}{'us/call':>10}{'ms':>9}{'share':>7}{'MB/call':>10}{'GB/s':>9}{'TFLOP/s':>9}")
        for r in sorted(sel, key=lambda r: -r["total_ms"]):
            out.append(f"  {r['op']:<44}{r['calls']:>6}{r['us_per_call']:>10.2f}{r['total_ms']:>9.3f}"
                       f"{100 * r['total_ms'] / total:>6.1f}%{r['mb_per_call']:>10.3f}{r['gb_s']:>9.1f}{r['tflop_s']:>9.2f}")
    return "\n".join(out)
