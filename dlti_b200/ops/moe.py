"""Gated activations and mixtures of experts (csrc/moe.cu); PyTorch restatements for CPU tensors. Conventions as in ops/stack.py.

A step's (token, choice) pairs are numbered token * top + choice. The router writes every expert's pairs as a list; the first
grouped GEMM gathers its rows by these lists and the second scatters by them, so no permuted copy of the inputs is made."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..models.stack import MoeMlp, mlp_sections, round8
from . import _lib
from .gemm import gemm_relu2, gemm_skinny_acc, gemm_swiglu
from .stack import _F, _I, _L, _V, _p, act, linear, relu2

LIMIT_OFF = 0.0              # limit of a plain SwiGLU: silu(g) * u without clipping


@dataclass
class ExpertSum:
    """A feed-forward's output that is still to be added up: sum over k of weights[t, k] * rows[t * top + k], plus shared (None:
    nothing) times share[t] (None: one). counts: the router's pair counters, which the consumer leaves zero."""
    rows: torch.Tensor
    weights: torch.Tensor
    shared: torch.Tensor | None
    counts: torch.Tensor | None = None
    share: torch.Tensor | None = None

    def value(self, d):
        T, top = self.weights.shape
        y = (self.rows[:, :d].float().view(T, top, d) * self.weights[:, :, None]).sum(1)
        if self.shared is None:
            return y
        s = self.shared[:, :d].float()
        return y + (s if self.share is None else s * self.share[:, None])


def _gated(g, u, limit):
    if limit == LIMIT_OFF:
        return torch.nn.functional.silu(g) * u
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def gated_act(p, og: int, ou: int, ff: int, limit: float, dtype, acc=False):
    """Activation of the projection columns [og, og + ff) (gate) and [ou, ou + ff) (up): silu(g) u, or with a limit
    g sigmoid(1.702 g) (u + 1) of the clipped values."""
    if not _lib.use_native(p):
        return _gated(p[:, og:og + ff].float(), p[:, ou:ou + ff].float(), limit).to(dtype)
    h = act(p.shape[0], ff, dtype, p.device)
    _route(p, None, 0, None, None, act_of=(og, ou, ff, limit, h), acc=acc)
    return h


def swiglu(h, w, ff: int, dtype, acc=False):
    """silu(gate) * up of the merged projection w = [gate rows, up rows], each rounded up to 8."""
    if h.is_cuda and not acc and dtype == torch.bfloat16 and ff % 128 == 0:
        return gemm_swiglu(h, w)                       # activation in the GEMM for large steps
    p = gemm_skinny_acc(h, w) if acc else linear(h, w)
    return gated_act(p, 0, round8(ff), ff, LIMIT_OFF, dtype, acc=acc)


_counters: dict = {}


def _counts(device, n: int) -> torch.Tensor:
    """Zero-on-entry pair counters: the op that adds the experts' outputs up leaves them zero again."""
    key = (str(device), n)
    if key not in _counters:
        _counters[key] = torch.zeros(n, dtype=torch.int32, device=device)
    return _counters[key]


_ACT = {"swiglu": 1, "relu2": 2}       # activations of the grouped GEMM (0: none)


def _route(p, logits, col: int, correction, e: MoeMlp | None, act_of=None, acc=False, share=None):
    """One launch: routing of the fp32 logits [T, >= col + experts] at column col, the sigmoid of one more column (share = (column,
    destination [T])), and / or the activation act_of = (gate column (-1: square of relu of the other), up column, ff, limit,
    destination) of the projection rows p. acc: both read the decode GEMM's accumulator and leave it zero."""
    T = (p if p is not None else logits).shape[0]
    dev = (p if p is not None else logits).device
    wgt = lists = counts = None
    if e is not None:
        wgt = torch.empty((T, e.top), dtype=torch.float32, device=dev)
        lists = torch.empty((e.experts, T), dtype=torch.int32, device=dev)
        counts = _counts(dev, e.experts)
    sg, sigma = share or (-1, None)
    og, ou, ff, limit, h = act_of or (0, 0, 0, 0.0, None)
    f = _lib.fn("dlti_moe_route", [_V, _L, _I, _V, _I, _I, _I, _I, _F, _I, _V, _V, _V, _I, _V, _V, _L, _I, _I, _I, _F, _V, _L, _L, _I, _I, _V])
    _lib.check(f(_p(logits), 0 if logits is None else logits.stride(0), col, _p(correction), e.experts if e else 0, e.top if e else 0,
                 e.groups if e else 1, e.keep if e else 1, e.scale if e else 1.0, int(e is not None and e.score == "softmax"), _p(wgt), _p(lists),
                 _p(counts), sg, _p(sigma), _p(p) if h is not None else None, p.stride(0) if p is not None else 0, og, ou, ff, float(limit), _p(h),
                 0 if h is None else h.stride(0), T, int(acc), _lib.dtype_code(h.dtype) if h is not None else _lib.DT_BF16, _lib.stream_ptr()),
               "moe_route")
    return wgt, lists, counts


def route_ref(z, correction, e: MoeMlp):
    """Router logits [T, experts] -> (chosen experts [T, top], weights [T, top])."""
    if e.score == "softmax":
        c, idx = (z + correction).topk(e.top, -1)
        return idx, torch.softmax(c, -1) * e.scale
    s = torch.sigmoid(z)
    c = s + correction
    T, n = z.shape[0], e.experts // e.groups
    if e.keep < e.groups:
        best = c.view(T, e.groups, n).topk(min(2, n), -1).values.sum(-1).topk(e.keep, -1).indices
        open_ = torch.zeros(T, e.groups, dtype=torch.bool).scatter_(1, best, True)
        c = c.masked_fill(~open_.repeat_interleave(n, 1), float("-inf"))
    idx = c.topk(e.top, -1).indices
    w = s.gather(1, idx)
    return idx, w / (w.sum(-1, keepdim=True) + 1e-20) * e.scale


def grouped_gemm(x, w, lists, counts, out, *, rows: int, pairs_per_row: int, up: bool = False, limit: float = 0.0, act: str = "swiglu"):
    """Products of the pairs of every expert's list with its weights w [E, >= rows, K]. up: rows x[pair // pairs_per_row]; the
    activations go to out one list after the other ("swiglu", clipped: rows 2 r and 2 r + 1 of w are gate and up of output r; "relu2":
    row r is). Otherwise: rows of x in that order; results go to out[pair]."""
    E, K, T = w.shape[0], w.shape[2], lists.shape[1]
    f = _lib.fn("dlti_moe_gemm", [_V, _L, _L, _I, _V, _L, _I, _I, _V, _V, _I, _I, _I, _I, _F, _V, _L, _I, _I, _V])
    _lib.check(f(_p(x), x.stride(0), x.shape[0], pairs_per_row, _p(w), w.stride(1), w.stride(0) // w.stride(1), E, _p(lists), _p(counts), T,
                 rows, _ACT[act] if up else 0, K, float(limit), _p(out), out.stride(0), out.shape[0], _lib.dtype_code(x.dtype), _lib.stream_ptr()), "moe_gemm")
    return out


def moe(h, e: MoeMlp, lw, dtype, mm, acc=False) -> ExpertSum:
    """Mixture of experts of the rows h; mm: the GEMM for the shared expert's output (its accumulator with acc)."""
    T, d = h.shape
    sec = mlp_sections(e)
    og, ou = (sec["gate"] if e.gated else -1, sec["up"]) if e.shared_ff else (0, 0)
    sg = sec["sg"] if e.shared_gate else -1
    if not _lib.use_native(h):
        p = linear(h, lw["w_up"], out_dtype=torch.float32)
        idx, wgt = route_ref(p[:, sec["router"]:sec["router"] + e.experts], lw["correction"], e)
        rows = torch.zeros(T * e.top, d)
        for j in range(e.experts):
            pair = (idx.flatten() == j).nonzero()[:, 0]
            if len(pair):
                gu = h[pair // e.top].float() @ lw["e_up"][j].float().t()
                a = (_gated(gu[:, 0:2 * e.ff:2], gu[:, 1:2 * e.ff:2], e.limit) if e.gated else torch.relu(gu[:, :e.ff]).square()).to(dtype)
                rows[pair] = a.float() @ lw["e_down"][j, :d].float().t()
        shared = None
        if e.shared_ff:
            shared = mm(gated_act(p, og, ou, e.shared_ff, e.shared_limit, dtype) if e.gated else relu2(p[:, ou:], e.shared_ff, dtype), lw["w_down"])
        return ExpertSum(rows.to(dtype), wgt, shared, share=torch.sigmoid(p[:, sg]) if sg >= 0 else None)
    hs, act_of, share = None, None, None
    if e.shared_gate:
        share = torch.empty(T, dtype=torch.float32, device=h.device)
    if acc:
        p = gemm_skinny_acc(h, lw["w_up"])
        if e.shared_ff:
            hs = act(T, e.shared_ff, dtype, h.device)
            act_of = (og, ou, e.shared_ff, e.shared_limit, hs)
        wgt, lists, counts = _route(p, p, sec["router"], lw["correction"], e, act_of, acc=True, share=(sg, share))
    else:
        r0 = sec["router"]
        z = linear(h, lw["w_up"][r0:], out_dtype=torch.float32)
        p = None
        if e.shared_ff and not e.gated:
            hs = gemm_relu2(h, lw["w_up"][:r0], e.shared_ff)               # activation in the GEMM for large steps
        if e.shared_ff and hs is None:
            p, hs = linear(h, lw["w_up"][:r0]), act(T, e.shared_ff, dtype, h.device)
            act_of = (og, ou, e.shared_ff, e.shared_limit, hs)
        wgt, lists, counts = _route(p, z, 0, lw["correction"], e, act_of, share=(sg - r0 if sg >= 0 else -1, share))
    a = act(T * e.top, e.ff, dtype, h.device)
    grouped_gemm(h, lw["e_up"], lists, counts, a, rows=e.ff, pairs_per_row=e.top, up=True, limit=e.limit, act=e.act)
    rows = act(T * e.top, d, dtype, h.device)
    grouped_gemm(a, lw["e_down"], lists, counts, rows, rows=d, pairs_per_row=1)
    return ExpertSum(rows, wgt, mm(hs, lw["w_down"]) if e.shared_ff else None, counts, share)
