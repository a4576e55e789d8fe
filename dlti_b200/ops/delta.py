"""Gated delta rule (csrc/delta.cu); PyTorch restatement for CPU tensors. Conventions as in ops/stack.py."""
from __future__ import annotations

import torch

from . import _lib
from .stack import _CHUNKED_FROM, _I, _L, _V, Rows, _conv_args, _p, act

UNIT_EPS = 1e-6              # of the unit norms of queries and keys


def delta_scan_ref(q, k, v, gates, A_log, dt_bias, state, rows: Rows, heads, groups, N, P, conv):
    T, dtype = q.shape[0], v.dtype
    unit = lambda x: x / torch.sqrt(x.square().sum(-1, keepdim=True) + UNIT_EPS)
    rep = lambda x: x.repeat_interleave(heads // groups, 1)
    qf, kf = (rep(unit(x.float().reshape(T, groups, N))) for x in (q, k))
    qf = qf * N ** -0.5
    vf = v.float().reshape(T, heads, P)
    g = torch.exp(-torch.exp(A_log) * torch.nn.functional.softplus(gates[:, :heads].float() + dt_bias, threshold=1e9))
    beta = torch.sigmoid(gates[:, heads:2 * heads].float())
    out = torch.zeros(T, heads, P)
    src, col, cst = conv
    for s in range(rows.nseq):
        r0, n, start = rows.bounds(s)
        slot = int(rows.state[s])
        S = state[slot].clone() if start > 0 and slot >= 0 else torch.zeros(heads, N, P)
        for t in range(r0, r0 + n):
            S = g[t][:, None, None] * S
            u = beta[t][:, None] * (vf[t] - (kf[t][:, :, None] * S).sum(1))
            S = S + kf[t][:, :, None] * u[:, None, :]
            out[t] = (qf[t][:, :, None] * S).sum(1)
        if slot >= 0:
            state[slot] = S
            if cst is not None:
                h = cst[slot] if start > 0 else torch.zeros_like(cst[slot])
                x = torch.cat([h, src[r0:r0 + n, col:col + cst.shape[2]].to(h.dtype)])
                cst[slot] = x[x.shape[0] - cst.shape[1]:].clone()
    return out.reshape(T, -1).to(dtype)


def delta_scan(q, k, v, gates, A_log, dt_bias, state, rows: Rows, heads, groups, N, P, conv_src=None, conv_col=0, conv_state=None):
    """Gated delta rule over the rows of every sequence: q, k [T, groups * N], v [T, heads * P] views after their convolutions;
    gates [T, >= 2 heads] raw fp32 numbers of the decay, then of the step; state [slots, heads, N, P] fp32 updated in place;
    conv_state renewed from the rows of conv_src as in linear_scan."""
    conv = (conv_src, conv_col, conv_state)
    if not _lib.use_native(q):
        return delta_scan_ref(q, k, v, gates, A_log, dt_bias, state, rows, heads, groups, N, P, conv)
    out = act(q.shape[0], heads * P, v.dtype, q.device)
    ws = None

    def run(seq0, nseq, chunked):
        f = _lib.fn("dlti_delta_scan", [_V, _L, _V, _L, _V, _L, _V, _L, _V, _V, _V, _V, _V, _V, _I, _I, _I, _I, _I, _I, _I, _V, _L, _V, _L, _I,
                                        _I, _I, _V, _V, _I, _I, _V])
        _lib.check(f(_p(q), q.stride(0), _p(k), k.stride(0), _p(v), v.stride(0), _p(gates), gates.stride(0), _p(A_log), _p(dt_bias), _p(state),
                     _p(rows.state), _p(rows.ctx), _p(rows.cu), rows.nd, seq0, nseq, heads, groups, N, P, _p(out), out.stride(0), *_conv_args(conv),
                     _p(ws) if chunked else None, rows.max_seqlen if chunked else 0, _lib.dtype_code(v.dtype), _lib.stream_ptr()), "delta_scan")

    nd, nseq = rows.nd, rows.nseq
    if nseq > nd and q.dtype == torch.bfloat16 and N % 8 == 0 and P % 8 == 0 and N <= 256 and rows.max_seqlen >= _CHUNKED_FROM:
        if nd:
            run(0, nd, False)
        size = _lib.fn("dlti_delta_workspace", [_L, _I, _I], restype=_L)(q.shape[0] - nd, nseq - nd, heads)
        ws = torch.empty(size, dtype=torch.uint8, device=q.device)
        run(nd, nseq - nd, True)
    else:
        run(0, nseq, False)
    return out
