"""Ops of models with RMS norms on the sublayer inputs (csrc/prenorm.cu); PyTorch restatements for CPU tensors. Conventions as in
ops/stack.py."""
from __future__ import annotations

import torch

from . import _debug, _lib
from .moe import ExpertSum
from .stack import _F, _I, _L, _V, _p, _rms, act


def between_(x, y, pre, eps, dtype, *, mult=1.0, post=None, embed=None, fresh=False, copy=False, acc=False):
    """Between two sublayers, on the fp32 residual [T, d] in place: x (zero if fresh) += mult * y, += the embedding rows embed = (ids,
    table, scale). y: the finished sublayer's output, at least d columns (acc: the decode GEMM's accumulator), an ExpertSum or None;
    with post its RMS norm times post is added instead. Returns the RMS norm of x times pre in the compute dtype; without pre x
    itself (copy) or None."""
    T, d = x.shape
    e = y if isinstance(y, ExpertSum) else None
    if embed is not None:
        _debug.check_range("prenorm_between", "ids", embed[0], 0, embed[1].shape[0])
    if not _lib.use_native(x):
        if fresh:
            x.zero_()
        if y is not None:
            v = (e.value(d) if e is not None else y[:, :d]).float()
            x += mult * (v if post is None else _rms(v, eps) * post)
        if embed is not None:
            x += embed[1][embed[0]].float() * embed[2]
        return (_rms(x, eps) * pre).to(dtype) if pre is not None else x.to(dtype, copy=True) if copy else None
    h = act(T, d, dtype, x.device) if pre is not None or copy else None
    if e is not None:
        y = e.shared
    ids, table, scale = embed or (None, None, 0.0)
    f = _lib.fn("dlti_prenorm_between", [_V, _V, _L, _V, _L, _V, _I, _V, _V, _I, _F, _V, _V, _V, _L, _F, _I, _V, _V, _L, _L, _I, _F, _I, _I, _V])
    _lib.check(f(_p(x), _p(y), 0 if y is None else y.stride(0), _p(e.rows) if e else None, e.rows.stride(0) if e else 0,
                 _p(e.weights) if e else None, e.weights.shape[1] if e else 0, _p(e.share) if e else None, _p(e.counts) if e else None,
                 e.counts.numel() if e and e.counts is not None else 0, float(mult), _p(post), _p(ids), _p(table),
                 0 if table is None else table.shape[0], float(scale), int(fresh), _p(pre), _p(h), 0 if h is None else h.stride(0), T, d, float(eps),
                 int(acc and y is not None), _lib.dtype_code(dtype), _lib.stream_ptr()), "prenorm_between")
    return h


def token_gate(u, ids, table, col: int, n: int, dtype, acc=False):
    """gelu(u) (tanh form) times the columns [col, col + n) of the tokens' rows of `table`."""
    T = u.shape[0]
    _debug.check_range("token_gate", "ids", ids, 0, table.shape[0])
    if not _lib.use_native(u):
        return (torch.nn.functional.gelu(u[:, :n].float(), approximate="tanh") * table[ids][:, col:col + n].float()).to(dtype)
    h = act(T, n, dtype, u.device)
    f = _lib.fn("dlti_token_gate", [_V, _L, _V, _V, _L, _L, _I, _I, _V, _L, _L, _I, _I, _V])
    _lib.check(f(_p(u), u.stride(0), _p(ids), _p(table), table.stride(0), table.shape[0], col, n, _p(h), h.stride(0), T, int(acc),
                 _lib.dtype_code(dtype), _lib.stream_ptr()), "token_gate")
    return h
