"""Ops of models with dynamic tanh norms before and after every sublayer (csrc/dyt.cu); PyTorch restatements for CPU tensors.
Conventions as in ops/stack.py. A norm is a tuple (alpha [1], w [d], b [d]): tanh(alpha x) * w + b."""
from __future__ import annotations

import torch

from . import _debug, _lib
from .moe import ExpertSum
from .stack import _F, _I, _L, _V, _p, act


def _norm(x, n):
    return torch.tanh(n[0] * x) * n[1] + n[2]


def _three(n):
    return (None, None, None) if n is None else tuple(_p(t) for t in n)


def embed_tanh(ids, table, scale: float, norm, dtype):
    """Residual rows x = table[ids] * scale [T, d] fp32 and norm(x) in the compute dtype."""
    _debug.check_range("embed_tanh", "ids", ids, 0, table.shape[0])
    T, d = ids.numel(), table.shape[1]
    if not _lib.use_native(table):
        x = table[ids].float() * scale
        return x, _norm(x, norm).to(dtype)
    x = torch.empty((T, d), dtype=torch.float32, device=table.device)
    h = act(T, d, dtype, table.device)
    f = _lib.fn("dlti_tanh_embed", [_V, _V, _L, _F, _V, _V, _V, _V, _V, _L, _L, _I, _I, _V])
    _lib.check(f(_p(ids), _p(table), table.shape[0], float(scale), *_three(norm), _p(x), _p(h), h.stride(0), T, d, _lib.dtype_code(dtype),
                 _lib.stream_ptr()), "tanh_embed")
    return x, h


def tanh_between_(x, y, post, pre, dtype, acc=False):
    """Between two sublayers: x += post(y) in place on the fp32 residual [T, d]; returns pre(x) in the compute dtype (None without
    pre). y: the finished sublayer's output, at least d columns (acc: the decode GEMM's accumulator), or an ExpertSum."""
    T, d = x.shape
    e = y if isinstance(y, ExpertSum) else None
    if not _lib.use_native(x):
        x += _norm((e.value(d) if e is not None else y[:, :d]).float(), post)
        return None if pre is None else _norm(x, pre).to(dtype)
    h = act(T, d, dtype, x.device) if pre is not None else None
    if e is not None:
        y = e.shared
    f = _lib.fn("dlti_tanh_between", [_V, _V, _L, _V, _L, _V, _I, _V, _I, _V, _V, _V, _V, _V, _V, _V, _L, _L, _I, _I, _I, _V])
    _lib.check(f(_p(x), _p(y), 0 if y is None else y.stride(0), _p(e.rows) if e else None, e.rows.stride(0) if e else 0,
                 _p(e.weights) if e else None, e.weights.shape[1] if e else 0, _p(e.counts) if e else None,
                 e.counts.numel() if e and e.counts is not None else 0,
                 *_three(post), *_three(pre), _p(h), 0 if h is None else h.stride(0), T, d, int(acc and y is not None),
                 _lib.dtype_code(dtype), _lib.stream_ptr()), "tanh_between")
    return h


def tanh_rows(x, idx, norm, dtype):
    """norm(x[idx]) in the compute dtype; idx None = all rows."""
    if not _lib.use_native(x):
        return _norm(x if idx is None else x[idx], norm).to(dtype)
    rows, d = x.shape[0] if idx is None else idx.numel(), x.shape[1]
    h = act(rows, d, dtype, x.device)
    f = _lib.fn("dlti_tanh_rows", [_V, _V, _V, _V, _V, _V, _L, _L, _I, _I, _V])
    _lib.check(f(_p(x), _p(idx), *_three(norm), _p(h), h.stride(0), rows, d, _lib.dtype_code(dtype), _lib.stream_ptr()), "tanh_rows")
    return h
