"""Ops of pre-norm layers on several residual streams (csrc/streams.cu): hyper-connections with the layer norm and the input
convolution of a sublayer, PolyNorm; PyTorch restatements for CPU tensors. Conventions as in ops/stack.py; the streams of a
step are x [T, S, d] fp32."""
from __future__ import annotations

import torch

from . import _debug, _lib
from .gemm import gemm, gemm_skinny_acc
from .stack import _F, _I, _L, _V, Rows, _p, _rms, act, linear


def embed_streams(ids, table, streams: int, scale: float):
    """Every stream starts as table[ids] * scale."""
    _debug.check_range("embed_streams", "ids", ids, 0, table.shape[0])
    T, d = ids.numel(), table.shape[1]
    if not _lib.use_native(table):
        return (table[ids].float() * scale)[:, None].repeat(1, streams, 1)
    x = torch.empty((T, streams, d), dtype=torch.float32, device=table.device)
    f = _lib.fn("dlti_embed_streams", [_V, _V, _V, _L, _I, _I, _L, _F, _I, _V])
    _lib.check(f(_p(ids), _p(table), _p(x), T, streams, d, table.shape[0], float(scale), _lib.dtype_code(table.dtype), _lib.stream_ptr()),
               "embed_streams")
    return x


def hyper_(x, y, mix, w_out, w_in, norm, eps, dtype, conv=None, idx=None, acc=False):
    """Between two sublayers. y (None: nothing): the finished sublayer's output, x_t <- sum_s mix[s, t] x_s + w_out[t] y in place.
    norm (None: nothing is read): the next sublayer's layer_norm(sum_s w_in[s] x_s) * norm (w_in None: plain sum), of the rows idx.
    conv = (weights [taps, >= d], state [slots, taps - 1, d], rows), one token per sequence: h + causal convolution of h."""
    T, S, d = x.shape
    if not _lib.use_native(x):
        if y is not None:
            x.copy_(torch.einsum("st,nsd->ntd", mix, x) + w_out[None, :, None] * y[:, None, :d].float())
        if norm is None:
            return None
        u = (x if idx is None else x[idx])
        u = u.sum(1) if w_in is None else torch.einsum("s,nsd->nd", w_in, u)
        u = u - u.mean(-1, keepdim=True)
        h = (_rms(u, eps) * norm).to(dtype)
        return h if conv is None else canon(h, conv[0], conv[1], conv[2])
    h = act(T if idx is None else idx.numel(), d, dtype, x.device) if norm is not None else None
    cw, cs, rows = conv if conv is not None else (None, None, None)
    f = _lib.fn("dlti_hyper", [_V, _I, _I, _V, _L, _V, _V, _V, _V, _F, _V, _I, _I, _V, _V, _V, _V, _L, _V, _L, _I, _I, _V])
    _lib.check(f(_p(x), S, d, _p(y), 0 if y is None else y.stride(0), _p(mix), _p(w_out), _p(w_in), _p(norm), float(eps), _p(cw),
                 0 if cw is None else cw.stride(0), 0 if cw is None else cw.shape[0], _p(cs), None if rows is None else _p(rows.state),
                 None if rows is None else _p(rows.ctx), _p(h), 0 if h is None else h.stride(0), _p(idx), T if idx is None else idx.numel(),
                 int(acc), _lib.dtype_code(dtype), _lib.stream_ptr()), "hyper")
    return h


def canon(h, w, state, rows: Rows):
    """h + causal convolution of h over the rows of every sequence; w [taps, >= d] tap-major, state [slots, taps - 1, d] = inputs of
    earlier steps, renewed."""
    T, d = h.shape
    taps = w.shape[0]
    if not _lib.use_native(h):
        out = h.clone()
        for s in range(rows.nseq):
            r0, n, start = rows.bounds(s)
            slot = int(rows.state[s])
            old = state[slot] if start > 0 and slot >= 0 else torch.zeros(taps - 1, d, dtype=h.dtype)
            x = torch.cat([old, h[r0:r0 + n]])
            xf = x.float()
            out[r0:r0 + n] = (xf[taps - 1:] + sum(w[k, :d] * xf[k:k + n] for k in range(taps))).to(h.dtype)
            if slot >= 0 and taps > 1:
                state[slot] = x[x.shape[0] - (taps - 1):]
        return out
    out = act(T, d, h.dtype, h.device)
    f = _lib.fn("dlti_canon", [_V, _L, _I, _I, _V, _I, _V, _V, _V, _V, _I, _I, _I, _I, _V, _L, _I, _V])
    for seq0, nseq, longest in ((0, rows.nd, 1), (rows.nd, rows.nseq - rows.nd, rows.max_seqlen)):
        if nseq:
            _lib.check(f(_p(h), h.stride(0), d, taps, _p(w), w.stride(0), _p(state), _p(rows.state), _p(rows.ctx), _p(rows.cu), rows.nd, seq0,
                         nseq, longest, _p(out), out.stride(0), _lib.dtype_code(h.dtype), _lib.stream_ptr()), "canon")
    return out


def poly_norm(z, ff, coef, eps, dtype, acc=False):
    """a N(z) + b N(z^2) + c N(z^3) + e of the first ff columns, N(y) = y / sqrt(mean y^2 + eps); coef = (a, b, c, e)."""
    T = z.shape[0]
    if not _lib.use_native(z):
        y = z[:, :ff].float()
        a, b, c, e = coef
        return (a * _rms(y, eps) + b * _rms(y * y, eps) + c * _rms(y * y * y, eps) + e).to(dtype)
    h = act(T, ff, dtype, z.device)
    f = _lib.fn("dlti_poly_norm", [_V, _L, _V, _V, _L, _L, _I, _F, _I, _I, _V])
    _lib.check(f(_p(z), z.stride(0), _p(coef), _p(h), h.stride(0), T, ff, float(eps), int(acc), _lib.dtype_code(dtype), _lib.stream_ptr()),
               "poly_norm")
    return h


def linear_split(a, w, split: int):
    """linear with its columns from `split` on as an fp32 result of their own: (a · w[:split]^T, fp32 a · w[split:]^T)."""
    if not _lib.use_native(a) or a.dtype == torch.float32:
        y = linear(a, w, out_dtype=torch.float32)
        return y[:, :split].to(a.dtype), y[:, split:]
    T, N = a.shape[0], w.shape[0]
    if T > 256:
        return gemm(a, w[:split]), gemm(a, w[split:], out_dtype=torch.float32)
    acc = gemm_skinny_acc(a, w)
    main, tail = act(T, split, a.dtype, a.device), torch.empty((T, N - split), dtype=torch.float32, device=a.device)
    f = _lib.fn("dlti_split_rows", [_V, _V, _L, _V, _L, _L, _I, _I, _I, _V])
    _lib.check(f(_p(acc), _p(main), main.stride(0), _p(tail), tail.stride(0), T, N, split, _lib.dtype_code(a.dtype), _lib.stream_ptr()), "split_rows")
    return main, tail
