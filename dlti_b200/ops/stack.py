"""Ops of the layer-stack models (models/stack.py; more of them in streams.py and latent.py): kernels in csrc/stack.cu,
recurrent.cu, attention_paged.cu and gemm_f32.cu; PyTorch restatements for CPU tensors, as in the other op modules.

Activations are [rows, n] views whose row pitch is a multiple of 8 elements (`act`). The residual stream is fp32.
Ops with `acc=True` consume the fp32 accumulator of gemm_skinny_acc and leave it zero."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import torch

from ..models.stack import round8
from . import _debug, _lib
from .gemm import gemm, gemm_skinny, gemm_skinny_acc

_V, _I, _L, _F = C.c_void_p, C.c_int, C.c_longlong, C.c_float
_p = _lib.ptr


def act(rows: int, n: int, dtype, device) -> torch.Tensor:
    return torch.empty((rows, round8(n)), dtype=dtype, device=device)[:, :n]


def linear(a: torch.Tensor, w: torch.Tensor, out_dtype=None) -> torch.Tensor:
    """a [T, K] · w [N, K]^T -> [T, N]; N is a multiple of 8 (stack weights are padded)."""
    if not _lib.use_native(a):
        return (a.float() @ w.float().t()).to(out_dtype or a.dtype)
    if a.dtype == torch.float32:
        M, K = a.shape
        N = w.shape[0]
        out = torch.empty((M, N), dtype=torch.float32, device=a.device)
        f = _lib.fn("dlti_gemm_f32", [_V, _V, _V, _I, _I, _I, _L, _L, _L, _V])
        _lib.check(f(_p(a), _p(w), _p(out), M, N, K, a.stride(0), w.stride(0), out.stride(0), _lib.stream_ptr()), "gemm_f32")
        return out
    if a.shape[0] <= 256 and out_dtype in (None, a.dtype):
        return gemm_skinny(a, w)
    return gemm(a, w, out_dtype=out_dtype)


def linear_f32(a: torch.Tensor, w: torch.Tensor, scale: float = 1.0, cap: float = 0.0) -> torch.Tensor:
    """linear times scale with an fp32 result (logits); cap > 0: cap * tanh(that / cap)."""
    if not _lib.use_native(a):
        y = linear(a, w, out_dtype=torch.float32) * scale
        return cap * torch.tanh(y / cap) if cap else y
    if a.dtype == torch.float32:
        acc, alpha = linear(a, w), scale
    elif a.shape[0] > 256:
        acc, alpha = gemm(a, w, out_dtype=torch.float32, alpha=scale), 1.0
    else:
        acc = gemm_skinny_acc(a, w)
        out = torch.empty_like(acc)
        _take_rows(acc, out, scale, cap, True)
        return out
    if alpha != 1.0 or cap:
        _take_rows(acc, acc, alpha, cap, False)
    return acc


def _take_rows(src, out, scale, cap, clear):
    f = _lib.fn("dlti_take_rows", [_V, _V, _F, _F, _I, _L, _I, _V])
    _lib.check(f(_p(src), _p(out), float(scale), float(cap), int(clear), src.shape[0], src.shape[1], _lib.stream_ptr()), "take_rows")


# ---- rows --------------------------------------------------------------------------------------------------
def embed_rows(ids, table):
    """Token rows as the fp32 residual stream [T, d] and as the first GEMM's input (the same tensor in fp32)."""
    _debug.check_range("embed_rows", "ids", ids, 0, table.shape[0])
    T, d = ids.numel(), table.shape[1]
    if not _lib.use_native(table):
        x = table[ids].float()
        return x, (x if table.dtype == torch.float32 else table[ids])
    x = torch.empty((T, d), dtype=torch.float32, device=table.device)
    xa = None if table.dtype == torch.float32 else act(T, d, table.dtype, table.device)
    f = _lib.fn("dlti_embed_rows", [_V, _V, _V, _V, _L, _L, _I, _L, _I, _V])
    _lib.check(f(_p(ids), _p(table), _p(x), _p(xa), 0 if xa is None else xa.stride(0), T, d, table.shape[0],
                 _lib.dtype_code(table.dtype), _lib.stream_ptr()), "embed_rows")
    return x, (x if xa is None else xa)


def _rms(x, eps):
    return x / torch.sqrt(x.square().mean(-1, keepdim=True) + eps)


def post_norm_add_(y, x, w, eps, one_plus, dtype, acc=False, want=True):
    """x += norm(y) * w (1 + w with one_plus), in place on the fp32 residual [T, d]; y has at least d columns. Returns
    the new residual as the next GEMM's input (x itself in fp32; None unless want)."""
    T, d = x.shape
    if not _lib.use_native(x):
        x += _rms(y[:, :d].float(), eps) * (w + 1 if one_plus else w)
        return x if dtype == torch.float32 else x.to(dtype)
    xa = None if dtype == torch.float32 or not want else act(T, d, dtype, x.device)
    f = _lib.fn("dlti_post_norm_add", [_V, _L, _V, _V, _V, _L, _L, _I, _F, _I, _I, _I, _V])
    _lib.check(f(_p(y), y.stride(0), _p(x), _p(w), _p(xa), 0 if xa is None else xa.stride(0), T, d, float(eps), int(one_plus),
                 int(acc), _lib.dtype_code(dtype), _lib.stream_ptr()), "post_norm_add")
    return x if dtype == torch.float32 else xa


def rms_rows(x, idx, w, eps, one_plus, dtype):
    """norm(x[idx]) * w in the compute dtype; idx None = all rows."""
    if not _lib.use_native(x):
        xs = x if idx is None else x[idx]
        return (_rms(xs, eps) * (w + 1 if one_plus else w)).to(dtype)
    rows = x.shape[0] if idx is None else idx.numel()
    out = act(rows, x.shape[1], dtype, x.device)
    f = _lib.fn("dlti_rms_rows", [_V, _V, _V, _V, _L, _L, _I, _F, _I, _I, _V])
    _lib.check(f(_p(x), _p(idx), _p(w), _p(out), out.stride(0), rows, x.shape[1], float(eps), int(one_plus),
                 _lib.dtype_code(dtype), _lib.stream_ptr()), "rms_rows")
    return out


def relu2(u, ff, dtype, acc=False):
    """Square of relu of the first ff columns."""
    if not _lib.use_native(u):
        return torch.relu(u[:, :ff].float()).square().to(dtype)
    T = u.shape[0]
    h = act(T, ff, dtype, u.device)
    f = _lib.fn("dlti_relu2", [_V, _L, _V, _L, _L, _I, _I, _I, _V])
    _lib.check(f(_p(u), u.stride(0), _p(h), h.stride(0), T, ff, int(acc), _lib.dtype_code(dtype), _lib.stream_ptr()), "relu2")
    return h


def gated_norm(y, gate, w, eps, groups, gate_first, acc=False, silu=False):
    """gate_first: norm(y * silu(gate)) * w; else norm(y) * w * sigmoid(gate), with silu: norm(y) * w * silu(gate). The norm runs
    over `groups` equal parts of the row. gate: [T, >= n] view (a section of a projection; of its accumulator with acc)."""
    T, n = y.shape
    if not _lib.use_native(y):
        g = gate[:, :n].float()
        v = y.float() * torch.nn.functional.silu(g) if gate_first else y.float()
        v = _rms(v.reshape(T, groups, -1), eps).reshape(T, n) * w
        return (v if gate_first else v * (torch.nn.functional.silu(g) if silu else torch.sigmoid(g))).to(y.dtype)
    out = act(T, n, y.dtype, y.device)
    f = _lib.fn("dlti_gated_norm", [_V, _L, _V, _L, _V, _V, _L, _L, _I, _I, _F, _I, _I, _I, _V])
    _lib.check(f(_p(y), y.stride(0), _p(gate), gate.stride(0), _p(w), _p(out), out.stride(0), T, n, groups, float(eps),
                 1 if gate_first else 2 if silu else 0, int(acc), _lib.dtype_code(y.dtype), _lib.stream_ptr()), "gated_norm")
    return out


# ---- attention ---------------------------------------------------------------------------------------------
_tables: dict = {}


def rope_tables(max_pos: int, dims: int, base: float, device):
    """fp32 cos / sin [max_pos, dims/2] of position * base^(-2i/dims), the angle taken in double precision."""
    key = (max_pos, dims, base, str(device))
    t = _tables.get(key)
    if t is None:
        f = base ** (-torch.arange(0, dims, 2, dtype=torch.float64) / dims)
        a = torch.arange(max_pos, dtype=torch.float64)[:, None] * f[None, :]
        t = _tables[key] = (a.cos().float().to(device), a.sin().float().to(device))
    return t


@dataclass
class Rows:
    """Where a step's token rows belong: nd decode rows (sequence s = row s), then prompt rows; sequence nd + i owns rows
    nd + cu[i] ... nd + cu[i + 1]. ctx[s] = tokens of sequence s after the step, pos[t] / seq[t] = position and sequence
    of row t, slots[t] = its cache slot (-1: none), state[s] = recurrent-state slot (-1: none)."""
    pos: torch.Tensor
    seq: torch.Tensor
    slots: torch.Tensor
    ctx: torch.Tensor
    cu: torch.Tensor | None
    tables: torch.Tensor
    state: torch.Tensor
    nd: int
    max_seqlen: int
    max_ctx: int

    @property
    def nseq(self) -> int:
        return self.nd + (0 if self.cu is None else self.cu.numel() - 1)

    def bounds(self, s: int) -> tuple[int, int, int]:
        """(first row, rows, first position) of sequence s (host side; CPU restatements only)."""
        if s < self.nd:
            r0, n = s, 1
        else:
            r0 = self.nd + int(self.cu[s - self.nd])
            n = int(self.cu[s - self.nd + 1]) - int(self.cu[s - self.nd])
        return r0, n, int(self.ctx[s]) - n


@dataclass
class Pieces:
    """The prompt rows of a step as independent causal sequences for one kind of attention: a prompt is cut at every
    chunk edge, and a portion that continues a chunk (or a window) has the cached keys and values that its rows can see laid
    out in front of them. cu [n + 1]: boundaries in that extended layout; longest: its longest piece. With cached rows (prefix > 0): q0 [n]
    = cached rows of a piece, out0 [n] = prompt row of its first own row, dst [prompt rows] = extended row of each prompt
    row, prow / pslot [prefix] = extended row and cache slot of each cached token."""
    cu: torch.Tensor
    longest: int
    rows: int
    prefix: int = 0
    q0: torch.Tensor | None = None
    out0: torch.Tensor | None = None
    dst: torch.Tensor | None = None
    prow: torch.Tensor | None = None
    pslot: torch.Tensor | None = None


PACKED_HD = 128              # head columns of the packed layout


def qk_norm_rope_cache(proj, sec, m, q_norm, k_norm, eps, rows: Rows, tabs, kc, vc, dtype, packed: Pieces | None = None, acc=False):
    """Merged projection rows -> rotated queries (each head normalised first when norms are given), keys and values in
    the paged cache at rows.slots, and the sigmoid of the head gates [T, H] (None without gates).
    packed: return [q heads | k heads | v heads] rows instead, heads padded to 128 columns, the prompt rows in the extended
    layout of `packed`; keys and values of a layer without own ones, and of cached rows, are copied from the cache."""
    T, H, G = proj.shape[0], m.heads, m.kv_heads
    own = "k" in sec
    rot = m.rope.dims if m.rope is not None else 0
    _debug.check_range("qk_norm_rope_cache", "slots", rows.slots, 0, kc.shape[0] * kc.shape[1], allow=-1)
    if not _lib.use_native(proj):
        ok = rows.slots >= 0
        kf, vf = kc.view(-1, G, kc.shape[3]), vc.view(-1, G, vc.shape[3])

        def prep(name, heads, nw):
            x = proj[:, sec[name]:sec[name] + heads * m.dim].float().reshape(T, heads, m.dim)
            if nw is not None:
                x = _rms(x, eps) * nw
            if rot:
                c, s = (t[rows.pos.long()][:, None, :] for t in tabs)
                h = rot // 2
                a, b = (x[..., 0:rot:2], x[..., 1:rot:2]) if m.rope.interleaved else (x[..., :h], x[..., h:rot])
                u, v = a * c - b * s, b * c + a * s
                r = torch.stack([u, v], -1).flatten(-2) if m.rope.interleaved else torch.cat([u, v], -1)
                x = torch.cat([r, x[..., rot:]], -1)
            return x.to(dtype)

        q = prep("q", H, q_norm)
        if own:
            k = prep("k", G, k_norm)
            v = proj[:, sec["v"]:sec["v"] + G * m.vdim].reshape(T, G, m.vdim).to(dtype)
            kf[rows.slots[ok], :, :m.dim] = k[ok]
            vf[rows.slots[ok], :, :m.vdim] = v[ok]
        gate = torch.sigmoid(proj[:, sec["g"]:sec["g"] + H].float()) if "g" in sec else None
        return q.reshape(T, -1), gate
    dev = proj.device
    gate = torch.empty((T, H), dtype=torch.float32, device=dev) if "g" in sec else None
    kp = vp = dst = None
    if packed is not None:
        hd = PACKED_HD
        n = rows.nd + packed.rows
        q = (torch.empty if m.dim == m.vdim == hd else torch.zeros)((n, (H + 2 * G) * hd), dtype=dtype, device=dev)
        kp, vp, dst = q[:, H * hd:], q[:, (H + G) * hd:], packed.dst
    else:
        hd = round8(m.dim)
        q = torch.empty((T, H * hd), dtype=dtype, device=dev)
    f = _lib.fn("dlti_qk_norm_rope_cache", [_V, _L, _I, _I, _I, _I, _V, _V, _F, _V, _V, _V, _I, _I, _V, _V, _V, _I, _I, _V, _L, _I, _V,
                                            _V, _V, _I, _V, _L, _I, _I, _I, _I, _I, _I, _V])
    _lib.check(f(_p(proj), proj.stride(0), sec["q"], sec["k"] if own else -1, sec["v"] if own else -1, sec["g"] if "g" in sec else -1,
                 _p(q_norm), _p(k_norm), float(eps), _p(rows.pos), _p(tabs[0]) if rot else None, _p(tabs[1]) if rot else None, rot,
                 int(m.rope.interleaved) if rot else 1, _p(rows.slots), _p(kc), _p(vc), kc.shape[3], vc.shape[3], _p(q), q.stride(0), hd,
                 _p(kp), _p(vp), _p(dst), rows.nd, _p(gate), T, H, G, m.dim, m.vdim, int(acc), _lib.dtype_code(dtype),
                 _lib.stream_ptr()), "qk_norm_rope_cache")
    if packed is not None and packed.prefix:
        prefix_rows(q[rows.nd:], m, packed, kc, vc)
    return q, gate


_factors: dict = {}


def temp_table(max_pos: int, temp, device):
    """fp32 factors [max_pos] of the queries by position (models.stack.QueryTemp), from double precision."""
    key = (max_pos, temp, str(device))
    if key not in _factors:
        p = torch.arange(max_pos, dtype=torch.int64)
        _factors[key] = (1 + temp.coef * torch.log(((p + 1) // temp.every + 1).double())).float().to(device)
    return _factors[key]


def conv_qkv(proj, sec, m, lw, factors, eps, rows: Rows, state, kc, vc, dtype, packed: Pieces | None = None, acc=False):
    """Merged projection rows -> convolved (m.conv; state [slots, taps - 1, columns before g] holds the inputs of earlier steps and is
    renewed) queries and keys with per-head norms, queries times factors[position] (None: one), values; keys and values in the paged
    cache at rows.slots. packed: as in qk_norm_rope_cache. acc (decode rows only): the projection is the decode GEMM's accumulator.
    Returns (queries or packed rows, the projected output gates [T, H * vdim] before their sigmoid or None)."""
    T, H, G, taps, dev = proj.shape[0], m.heads, m.kv_heads, m.conv, proj.device
    _debug.check_range("conv_qkv", "slots", rows.slots, 0, kc.shape[0] * kc.shape[1], allow=-1)
    qn, kn, w = lw.get("q_norm"), lw.get("k_norm"), lw.get("conv")
    gate = proj[:, sec["g"]:sec["g"] + H * m.vdim] if m.out_gate else None
    if not _lib.use_native(proj):
        span = sec["v"] + round8(G * m.vdim)
        x = proj[:, :span].float()
        if taps:
            y = torch.zeros(T, span)
            for s in range(rows.nseq):
                r0, n, start = rows.bounds(s)
                slot = int(rows.state[s])
                h = state[slot].float() if state is not None and start > 0 and slot >= 0 else torch.zeros(taps - 1, span)
                u = torch.cat([h, x[r0:r0 + n]])
                y[r0:r0 + n] = sum(w[k, :span] * u[k:k + n] for k in range(taps))
                if slot >= 0 and state is not None:
                    state[slot] = u[n:].to(dtype)
            x = y
        q, k, v = (x[:, sec[c]:sec[c] + n * d].reshape(T, n, d) for c, n, d in (("q", H, m.dim), ("k", G, m.dim), ("v", G, m.vdim)))
        q, k = (t if g is None else _rms(t, eps) * g for t, g in ((q, qn), (k, kn)))
        if factors is not None:
            q = q * factors[rows.pos.long()][:, None, None]
        ok = rows.slots >= 0
        kc.view(-1, G, kc.shape[3])[rows.slots[ok], :, :m.dim] = k.to(dtype)[ok]
        vc.view(-1, G, vc.shape[3])[rows.slots[ok], :, :m.vdim] = v.to(dtype)[ok]
        return q.to(dtype).reshape(T, -1), gate
    if acc and gate is not None:
        gate = act(T, H * m.vdim, dtype, dev)
    kp = vp = dst = None
    if packed is not None:
        hd, n = PACKED_HD, rows.nd + packed.rows
        q = (torch.empty if m.dim == m.vdim == hd else torch.zeros)((n, (H + 2 * G) * hd), dtype=dtype, device=dev)
        kp, vp, dst = q[:, H * hd:], q[:, (H + G) * hd:], packed.dst
    else:
        hd = round8(m.dim)
        q = torch.empty((T, H * hd), dtype=dtype, device=dev)
    f = _lib.fn("dlti_conv_qkv", [_V, _L, _I, _I, _I, _I, _V, _I, _I, _V, _I, _V, _V, _V, _V, _I, _I, _V, _V, _F, _V, _V, _V, _V, _V, _I, _I, _V,
                                  _L, _I, _V, _V, _V, _V, _L, _L, _I, _I, _I, _I, _I, _I, _V])
    _lib.check(f(_p(proj), proj.stride(0), sec["q"], sec["k"], sec["v"], sec["g"] if m.out_gate else -1, _p(w), taps, 0 if w is None else w.stride(0),
                 _p(state), 0 if state is None else state.shape[2], _p(rows.state), _p(rows.seq), _p(rows.ctx), _p(rows.cu), rows.nd, rows.nseq,
                 _p(qn), _p(kn), float(eps), _p(factors), _p(rows.pos), _p(rows.slots), _p(kc), _p(vc), kc.shape[3], vc.shape[3],
                 _p(q), q.stride(0), hd, _p(kp), _p(vp), _p(dst), _p(gate) if acc else None, gate.stride(0) if acc and gate is not None else 0, T,
                 H, G, m.dim, m.vdim, int(acc), _lib.dtype_code(dtype), _lib.stream_ptr()), "conv_qkv")
    if packed is not None and packed.prefix:
        prefix_rows(q[rows.nd:], m, packed, kc, vc)
    return q, gate


def prefix_rows(buf, m, packed: Pieces, kc, vc):
    """Cached keys and values in front of the portions of a step: packed prompt rows buf [rows, (H + 2 G) * 128]."""
    f = _lib.fn("dlti_prefix_rows", [_V, _L, _I, _V, _V, _V, _V, _I, _I, _I, _I, _L, _V])
    _lib.check(f(_p(buf), buf.stride(0), PACKED_HD, _p(packed.prow), _p(packed.pslot), _p(kc), _p(vc), kc.shape[3], vc.shape[3], m.heads,
                 m.kv_heads, packed.prefix, _lib.stream_ptr()), "prefix_rows")


def qkv_rows(proj, sec, m, lw, eps, rows: Rows, first, kc, vc, dtype, packed: Pieces | None = None, acc=False):
    """Merged projection rows + bias -> queries and keys normed over the whole row (m.row_norm), values mixed with `first` [T, G *
    vdim], the values of the first mixing layer (None: this layer mixes nothing in); keys and values go to the paged cache at
    rows.slots. packed: as in qk_norm_rope_cache. Returns (queries or packed rows, values [T, G * vdim] before mixing, if they are
    the first)."""
    T, H, G = proj.shape[0], m.heads, m.kv_heads
    _debug.check_range("qkv_rows", "slots", rows.slots, 0, kc.shape[0] * kc.shape[1], allow=-1)
    b = lw.get("b_in")
    qn, kn = (lw["q_norm"], lw["k_norm"]) if m.row_norm else (None, None)
    keep = m.v_mix and first is None
    if not _lib.use_native(proj):
        p = proj.float() if b is None else proj.float() + b
        q, k, v = (p[:, sec[s]:sec[s] + n] for s, n in (("q", H * m.dim), ("k", G * m.dim), ("v", G * m.vdim)))
        if m.row_norm:
            q, k = _rms(q, eps) * qn, _rms(k, eps) * kn
        own = v.to(dtype)
        if m.v_mix and not keep:
            v = v + lw["v_mix"] * (first.float() - v)
        ok = rows.slots >= 0
        kc.view(-1, G, kc.shape[3])[rows.slots[ok], :, :m.dim] = k.reshape(T, G, m.dim).to(dtype)[ok]
        vc.view(-1, G, vc.shape[3])[rows.slots[ok], :, :m.vdim] = v.reshape(T, G, m.vdim).to(dtype)[ok]
        return q.to(dtype), own if keep else None
    dev = proj.device
    if packed is not None:
        hd, n = PACKED_HD, rows.nd + packed.rows
        q = (torch.empty if m.dim == m.vdim == hd else torch.zeros)((n, (H + 2 * G) * hd), dtype=dtype, device=dev)
        kp, vp, dst = q[:, H * hd:], q[:, (H + G) * hd:], packed.dst
    else:
        hd, kp, vp, dst = round8(m.dim), None, None, None
        q = torch.empty((T, H * hd), dtype=dtype, device=dev)
    own = act(T, G * m.vdim, dtype, dev) if keep else None
    mix = first if m.v_mix and not keep else None
    f = _lib.fn("dlti_qkv_rows", [_V, _L, _I, _I, _I, _V, _V, _V, _F, _V, _L, _V, _V, _L, _V, _V, _V, _I, _I, _V, _L, _I, _V, _V, _V, _I, _L, _I,
                                  _I, _I, _I, _I, _I, _V])
    _lib.check(f(_p(proj), proj.stride(0), sec["q"], sec["k"], sec["v"], _p(b), _p(qn), _p(kn), float(eps), _p(mix), 0 if mix is None else
                 mix.stride(0), _p(lw["v_mix"]) if mix is not None else None, _p(own), 0 if own is None else own.stride(0), _p(rows.slots), _p(kc),
                 _p(vc), kc.shape[3], vc.shape[3], _p(q), q.stride(0), hd, _p(kp), _p(vp), _p(dst), rows.nd, T, H, G, m.dim, m.vdim, int(acc),
                 _lib.dtype_code(dtype), _lib.stream_ptr()), "qkv_rows")
    if packed is not None and packed.prefix:
        prefix_rows(q[rows.nd:], m, packed, kc, vc)
    return q, own


def paged_attention_ref(q, m, rows: Rows, kc, vc, gate, sink=None, bias=None, out_gate=None):
    """Every row against the cached keys of its sequence that it may see."""
    T, H, G = q.shape[0], m.heads, m.kv_heads
    bs, hd = kc.shape[1], q.shape[1] // H
    kf, vf = kc.view(-1, G, kc.shape[3]).float(), vc.view(-1, G, vc.shape[3]).float()
    out = torch.zeros(T, H, m.vdim)
    for t in range(T):
        s, p = int(rows.seq[t]), int(rows.pos[t])
        lo = p // m.chunk * m.chunk if m.chunk else max(0, p - m.window + 1) if m.window else 0
        j = torch.arange(lo, min(p + 1, int(rows.ctx[s])))
        if not len(j):
            continue
        sl = rows.tables[s, j // bs].long() * bs + j % bs
        k = kf[sl][..., :m.dim].repeat_interleave(H // G, 1)
        v = vf[sl][..., :m.vdim].repeat_interleave(H // G, 1)
        qq = q[t].float().view(H, hd)[:, :m.dim]
        x = torch.einsum("hd,jhd->hj", qq, k) * m.scale
        if m.softcap:
            x = m.softcap * torch.tanh(x / m.softcap)
        if bias is not None:
            far = p - j >= bias.shape[1]
            x = x + bias[:, (p - j).clamp(max=bias.shape[1] - 1)].masked_fill(far, 0.0)
        if sink is not None:
            x = torch.cat([x, sink[:, None]], 1)
        out[t] = torch.einsum("hj,jhd->hd", torch.softmax(x, -1)[:, :len(j)], v)
    if gate is not None:
        out *= gate[:, :, None]
    if out_gate is not None:
        out *= torch.sigmoid(out_gate.float()).view(T, H, m.vdim)
    return out.reshape(T, -1).to(q.dtype)


def _more(bias, out_gate):
    """Score biases and output gates as the attention kernels take them."""
    return (_p(bias), 0 if bias is None else bias.shape[1], _p(out_gate), 0 if out_gate is None else out_gate.stride(0))


_MORE = [_V, _I, _V, _L]


def attn_rows(q, m, rows: Rows, kc, vc, gate, out, sink=None, bias=None, out_gate=None):
    """fp32-arithmetic attention of the rows of q, one warp per (row, head)."""
    hd = q.shape[1] // m.heads
    f = _lib.fn("dlti_attn_rows", [_V, _L, _I, _V, _V, _I, _I, _V, _I, _I, _V, _V, _V, _I, _I, _I, _I, _I, _I, _F, _F, _V, _V, *_MORE, _V, _L, _L, _I, _V])
    _lib.check(f(_p(q), q.stride(0), hd, _p(kc), _p(vc), kc.shape[3], vc.shape[3], _p(rows.tables), rows.tables.shape[1], kc.shape[1],
                 _p(rows.ctx), _p(rows.seq), _p(rows.pos), m.heads, m.kv_heads, m.dim, m.vdim, m.chunk, m.window, m.scale, m.softcap,
                 _p(gate), _p(sink), *_more(bias, out_gate), _p(out), out.stride(0), q.shape[0], _lib.dtype_code(q.dtype), _lib.stream_ptr()), "attn_rows")
    return out


_ws: dict = {}
_ws_retired: list = []


def _workspace(device, floats: int) -> torch.Tensor:
    ws = _ws.get(str(device))
    if ws is None or ws.numel() < floats:
        if ws is not None:
            _ws_retired.append(ws)             # captured CUDA graphs may still point at it
        ws = _ws[str(device)] = torch.empty(max(floats, 1 << 20), dtype=torch.float32, device=device)
    return ws


def attn_paged_decode(q, m, rows: Rows, kc, vc, gate, out, splits: int | None = None, sink=None, bias=None, out_gate=None):
    """Decode rows (bf16): row b of q against the visible keys of sequence b, split over CTAs."""
    B, hd, bs = q.shape[0], q.shape[1] // m.heads, kc.shape[1]
    if splits is None:
        reach = min(rows.max_ctx or 1 << 30, m.chunk or m.window or 1 << 30, rows.tables.shape[1] * bs)
        ctas = max(1, B) * m.kv_heads * -(-(m.heads // m.kv_heads) // 16)
        splits = max(1, min(32, 3 * 148 // ctas, -(-reach // 64)))     # one wave of three CTAs per SM
    ws = _workspace(q.device, B * m.heads * splits * (m.vdim + 2)) if splits > 1 else None
    f = _lib.fn("dlti_attn_paged_decode", [_V, _L, _I, _V, _V, _I, _I, _V, _I, _I, _V, _I, _I, _I, _I, _I, _I, _I, _F, _F, _V, _V, *_MORE, _I, _V, _V, _L, _V])
    _lib.check(f(_p(q), q.stride(0), hd, _p(kc), _p(vc), kc.shape[3], vc.shape[3], _p(rows.tables), rows.tables.shape[1], bs,
                 _p(rows.ctx), B, m.heads, m.kv_heads, m.dim, m.vdim, m.chunk, m.window, m.scale, m.softcap, _p(gate), _p(sink),
                 *_more(bias, out_gate), splits, _p(ws),
                 _p(out), out.stride(0), _lib.stream_ptr()), "attn_paged_decode")
    return out


def attn_paged_prefill(q, m, rows: Rows, kc, vc, gate, out, sink=None, bias=None, out_gate=None):
    """Prompt rows (bf16): q, gate and out cover all rows of the step."""
    hd = q.shape[1] // m.heads
    f = _lib.fn("dlti_attn_paged_prefill", [_V, _L, _I, _V, _V, _I, _I, _V, _I, _I, _V, _V, _I, _I, _I, _I, _I, _I, _I, _I, _I, _F, _F, _V, _V,
                                            *_MORE, _V, _L, _V])
    _lib.check(f(_p(q), q.stride(0), hd, _p(kc), _p(vc), kc.shape[3], vc.shape[3], _p(rows.tables), rows.tables.shape[1], kc.shape[1],
                 _p(rows.ctx), _p(rows.cu), rows.nd, rows.nseq - rows.nd, rows.max_seqlen, m.heads, m.kv_heads, m.dim, m.vdim, m.chunk,
                 m.window, m.scale, m.softcap, _p(gate), _p(sink), *_more(bias, out_gate), _p(out), out.stride(0), _lib.stream_ptr()),
               "attn_paged_prefill")
    return out


def packed_attention(qkv, m, rows: Rows, pieces: Pieces, kc, vc, gate, sink=None, bias=None, out_gate=None):
    """Attention of a step from the packed rows of qk_norm_rope_cache, qkv_rows or conv_qkv: decode rows through the pages, prompt rows through the
    varlen tcgen05 kernel. Needs heads of up to 128 dimensions, values in multiples of 8."""
    T, H, nd = rows.pos.numel(), m.heads, rows.nd
    out = act(T, H * m.vdim, qkv.dtype, qkv.device)
    if nd:
        attn_paged_decode(qkv[:nd, :H * PACKED_HD], m, rows, kc, vc, gate, out, sink=sink, bias=bias, out_gate=out_gate)
    attn_fwd_split(qkv[nd:], m, H, m.kv_heads, pieces, None if gate is None else gate[nd:], out[nd:], sink=sink, bias=bias,
                   out_gate=None if out_gate is None else out_gate[nd:])
    return out


PACKED_BIAS = 4096           # distances with a bias of their own that the packed prompt kernel has room for


def attn_fwd_split(qkv, m, heads, kv_heads, pieces: Pieces, gate, out, sink=None, bias=None, out_gate=None):
    """Causal attention of packed rows [q heads | k heads | v heads], each 128 columns, within every piece."""
    f = _lib.fn("dlti_attn_fwd_split", [_V, _V, _L, _V, _V, _V, _V, _V, _I, _I, _L, _I, _I, _I, _I, _F, _F, *_MORE, _V])
    _lib.check(f(_p(qkv), _p(out), out.stride(0), _p(gate), _p(sink), _p(pieces.cu), _p(pieces.q0), _p(pieces.out0), pieces.cu.numel() - 1,
                 pieces.longest, qkv.shape[0], heads, kv_heads, m.vdim, m.window, m.scale, m.softcap, *_more(bias, out_gate),
                 _lib.stream_ptr()), "attn_fwd_split")


def paged_attention(q, m, rows: Rows, kc, vc, gate, sink=None, bias=None, out_gate=None):
    """Attention of every row of a step over the paged cache -> [T, heads * vdim], head outputs times `gate` [T, H]. bias [H, n]: added
    to the scores at the distances below n; out_gate [T, heads * vdim]: outputs are multiplied by its sigmoid."""
    more = dict(sink=sink, bias=bias, out_gate=out_gate)
    if not _lib.use_native(q):
        return paged_attention_ref(q, m, rows, kc, vc, gate, **more)
    _debug.check_paged("paged_attention", rows.tables, rows.ctx, kc.shape[0], kc.shape[1])
    out = act(q.shape[0], m.heads * m.vdim, q.dtype, q.device)
    if q.dtype == torch.float32 or max(kc.shape[3], vc.shape[3]) > 256:
        return attn_rows(q, m, rows, kc, vc, gate, out, **more)
    if rows.nd:
        attn_paged_decode(q[:rows.nd], m, rows, kc, vc, gate, out, **more)
    if rows.nseq > rows.nd:
        attn_paged_prefill(q, m, rows, kc, vc, gate, out, **more)
    return out


# ---- recurrences -------------------------------------------------------------------------------------------
def short_conv(proj, col, C_, w, b, state, rows: Rows, dtype, acc=False, width=0, split=0):
    """silu of the causal convolution of channels [col, col + C_) of the projection rows; w [taps, >= C_] tap-major,
    state [slots, taps - 1, C_] = inputs of earlier steps (read only; linear_scan's tail job renews it). Returns (out
    [T, C_], proj): with acc (decode rows only) proj is the projection rounded to the compute dtype, else as given. split > 0 (with
    acc): columns from split on as an fp32 result of their own, (out, proj [T, split], fp32 columns)."""
    T, taps = proj.shape[0], w.shape[0]
    if not _lib.use_native(proj):
        out = torch.zeros(T, C_)
        for s in range(rows.nseq):
            r0, n, start = rows.bounds(s)
            x = proj[r0:r0 + n, col:col + C_].float()
            slot = int(rows.state[s])
            h = state[slot].float() if state is not None and start > 0 and slot >= 0 else torch.zeros(taps - 1, C_)
            x = torch.cat([h, x])
            out[r0:r0 + n] = b[:C_] + sum(w[k, :C_] * x[k:k + n] for k in range(taps))
        return torch.nn.functional.silu(out).to(dtype), proj
    out = act(T, C_, dtype, proj.device)
    raw = act(T, split or width, dtype, proj.device) if acc else None
    tail = torch.empty((T, width - split), dtype=torch.float32, device=proj.device) if split else None
    f = _lib.fn("dlti_short_conv", [_V, _L, _I, _I, _I, _V, _V, _I, _V, _V, _V, _V, _V, _I, _V, _L, _V, _L, _I, _V, _L, _I, _L, _I, _I, _V])
    _lib.check(f(_p(proj), proj.stride(0), col, C_, taps, _p(w), _p(b), w.stride(0), _p(state), _p(rows.state), _p(rows.seq),
                 _p(rows.ctx), _p(rows.cu), rows.nd, _p(out), out.stride(0), _p(raw), 0 if raw is None else raw.stride(0), width, _p(tail),
                 0 if tail is None else tail.stride(0), split, T, int(acc), _lib.dtype_code(dtype), _lib.stream_ptr()), "short_conv")
    return (out, raw, tail) if split else (out, raw if acc else proj)


@dataclass
class Decay:
    """Decay and step size of a recurrence: a constant factor per head (const), or per token from raw step sizes dt
    (softplus(dt + bias), decay exp(-exp(A_log) * step))."""
    const: torch.Tensor | None = None
    dt: torch.Tensor | None = None
    dt_bias: torch.Tensor | None = None
    A_log: torch.Tensor | None = None
    D: torch.Tensor | None = None


def linear_scan_ref(q, k, v, decay: Decay, state, rows: Rows, heads, groups, N, P, silu, conv_src, conv_col, conv_state):
    T, dtype = q.shape[0], v.dtype
    f = (lambda x: torch.nn.functional.silu(x.float()).to(dtype).float()) if silu else (lambda x: x.float())
    rep = heads // groups
    qf, kf = (f(x).reshape(T, groups, N).repeat_interleave(rep, 1) for x in (q, k))
    vf = f(v).reshape(T, heads, P)
    if decay.const is not None:
        st, a = torch.ones(T, heads), decay.const.expand(T, heads)
    else:
        st = torch.nn.functional.softplus(decay.dt.float() + decay.dt_bias, threshold=1e9)
        a = torch.exp(-torch.exp(decay.A_log) * st)
    out = torch.zeros(T, heads, P)
    for s in range(rows.nseq):
        r0, n, start = rows.bounds(s)
        slot = int(rows.state[s])
        S = state[slot].clone() if start > 0 and slot >= 0 else torch.zeros(heads, N, P)
        for t in range(r0, r0 + n):
            S = a[t][:, None, None] * S + kf[t][:, :, None] * (st[t][:, None] * vf[t])[:, None, :]
            out[t] = (qf[t][:, :, None] * S).sum(1)
        if slot >= 0:
            state[slot] = S
            if conv_state is not None:
                rest = conv_state.shape[1]
                h = conv_state[slot] if start > 0 else torch.zeros_like(conv_state[slot])
                x = torch.cat([h, conv_src[r0:r0 + n, conv_col:conv_col + conv_state.shape[2]].to(h.dtype)])
                conv_state[slot] = x[x.shape[0] - rest:].clone()
    if decay.D is not None:
        out += decay.D[:, None] * vf
    return out.reshape(T, -1).to(dtype)


def linear_scan(q, k, v, decay: Decay, state, rows: Rows, heads, groups, N, P, silu=False, conv_src=None, conv_col=0, conv_state=None):
    """S <- a S + k (step v)^T, o = S^T q (+ D v) over the rows of every sequence; q, k [T, groups * N] views, v [T,
    heads * P], state [slots, heads, N, P] fp32 updated in place. silu: applied to q, k, v first (prompt rows of the views
    may be overwritten with it). conv_state: renewed
    from the rows of conv_src (see short_conv)."""
    if not _lib.use_native(q):
        return linear_scan_ref(q, k, v, decay, state, rows, heads, groups, N, P, silu, conv_src, conv_col, conv_state)
    out = act(q.shape[0], heads * P, v.dtype, q.device)
    nd, nseq = rows.nd, rows.nseq
    conv = (conv_src, conv_col, conv_state)
    if nseq > nd and q.dtype == torch.bfloat16 and N % 8 == 0 and P % 8 == 0 and N <= 256 and rows.max_seqlen >= _CHUNKED_FROM:
        if nd:
            _scan_tokens(q, k, v, decay, state, rows, 0, nd, heads, groups, N, P, silu, conv, out)
        if silu:
            for x in _merge_sections(q, k, v):
                silu_rows_(x[nd:])
        _scan_chunked(q, k, v, decay, state, rows, nd, nseq - nd, heads, groups, N, P, conv, out)
    else:
        _scan_tokens(q, k, v, decay, state, rows, 0, nseq, heads, groups, N, P, silu, conv, out)
    return out


_CHUNKED_FROM = 16           # longest portion of a step from which the chunked kernel takes its prompts


def _merge_sections(*xs):
    """Neighbouring sections of one projection as a single view where only alignment padding (< 8 columns) lies between
    them, rounded up to whole 8-column pieces (padding columns are zero)."""
    out = []
    for x in xs:
        n = round8(x.shape[1])
        if out and x.stride(0) == out[-1].stride(0) and x.data_ptr() == out[-1].data_ptr() + out[-1].shape[1] * x.element_size():
            n += out.pop().shape[1]
            x = xs_base
        xs_base = x
        out.append(x.as_strided((x.shape[0], n), x.stride()))
    return out


def silu_rows_(x):
    """In place on a [rows, n] bf16 section of a projection, n a multiple of 8."""
    f = _lib.fn("dlti_silu_rows", [_V, _L, _L, _I, _I, _V])
    _lib.check(f(_p(x), x.stride(0), x.shape[0], x.shape[1], _lib.dtype_code(x.dtype), _lib.stream_ptr()), "silu_rows")


def _conv_args(conv):
    src, col, st = conv
    return (_p(src), 0 if src is None else src.stride(0), col, 0 if st is None else st.shape[1], 0 if st is None else st.shape[2], _p(st))


def _scan_tokens(q, k, v, decay, state, rows, seq0, nseq, heads, groups, N, P, silu, conv, out):
    f = _lib.fn("dlti_linear_scan", [_V, _L, _V, _L, _V, _L, _I, _I, _V, _V, _L, _V, _V, _V, _V, _V, _V, _V, _I, _I, _I, _I, _I, _I, _V,
                                     _L, _V, _L, _I, _I, _I, _V, _I, _V])
    dt = decay.dt
    _lib.check(f(_p(q), q.stride(0), _p(k), k.stride(0), _p(v), v.stride(0), heads // groups, int(silu), _p(decay.const), _p(dt),
                 0 if dt is None else dt.stride(0), _p(decay.dt_bias), _p(decay.A_log), _p(decay.D), _p(state), _p(rows.state),
                 _p(rows.ctx), _p(rows.cu), rows.nd, seq0, nseq, heads, N, P, _p(out), out.stride(0), *_conv_args(conv),
                 _lib.dtype_code(v.dtype), _lib.stream_ptr()), "linear_scan")


def _scan_chunked(q, k, v, decay, state, rows, seq0, nseq, heads, groups, N, P, conv, out):
    f = _lib.fn("dlti_linear_scan_chunked", [_V, _L, _V, _L, _V, _L, _I, _V, _V, _L, _V, _V, _V, _V, _V, _V, _V, _I, _I, _I, _I, _I, _I,
                                             _V, _L, _V, _L, _I, _I, _I, _V, _V])
    dt = decay.dt
    _lib.check(f(_p(q), q.stride(0), _p(k), k.stride(0), _p(v), v.stride(0), heads // groups, _p(decay.const), _p(dt),
                 0 if dt is None else dt.stride(0), _p(decay.dt_bias), _p(decay.A_log), _p(decay.D), _p(state), _p(rows.state),
                 _p(rows.ctx), _p(rows.cu), rows.nd, seq0, nseq, heads, N, P, _p(out), out.stride(0), *_conv_args(conv),
                 _lib.stream_ptr()), "linear_scan_chunked")


def mlstm_scan_ref(q, k, v, gates, gate_b, cap, state, vec, rows: Rows, heads, N, P):
    T, dtype = q.shape[0], v.dtype
    qf, kf, vf = q.float().reshape(T, heads, N) * N ** -0.5, k.float().reshape(T, heads, N), v.float().reshape(T, heads, P)
    g = cap * torch.tanh((gates[:, :2 * heads] + gate_b) / cap)
    li, lf = g[:, :heads], torch.nn.functional.logsigmoid(g[:, heads:])
    out = torch.zeros(T, heads, P)
    sl = -(-P // 32)
    for s in range(rows.nseq):
        r0, n, start = rows.bounds(s)
        slot = int(rows.state[s])
        have = start > 0 and slot >= 0
        S = state[slot].clone() if have else torch.zeros(heads, N, P)
        w = vec[slot].view(heads, sl, N + 1)[:, 0].clone() if have else torch.zeros(heads, N + 1)
        nv, m = w[:, :N], w[:, N]
        for t in range(r0, r0 + n):
            mn = torch.maximum(lf[t] + m, li[t])
            a, b = 1 + torch.expm1(lf[t] + m - mn), torch.exp(li[t] - mn)
            m = mn
            S = a[:, None, None] * S + (b[:, None] * kf[t])[:, :, None] * vf[t][:, None, :]
            nv = a[:, None] * nv + b[:, None] * kf[t]
            den = torch.maximum((nv * qf[t]).sum(1).abs(), torch.exp(-m)) + 1e-6
            out[t] = (qf[t][:, :, None] * S).sum(1) / den[:, None]
        if slot >= 0:
            state[slot] = S
            vec[slot] = torch.cat([nv, m[:, None]], 1).repeat(1, sl)
    return out.reshape(T, -1).to(dtype)


def mlstm_vec(N: int, P: int) -> int:
    """fp32 numbers per head that an mLSTM keeps beside its matrix: n and m, once per slice of 32 value columns."""
    return -(-P // 32) * (N + 1)


def mlstm_scan(q, k, v, gates, gate_b, cap, state, vec, rows: Rows, heads, N, P):
    """mLSTM over the rows of every sequence: q, k [T, heads * N], v [T, heads * P] views; gates [T, >= 2 heads] raw fp32 log gates
    (input, then forget) with bias gate_b; state [slots, heads, N, P] and vec [slots, heads, mlstm_vec] updated in place."""
    if not _lib.use_native(q):
        return mlstm_scan_ref(q, k, v, gates, gate_b, cap, state, vec, rows, heads, N, P)
    out = act(q.shape[0], heads * P, v.dtype, q.device)
    f = _lib.fn("dlti_mlstm_scan", [_V, _L, _V, _L, _V, _L, _V, _L, _V, _F, _F, _V, _V, _V, _V, _V, _I, _I, _I, _I, _I, _I, _V, _L, _I, _I, _V])

    def run(seq0, nseq, chunked):
        _lib.check(f(_p(q), q.stride(0), _p(k), k.stride(0), _p(v), v.stride(0), _p(gates), gates.stride(0), _p(gate_b), float(cap), N ** -0.5,
                     _p(state), _p(vec), _p(rows.state), _p(rows.ctx), _p(rows.cu), rows.nd, seq0, nseq, heads, N, P, _p(out), out.stride(0),
                     int(chunked), _lib.dtype_code(v.dtype), _lib.stream_ptr()), "mlstm_scan")

    nd, nseq = rows.nd, rows.nseq
    if nseq > nd and q.dtype == torch.bfloat16 and N % 8 == 0 and P % 8 == 0 and N <= 256 and rows.max_seqlen >= _CHUNKED_FROM:
        if nd:
            run(0, nd, False)
        run(nd, nseq - nd, True)
    else:
        run(0, nseq, False)
    return out
