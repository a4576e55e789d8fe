"""Latent attention (csrc/latent.cu): one cached row [latent | rotated key part] per token for all heads. Decode rows, short
portions and fp32 take the absorbed form (queries moved into the latent space, attention over the cached rows themselves);
prompts take the expanded form (keys and values of every head by one GEMM, then causal attention)."""
from __future__ import annotations

import torch

from ..models.stack import AttentionMixer, LatentAttentionMixer, round8, round16
from . import _debug, _lib
from .gemm import gemm
from .stack import PACKED_HD, _F, _I, _L, _V, Pieces, Rows, _p, _rms, _workspace, act, attn_fwd_split, attn_paged_prefill, attn_rows


def _rotate(x, pos, rope, tabs):
    """First rope.dims coordinates of x [T, n, dim] turned by their position."""
    if rope is None:
        return x
    c, s = (t[pos.long()][:, None, :] for t in tabs)
    r, h = rope.dims, rope.dims // 2
    a, b = (x[..., 0:r:2], x[..., 1:r:2]) if rope.interleaved else (x[..., :h], x[..., h:r])
    u, v = a * c - b * s, b * c + a * s
    return torch.cat([torch.stack([u, v], -1).flatten(-2) if rope.interleaved else torch.cat([u, v], -1), x[..., r:]], -1)


def latent_attention_ref(proj, sec, m: LatentAttentionMixer, lw, eps, rows: Rows, tabs, cache, dtype):
    T, H, R = proj.shape[0], m.heads, m.kv_rank
    p = proj.float()
    q = p[:, sec["q"]:sec["q"] + H * m.qk_dim].reshape(T, H, m.qk_dim)
    c = _rms(p[:, sec["dkv"]:sec["dkv"] + R], eps) * lw["kv_norm"]
    k = _rotate(p[:, sec["dkv"] + R:sec["dkv"] + R + m.rot_dim][:, None], rows.pos, m.rope, tabs)[:, 0]
    flat, ok = cache.view(-1, m.pitch), rows.slots >= 0
    flat[rows.slots[ok], :R] = c[ok].to(dtype)
    flat[rows.slots[ok], m.rot_at:m.rot_at + m.rot_dim] = k[ok].to(dtype)
    qr = _rotate(q[..., m.dim:], rows.pos, m.rope, tabs)
    qa = torch.einsum("thd,hdr->thr", q[..., :m.dim], lw["w_uk"][:H * m.dim].float().view(H, m.dim, R))
    uv = lw["w_uv"][:H * m.vdim].float().view(H, m.vdim, R)
    out, bs = torch.zeros(T, H, m.vdim), cache.shape[1]
    for t in range(T):
        s = int(rows.seq[t])
        j = torch.arange(min(int(rows.pos[t]) + 1, int(rows.ctx[s])))
        if not len(j):
            continue
        row = flat[rows.tables[s, j // bs].long() * bs + j % bs].float()
        cc, kk = row[:, :R], row[:, m.rot_at:m.rot_at + m.rot_dim]
        sc = (qa[t] @ cc.t() + qr[t] @ kk.t()) * m.scale
        if m.sink:
            sc = torch.cat([sc, lw["sink"][:, None]], 1)
        out[t] = torch.einsum("hr,hvr->hv", torch.softmax(sc, -1)[:, :len(j)] @ cc, uv)
    if m.head_gate:
        out *= torch.sigmoid(p[:, sec["g"]:sec["g"] + H])[:, :, None]
    return out.reshape(T, -1).to(dtype)


def head_gemm(a, a_hd, b, out, o_hd, heads, K, N, kn):
    """out[t, h, :N] = a[t, h, :K] B_h with B_h = rows h K ... of b [H K, N] (kn) or the transpose of rows h N ... of b [H N, K];
    heads are a_hd / o_hd columns apart in a and out."""
    f = _lib.fn("dlti_head_gemm", [_V, _L, _I, _V, _L, _V, _L, _I, _L, _I, _I, _I, _I, _I, _V])
    _lib.check(f(_p(a), a.stride(0), a_hd, _p(b), b.stride(0), _p(out), out.stride(0), o_hd, a.shape[0], heads, K, N, int(kn),
                 _lib.dtype_code(a.dtype), _lib.stream_ptr()), "head_gemm")
    return out


def latent_decode(q, m: LatentAttentionMixer, rows: Rows, cache, gate, sink, out, splits: int | None = None, one_per_seq=True):
    """Absorbed attention (bf16) of the rows of q [n, heads * pitch] over the cached rows of their sequences (row t = newest token
    of sequence t with one_per_seq) -> out [n, heads * round16(kv_rank)], times gate."""
    n, bs, o_hd = q.shape[0], cache.shape[1], round16(m.kv_rank)
    tile = 16 if m.heads <= 16 else 32
    if splits is None:
        reach = min(rows.max_ctx or 1 << 30, rows.tables.shape[1] * bs)
        resident = 1 if m.pitch > 200 else 2                # CTAs of an SM (shared memory)
        splits = max(1, min(32, 148 * resident // max(1, n * -(-m.heads // tile)), -(-reach // 64)))
    ws = _workspace(q.device, n * m.heads * splits * (o_hd + 2)) if splits > 1 else None
    f = _lib.fn("dlti_latent_decode", [_V, _V, _I, _I, _V, _I, _I, _V, _V, _V, _L, _I, _F, _V, _V, _I, _I, _V, _V, _I, _V])
    _lib.check(f(_p(q), _p(cache), m.pitch, m.kv_rank, _p(rows.tables), rows.tables.shape[1], bs, _p(rows.ctx),
                 None if one_per_seq else _p(rows.seq), None if one_per_seq else _p(rows.pos), n, m.heads, m.scale, _p(sink), _p(gate), tile,
                 splits, _p(ws), _p(out), o_hd, _lib.stream_ptr()), "latent_decode")
    return out


def expand(m: LatentAttentionMixer, dtype, pieces: Pieces | None) -> bool:
    """Prompt rows of the step take the expanded form."""
    return pieces is not None and dtype == torch.bfloat16 and m.head_pitch <= 256


def latent_prep(proj, sec, m: LatentAttentionMixer, kv_norm, eps, rows: Rows, tabs, cache, dtype, pieces: Pieces | None, acc):
    """Projection rows -> cache rows at rows.slots, head gates, and the queries: absorbed rows (all of them without pieces, else
    the decode rows) as (unrotated [n, H * round8(dim)], latent-space rows [n, H * pitch] with the rotated part in place), prompt
    rows with pieces as the query columns of the packed rows (or [rows, H * head_pitch]) and their cache rows laid out for the
    expansion. Returns (qn, ql, packed, lat, gate, absorbed rows)."""
    T, H, dev = proj.shape[0], m.heads, proj.device
    nabs = rows.nd if pieces is not None else T
    gate = torch.empty((T, H), dtype=torch.float32, device=dev) if "g" in sec else None
    qn = ql = buf = lat = qdst = dst = None
    if nabs:
        qn = torch.empty((nabs, H * round8(m.dim)), dtype=dtype, device=dev)
        ql = torch.empty((nabs, H * m.pitch), dtype=dtype, device=dev)
    if pieces is not None:
        lat, dst = torch.empty((pieces.rows, m.pitch), dtype=dtype, device=dev), pieces.dst
        if m.head_pitch == PACKED_HD:
            buf, qdst = torch.empty((pieces.rows, 3 * H * PACKED_HD), dtype=dtype, device=dev), dst
            if pieces.prefix:
                buf[:, :H * PACKED_HD].zero_()             # cached rows have no query
        else:
            buf = torch.empty((T - nabs, H * m.head_pitch), dtype=dtype, device=dev)
    f = _lib.fn("dlti_latent_prep", [_V, _L, _I, _I, _I, _I, _I, _I, _I, _I, _I, _V, _V, _V, _V, _F, _V, _V, _I, _I, _I, _V, _I, _V, _V, _L, _I,
                                     _V, _V, _V, _V, _L, _I, _I, _V])
    _lib.check(f(_p(proj), proj.stride(0), sec["q"], sec["dkv"], sec["g"] if "g" in sec else -1, H, m.dim, m.rot_dim, m.kv_rank,
                 m.rope.dims if m.rope is not None else 0, int(m.rope.interleaved) if m.rope is not None else 1,
                 _p(tabs[0]) if tabs is not None else None, _p(tabs[1]) if tabs is not None else None, _p(rows.pos), _p(kv_norm), float(eps),
                 _p(rows.slots), _p(cache), m.pitch, m.rot_at, nabs, _p(qn), round8(m.dim), _p(ql), _p(buf), 0 if buf is None else buf.stride(0),
                 m.head_pitch, _p(lat), _p(qdst), _p(dst), _p(gate), T, int(acc), _lib.dtype_code(dtype), _lib.stream_ptr()), "latent_prep")
    return qn, ql, buf, lat, gate, nabs


def absorbed(qn, ql, m: LatentAttentionMixer, lw, rows: Rows, cache, gate, out):
    """Absorbed attention of the first rows of a step -> out [n, heads * vdim]."""
    n, H, R = ql.shape[0], m.heads, m.kv_rank
    sink = lw.get("sink")
    head_gemm(qn, round8(m.dim), lw["w_uk"], ql, m.pitch, H, m.dim, R, True)
    if ql.dtype == torch.float32 or R > 512:
        lm = AttentionMixer(H, 1, m.pitch, R, m.scale)
        o = attn_rows(ql, lm, rows, cache, cache, gate, torch.empty((n, H * R), dtype=ql.dtype, device=ql.device), sink=sink)
        o_hd = R
    else:
        o_hd = round16(R)
        o = latent_decode(ql, m, rows, cache, gate, sink, torch.empty((n, H * o_hd), dtype=ql.dtype, device=ql.device), one_per_seq=n == rows.nd)
    return head_gemm(o, o_hd, lw["w_uv"], out, m.vdim, H, R, m.vdim, False)


def expanded(buf, lat, m: LatentAttentionMixer, lw, w_expand, rows: Rows, cache, pieces: Pieces, gate, out):
    """Attention of the prompt rows of a step -> out [prompt rows, heads * vdim]."""
    H, hp = m.heads, m.head_pitch
    if pieces.prefix:
        f = _lib.fn("dlti_latent_rows", [_V, _V, _I, _V, _V, _L, _V])
        _lib.check(f(_p(lat), _p(cache), m.pitch, _p(pieces.prow), _p(pieces.pslot), pieces.prefix, _lib.stream_ptr()), "latent_rows")
    sink, lat = lw.get("sink"), lat[:, :m.cols]
    if hp == PACKED_HD:
        gemm(lat, w_expand, out=buf[:, H * hp:], two_cta=False)      # a short contraction: bound by the rows it writes
        attn_fwd_split(buf, m, H, H, pieces, gate, out, sink=sink)
        return out
    n = pieces.rows
    k, v = (gemm(lat, w).view(n, 1, H, hp) for w in (w_expand[:H * hp], w_expand[H * hp:]))
    tables = (pieces.cu[:-1, None] + torch.arange(pieces.longest, dtype=torch.int32, device=lat.device)).clamp_max(n - 1)
    own = Rows(rows.pos, rows.seq, rows.slots, rows.ctx[rows.nd:], rows.cu, tables, rows.state, 0, rows.max_seqlen, rows.max_ctx)
    return attn_paged_prefill(buf, AttentionMixer(H, H, m.qk_dim, m.vdim, m.scale), own, k, v, gate, out, sink=sink)


def latent_attention(proj, sec, m: LatentAttentionMixer, lw, w_expand, eps, rows: Rows, tabs, cache, dtype, pieces: Pieces | None = None, acc=False):
    """Merged projection rows [q | latent, rotated key part | gates] -> attention outputs [T, heads * vdim] of a step; the cached
    rows [blocks, block size, 1, pitch] are written at rows.slots."""
    _debug.check_range("latent_attention", "slots", rows.slots, 0, cache.shape[0] * cache.shape[1], allow=-1)
    if not _lib.use_native(proj):
        return latent_attention_ref(proj, sec, m, lw, eps, rows, tabs, cache, dtype)
    _debug.check_paged("latent_attention", rows.tables, rows.ctx, cache.shape[0], cache.shape[1])
    if not expand(m, dtype, pieces):
        pieces = None
    qn, ql, buf, lat, gate, n = latent_prep(proj, sec, m, lw["kv_norm"], eps, rows, tabs, cache, dtype, pieces, acc)
    out = act(proj.shape[0], m.heads * m.vdim, dtype, proj.device)
    if n:
        absorbed(qn, ql, m, lw, rows, cache, gate, out[:n])
    if pieces is not None:
        expanded(buf, lat, m, lw, w_expand, rows, cache, pieces, None if gate is None else gate[n:], out[n:])
    return out
