"""Logozen against its plain implementation (tests/ref_logozen.py): each mechanism alone, then whole models through the
engine in every kind of schedule. CPU runs use the ops' PyTorch restatements, GPU runs the kernels."""
import copy
import json
import math
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

from dlti_b200.models import logozen as LZ
from dlti_b200.models.stack import AttentionMixer, LatentAttentionMixer, Rope, Sections, mixer_sections, round8, round16
from dlti_b200.ops import _lib
from dlti_b200.ops import latent as LA
from dlti_b200.ops import stack as K
from dlti_b200.ops import streams as H
from tests import ref_logozen as R
from tests.logozen_util import CONFIGS, ZOO
from tests.stack_util import mixed_schedule, pieces_for, random_portions, row_errors, rows_for

F32, BF16 = torch.float32, torch.bfloat16
GPU = pytest.mark.gpu
MODES = [pytest.param("cpu", F32, id="cpu"), pytest.param("cuda", F32, marks=GPU, id="gpu-f32"),
         pytest.param("cuda", BF16, marks=GPU, id="gpu-bf16")]
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def tol(dtype, f32, bf16):
    return bf16 if dtype == BF16 else f32


def rel(a, b):
    return float((a.double().cpu() - b).norm() / b.norm())


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(g, *s):
    """Random values that every compute dtype represents."""
    return torch.randn(*s, generator=g).to(BF16)


def acts(x, device, dtype):
    """x as an activation view (row pitch a multiple of 8)."""
    out = K.act(x.shape[0], x.shape[1], dtype, device)
    out.copy_(x)
    return out


def padded(x, device):
    """fp32 [taps, channels] with a row pitch of a multiple of 8."""
    out = torch.zeros(x.shape[0], round8(x.shape[1]))
    out[:, :x.shape[1]] = x
    return out.to(device)


# ---- streams, norms, convolutions, activation --------------------------------------------------------------
@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("S,d", [(1, 100), (2, 136), (3, 1031), (4, 1024), (4, 4096), (6, 72), (3, 2052), (2, 5000)])
def test_streams_and_layer_norm(device, dtype, S, d):
    g = gen(S * d)
    x, y = torch.randn(5, S, d, generator=g) + 0.5, rnd(g, 5, d)
    mix, wo, wi, w = (torch.randn(*s, generator=g) for s in ((S, S), (S,), (S,), (d,)))
    dd = lambda t: t.to(device)
    want = R.streams_out(x.double().transpose(0, 1), y.double(), mix.double(), wo.double())
    read = R.layer_norm(R.streams_in(want, wi.double()), w.double(), 1e-3)
    xd = dd(x.clone())
    h = H.hyper_(xd, acts(y, device, dtype), dd(mix), dd(wo), dd(wi), dd(w), 1e-3, dtype)
    t = tol(dtype, 2e-6, 4e-3)
    assert rel(xd.transpose(0, 1), want) < 1e-6 and rel(h, read) < t
    idx = torch.tensor([4, 0, 4], device=device)                  # the model's final norm: plain sum, chosen rows
    assert rel(H.hyper_(xd, None, None, None, None, dd(w), 1e-3, dtype, idx=idx), R.layer_norm(want.sum(0), w.double(), 1e-3)[[4, 0, 4]]) < t
    xe = dd(x.clone())
    assert H.hyper_(xe, acts(y, device, dtype), dd(mix), dd(wo), None, None, 1e-3, dtype) is None and torch.equal(xe, xd)
    if device == "cuda" and dtype == BF16:
        acc = torch.zeros(5, round8(d), device=device)            # the decode GEMM's accumulator: consumed and left zero
        acc[:, :d] = dd(y).float()
        xf = dd(x.clone())
        hf = H.hyper_(xf, acc, dd(mix), dd(wo), dd(wi), dd(w), 1e-3, dtype, acc=True)
        assert torch.equal(xf, xd) and torch.equal(hf, h) and not acc.any()


@pytest.mark.parametrize("device,dtype", MODES)
def test_embedding_fills_every_stream(device, dtype):
    table = rnd(gen(1), 11, 36)
    ids = torch.tensor([3, 10, 0])
    x = H.embed_streams(ids.to(device), table.to(device, dtype), 3, 1.3)
    for s in range(3):
        assert rel(x[:, s], table.double()[ids] * 1.3) < 1e-6


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("d,taps", [(20, 3), (64, 4), (13, 1), (136, 2), (1032, 3), (40, 12)])
def test_input_convolution_over_portions(device, dtype, d, taps):
    """Inputs of earlier portions come from the state; portions shorter than the taps keep older ones. Steps of single rows take
    the form that is fused with the norm."""
    g = gen(d)
    cuts = [[1, 1, 1, 2, 30, 1, 3, 70], [40, 2, 2, 1, 1, 60], [3, 1, 1]]
    S, w, norm, wi = 2, rnd(g, d, taps), torch.rand(d, generator=g) + 0.5, torch.randn(2, generator=g)
    xs = [torch.randn(sum(c) + 5, S, d, generator=g) for c in cuts]
    dd = lambda t: t.to(device)
    want, wt = [], padded(w.t().float(), device)
    for x in xs:
        h = R.layer_norm(R.streams_in(x.double().transpose(0, 1), wi.double()), norm.double(), 1e-4)
        want.append(R.with_conv(h, w.double()))
    state = torch.full((len(cuts), taps - 1, d), 5.0, dtype=dtype, device=device)
    at, got = [0] * len(cuts), [[] for _ in cuts]

    def step(parts):
        live = sorted(parts, key=lambda s: not (parts[s] == 1 and at[s] > 0))
        nd = sum(parts[s] == 1 and at[s] > 0 for s in live)
        rows, _ = rows_for([(at[s], parts[s]) for s in live], nd, 16, device)
        rows.state = torch.tensor(live, dtype=torch.int32, device=device)
        x = dd(torch.cat([xs[s][at[s]:at[s] + parts[s]] for s in live]))
        single = nd == x.shape[0]
        h = H.hyper_(x, None, None, None, dd(wi), dd(norm), 1e-4, dtype, conv=(wt, state, rows) if single else None)
        h = h if single else H.canon(h, wt, state, rows)
        o = 0
        for s in live:
            got[s].append(h[o:o + parts[s]].cpu())
            o += parts[s]
            at[s] += parts[s]

    for i in range(max(map(len, cuts))):
        step({s: c[i] for s, c in enumerate(cuts) if i < len(c)})
    for parts in ({0: 1, 1: 1, 2: 1}, {1: 1}, {0: 1, 2: 1}, {0: 1, 1: 1}, {2: 1}, {0: 1}):
        step(parts)
    for s, (a, b) in enumerate(zip(got, want)):
        a = torch.cat(a)
        assert rel(a, b[:len(a)]) < tol(dtype, 3e-6, 6e-3), s


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("ff", [1, 61, 264, 2056, 8192])
def test_poly_norm(device, dtype, ff):
    g = gen(ff)
    z, coef = rnd(g, 7, ff) * 1.5, torch.tensor([0.7, -0.4, 0.9, 0.2])
    want = R.poly_norm(z.double(), coef.double(), 1e-4)
    h = H.poly_norm(acts(z, device, dtype), ff, coef.to(device), 1e-4, dtype)
    assert rel(h, want) < tol(dtype, 2e-6, 4e-3)
    if device == "cuda" and dtype == BF16:
        acc = torch.zeros(7, round8(ff), device=device)
        acc[:, :ff] = z.to(device).float()
        assert torch.equal(H.poly_norm(acc, ff, coef.to(device), 1e-4, dtype, acc=True), h) and not acc[:, :ff].any()


@pytest.mark.gpu
@pytest.mark.parametrize("T,split,tail", [(3, 64, 8), (200, 264, 16), (300, 64, 8), (1000, 136, 24)])
def test_projection_with_an_fp32_tail(T, split, tail):
    g = gen(T)
    a, w = rnd(g, T, 72).cuda(), (rnd(g, split + tail, 72) * 0.2).cuda()
    want = a.double().cpu() @ w.double().cpu().t()
    main, rest = H.linear_split(a, w, split)
    assert main.dtype == BF16 and rest.dtype == F32 and main.shape == (T, split) and rest.shape == (T, tail)
    assert rel(main, want[:, :split]) < 4e-3 and rel(rest, want[:, split:]) < 1e-5
    assert rel(H.linear_split(a, w, split)[1], want[:, split:]) < 1e-5      # the accumulator was left zero


# ---- latent attention --------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [pytest.param(F32, id="f32"), pytest.param(BF16, id="bf16")])
@pytest.mark.parametrize("T,heads,Kd,N", [(5, 3, 14, 44), (70, 2, 64, 72), (1, 5, 320, 128), (130, 4, 8, 8)])
@pytest.mark.parametrize("kn", [True, False])
@pytest.mark.gpu
def test_per_head_products(dtype, T, heads, Kd, N, kn):
    g = gen(T + N)
    ah, oh = round8(Kd) + 8, round8(N)
    a, b = rnd(g, T, heads, Kd), rnd(g, *((heads, Kd, N) if kn else (heads, N, Kd))) * 0.2
    ab = torch.full((T, heads, ah), 3.0, dtype=dtype)
    ab[..., :Kd] = a
    bb = torch.zeros(heads * (Kd if kn else N), round8(N if kn else Kd), dtype=dtype, device="cuda")[:, :N if kn else Kd]
    bb.copy_(b.flatten(0, 1))
    out = torch.full((T, heads * oh), 7.0, dtype=dtype, device="cuda")
    LA.head_gemm(ab.view(T, -1).cuda(), ah, bb, out, oh, heads, Kd, N, kn)
    want = torch.einsum("thk,hkn->thn" if kn else "thk,hnk->thn", a.double(), b.double())
    out = out.view(T, heads, oh)
    assert rel(out[..., :N], want) < tol(dtype, 1e-6, 4e-3) and bool((out[..., N:] == 7).all())


LATENT = [  # heads, dim, rot_dim, rotated, vdim, rank
    (3, 14, 10, 6, 18, 44), (2, 9, 5, 4, 7, 21), (6, 64, 64, 64, 128, 256), (3, 40, 24, 16, 72, 136), (20, 96, 48, 48, 136, 320), (35, 16, 16, 8, 24, 40),
    (1, 8, 8, 8, 8, 8), (4, 32, 32, 32, 64, 512), (2, 200, 56, 56, 24, 96), (17, 56, 16, 16, 64, 64)]


class LatentCase:
    """One latent attention layer with its cache: sequences of whole projections, fed in portions, beside the oracle."""

    def __init__(self, device, dtype, heads, dim, rot_dim, rotated, vdim, rank, lens, bs=16, seed=0, change=None):
        g = gen(heads * rank + seed)
        self.device, self.dtype, self.bs, self.lens = device, dtype, bs, lens
        self.m = m = LatentAttentionMixer(heads, dim, rot_dim, vdim, rank, 0.7 * (dim + rot_dim) ** -0.5, Rope(rotated, 3e3))
        self.sec = mixer_sections(m)
        lw = {"w_uk": rnd(g, heads * dim, rank) * rank ** -0.5, "w_uv": rnd(g, heads * vdim, rank) * rank ** -0.5, "sink": rnd(g, heads) + 3,
              "kv_norm": rnd(g, rank) * 0.2 + 1}
        self.p = {"uk": lw["w_uk"].double(), "uv": lw["w_uv"].double(), "sink": lw["sink"].double(), "dkv.norm": lw["kv_norm"].double()}
        cfg = LZ.LogozenConfig(hidden_size=8, vocab_size=8, norm_eps=1e-4, norm_one_plus=False, streams=1, canon=1, layers=[LZ.Layer(m)])
        w = LZ.StackWeights(cfg, device, dtype)
        for k, v in lw.items():
            w.layers[0][k][:v.shape[0]].copy_(v)
        w.finish()
        self.lw, self.w_expand = w.layers[0], w.derived[0].get("w_expand")
        self.q = [rnd(g, n, heads, dim + rot_dim) for n in lens]
        self.down = [rnd(g, n, rank + rot_dim) for n in lens]
        self.gate = [rnd(g, n, heads) for n in lens]
        if change:
            change(self)
        mm = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": m.scale, "rot": {"base": 3e3, "dims": rotated}}
        self.want = [R.latent_heads(q.double().flatten(1), d.double(), s.double(), self.p, mm, 1e-4) for q, d, s in zip(self.q, self.down, self.gate)]
        need = [-(-n // bs) for n in lens]
        perm = torch.randperm(sum(need) + 3, generator=g)
        self.tabs = torch.zeros(len(lens), max(need) + 1, dtype=torch.int32)
        o = 0
        for i, k in enumerate(need):
            self.tabs[i, :k] = perm[o:o + k]
            o += k
        self.cache = torch.full((sum(need) + 3, bs, 1, m.pitch), 9.0, dtype=dtype, device=device)       # leftovers of other sequences
        self.at, self.got = [0] * len(lens), [[] for _ in lens]
        self.tab_r = K.rope_tables(max(lens) + 1, rotated, 3e3, device)

    def step(self, parts, packed, acc=False):
        """parts: {sequence: next rows}; packed: prompt rows in the expanded form."""
        live = sorted(parts, key=lambda s: not (parts[s] == 1 and self.at[s] > 0))
        nd = sum(parts[s] == 1 and self.at[s] > 0 for s in live)
        rows, _ = rows_for([(self.at[s], parts[s]) for s in live], nd, self.bs, "cpu")
        rows.tables = self.tabs[live].contiguous()
        rows.slots = torch.tensor([int(rows.tables[i, p // self.bs]) * self.bs + p % self.bs for i, p in zip(rows.seq.tolist(), rows.pos.tolist())])
        pieces = pieces_for(rows, nd, self.device, self.bs) if packed and len(live) > nd else None
        rows = K.Rows(*[t.to(self.device) if torch.is_tensor(t) else t for t in vars(rows).values()])
        T, m = rows.pos.numel(), self.m
        proj = torch.zeros(T, self.sec.total)
        cut = lambda xs: torch.cat([xs[s][self.at[s]:self.at[s] + parts[s]].flatten(1) for s in live]).float()
        for k, xs in (("q", self.q), ("dkv", self.down), ("g", self.gate)):
            x = cut(xs)
            proj[:, self.sec[k]:self.sec[k] + x.shape[1]] = x
        proj = proj.to(self.device, F32 if acc else self.dtype)
        out = LA.latent_attention(proj, self.sec, m, self.lw, self.w_expand, 1e-4, rows, self.tab_r, self.cache, self.dtype, pieces, acc=acc)
        assert not acc or not proj.any()
        o = 0
        for s in live:
            self.got[s].append(out[o:o + parts[s]].cpu())
            o += parts[s]
            self.at[s] += parts[s]

    def check(self, t):
        for s, want in enumerate(self.want):
            got = torch.cat(self.got[s]).double()
            e = (got - want[:len(got)]).norm(dim=1) / want[:len(got)].square().sum(1).mean().sqrt()
            assert e.max() < t, (s, int(e.argmax()), float(e.max()))


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("shape", LATENT, ids=str)
@pytest.mark.parametrize("packed", [True, False])
def test_latent_attention_over_portions(device, dtype, shape, packed):
    """Absorbed and expanded forms, decode rows beside portions, portions around page borders."""
    c = LatentCase(device, dtype, *shape, [150, 75, 20, 33])
    for parts in ({0: 64, 1: 2, 2: 16}, {0: 1, 1: 15, 3: 31}, {2: 1, 0: 65, 1: 1}, {3: 2, 0: 1, 1: 1, 2: 1}, {0: 2, 1: 55}, {0: 1, 1: 1, 2: 1}, {0: 16}):
        c.step(parts, packed and device == "cuda" and dtype == BF16)
    if device == "cuda" and dtype == BF16:
        c.at[3], c.got[3] = 0, []                                 # the decode GEMM's accumulator
        c.step({3: 20}, packed, acc=True)
        c.step({3: 1}, packed, acc=True)
    c.check(tol(dtype, 1e-5, 2e-2))


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("key,query", [(0, 63), (0, 64), (63, 64), (64, 127), (15, 16), (16, 31), (5, 139), (138, 139), (139, 139), (0, 0), (1, 2)])
@pytest.mark.parametrize("shape", [(3, 14, 10, 6, 18, 44), (3, 40, 24, 16, 72, 136), (2, 96, 48, 32, 24, 64)], ids=str)
def test_one_key_stands_out(device, dtype, shape, key, query):
    """An unrotated coordinate of the shared key part makes one score far larger than the others; the key after the query must
    not be seen although it would win."""
    def spike(c):
        for x in (key, query + 1):
            if x < 140:
                c.down[0][x, -1] = 30
        c.q[0][query, :, -1] = 25
    n = 140
    for cuts in ([n], [query, 1, n - query - 1], [max(1, query - 5), 2 + query, n]):
        for packed in ([True, False] if device == "cuda" and dtype == BF16 else [False]):
            c = LatentCase(device, dtype, *shape, [n], change=spike)
            for x in cuts:
                if min(x, n - c.at[0]) > 0:
                    c.step({0: min(x, n - c.at[0])}, packed)
            c.check(tol(dtype, 1e-5, 4e-2))


@pytest.mark.gpu
@pytest.mark.parametrize("heads,rank,rot", [(16, 512, 64), (24, 192, 32), (33, 72, 16), (4, 128, 32)])
def test_decode_splits_of_the_absorbed_kernel(heads, rank, rot):
    g, bs, lens = gen(heads), 16, [(5, 1), (777, 1), (64, 1), (1023, 1), (0, 1)]
    rows, nb = rows_for(lens, 5, bs, "cuda")
    m = LatentAttentionMixer(heads, 8, rot, 8, rank, 0.5 * (rank + rot) ** -0.5)
    q, cache = rnd(g, 5, heads, m.pitch), rnd(g, nb, bs, 1, m.pitch)
    cache[..., rank:m.rot_at], cache[..., m.rot_at + rot:] = 0, 0
    sink, gate = torch.randn(heads, generator=g) + 4, torch.rand(5, heads, generator=g)
    want = torch.zeros(5, heads, rank, dtype=torch.float64)
    for i, (s, _) in enumerate(lens):
        j = torch.arange(s + 1)
        kv = cache.view(-1, m.pitch)[rows.tables[i].cpu()[j // bs].long() * bs + j % bs].double()
        sc = torch.cat([q[i].double() @ kv.t() * m.scale, sink.double()[:, None]], 1)
        want[i] = torch.softmax(sc, 1)[:, :-1] @ kv[:, :rank] * gate[i].double()[:, None]
    for splits in (1, 2, 5, 32, None):
        out = torch.full((5, heads * round16(rank)), 7.0, dtype=BF16, device="cuda")
        LA.latent_decode(q.view(5, -1).cuda(), m, rows, cache.cuda(), gate.cuda(), sink.cuda(), out, splits=splits)
        assert rel(out.view(5, heads, -1)[..., :rank], want) < 4e-3


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("heads,kv,dim,vdim", [(4, 2, 22, 18), (3, 3, 128, 72), (2, 1, 200, 136)])
def test_sinks_of_the_paged_attention(device, dtype, heads, kv, dim, vdim):
    """The general attention kernels take a sink per head too."""
    if device == "cpu":
        pytest.skip("kernels only")
    g, bs, lens, nd = gen(dim), 16, [(40, 1), (0, 1), (70, 1), (0, 75), (60, 9)], 3
    rows, nb = rows_for(lens, nd, bs, device)
    m = AttentionMixer(heads, kv, dim, vdim, dim ** -0.5)
    q, kc, vc = rnd(g, rows.pos.numel(), heads, dim), torch.zeros(nb, bs, kv, round8(dim), dtype=BF16), torch.zeros(nb, bs, kv, round8(vdim), dtype=BF16)
    kc[..., :dim], vc[..., :vdim] = rnd(g, nb, bs, kv, dim), rnd(g, nb, bs, kv, vdim)
    sink = torch.randn(heads, generator=g) + 3
    want = []
    for t in range(q.shape[0]):
        j = torch.arange(int(rows.pos[t]) + 1)
        sl = rows.tables.cpu()[int(rows.seq[t]), j // bs].long() * bs + j % bs
        k, v = (c.view(nb * bs, kv, -1)[sl].double().repeat_interleave(heads // kv, 1) for c in (kc, vc))
        sc = torch.cat([torch.einsum("hd,jhd->hj", q[t].double(), k[..., :dim]) * m.scale, sink.double()[:, None]], 1)
        want.append(torch.einsum("hj,jhd->hd", torch.softmax(sc, 1)[:, :-1], v[..., :vdim]).flatten())
    want = torch.stack(want)
    qb = torch.zeros(q.shape[0], heads, round8(dim), dtype=dtype)
    qb[..., :dim] = q
    qb, kc, vc, sink = qb.flatten(1).to(device), kc.to(device, dtype), vc.to(device, dtype), sink.to(device)
    out = K.act(q.shape[0], heads * vdim, dtype, device)
    K.attn_rows(qb, m, rows, kc, vc, None, out, sink=sink)
    assert rel(out, want) < tol(dtype, 1e-5, 4e-3)
    if dtype == BF16:
        for splits in (1, 3):
            out.zero_()
            K.attn_paged_decode(qb[:nd], m, rows, kc, vc, None, out, splits=splits, sink=sink)
            K.attn_paged_prefill(qb, m, rows, kc, vc, None, out, sink=sink)
            assert rel(out, want) < 4e-3


# ---- matrix memory -----------------------------------------------------------------------------------------
def _memory_case(device, dtype, heads, N, P, cuts, bias_i, bias_f, cap, seed=0, t=None):
    g = gen(N + P + seed)
    data, want = [], []
    for c in cuts:
        T = sum(c)
        # keys and queries that do not cancel in n . q, whose reciprocal would only magnify rounding; both signs of it
        q, k, v, z = rnd(g, T, heads, N) + 2, (rnd(g, T, heads, N) + 1) * 0.25, rnd(g, T, heads, P), rnd(g, T, 2 * heads).float() * 2
        q = q * torch.where(torch.rand(T, heads, 1, generator=g) < 0.5, -1, 1).to(BF16)
        data.append((q, k, v, z))
        zb = z.double() + torch.cat([bias_i, bias_f]).double()
        li, lf = R.soft_cap(zb[:, :heads], cap), R.log_sigmoid(R.soft_cap(zb[:, heads:], cap))
        want.append(R.matrix_memory(q.double() * N ** -0.5, k.double(), v.double(), li, lf))
    ssm = torch.full((len(cuts) + 1, heads, N, P), 3.0, device=device)     # slots hold leftovers
    vec = torch.full((len(cuts) + 1, heads, K.mlstm_vec(N, P)), 5.0, device=device)
    slot = list(range(len(cuts), 0, -1))
    at, got = [0] * len(cuts), [[] for _ in cuts]
    for i in range(max(map(len, cuts))):
        live = [s for s in range(len(cuts)) if i < len(cuts[s])]
        live.sort(key=lambda s: not (cuts[s][i] == 1 and at[s] > 0))
        nd = sum(cuts[s][i] == 1 and at[s] > 0 for s in live)
        rows, _ = rows_for([(at[s], cuts[s][i]) for s in live], nd, 16, device)
        rows.state = torch.tensor([slot[s] for s in live], dtype=torch.int32, device=device)
        q, k, v, z = (torch.cat([data[s][x][at[s]:at[s] + cuts[s][i]] for s in live]).flatten(1) for x in range(4))
        out = K.mlstm_scan(acts(q, device, dtype), acts(k, device, dtype), acts(v, device, dtype), acts(z, device, F32),
                           torch.cat([bias_i, bias_f]).to(device), cap, ssm, vec, rows, heads, N, P)
        o = 0
        for s in live:
            got[s].append(out[o:o + cuts[s][i]].cpu())
            o += cuts[s][i]
            at[s] += cuts[s][i]
    for a, b in zip(got, want):
        a = torch.cat(a).double().view(b.shape)
        e = (a - b).norm(dim=2) / b.square().sum(2).mean(0).sqrt()         # a head has its own size
        assert e.max() < (t or tol(dtype, 2e-5, 2e-2)), (int(e.argmax()), float(e.max()))
    assert bool((ssm[0] == 3).all()) and bool((vec[0] == 5).all())         # a slot nobody holds stays as it was


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("heads,N,P", [(4, 20, 12), (3, 72, 40), (2, 128, 96), (3, 256, 8), (1, 300, 4), (1, 8, 8), (5, 18, 70)])
@pytest.mark.parametrize("cap", [3.0, 15.0])
def test_matrix_memory_over_portions(device, dtype, heads, N, P, cap):
    """Long and short memories, heads whose gates stay below and above the running maximum's start, portions around the
    64-token chunk of the prompt kernel, states carried through slots."""
    cuts = [[64, 1, 1, 63, 17, 2], [130, 1, 40, 1], [1, 1, 2, 65]]
    _memory_case(device, dtype, heads, N, P, cuts, torch.linspace(-5, 9, heads), torch.linspace(9, -4, heads), cap)


@pytest.mark.parametrize("device,dtype", MODES)
def test_long_memory(device, dtype):
    """Open forget gates over many tokens, half of them decoded one by one: rounding must not add up."""
    _memory_case(device, dtype, 2, 16, 8, [[300] + [1] * 200], torch.tensor([-2.0, 3.0]), torch.tensor([11.0, 14.0]), 15.0, t=tol(dtype, 5e-5, 3e-2))


def test_the_running_maximum_and_the_floor_matter():
    """The oracle's own details show in its outputs: the maximum's start, the floor under the normaliser."""
    g = gen(5)
    q, k, v = (torch.randn(40, 1, 8, generator=g, dtype=torch.float64) for _ in range(3))
    li, lf = torch.full((40, 1), -6.0, dtype=torch.float64), torch.full((40, 1), -0.1, dtype=torch.float64)
    a = R.matrix_memory(q, k, v, li, lf)
    b = R.matrix_memory(q, k, v, li + 6, lf)                     # the same memory in a larger unit: not the same output
    assert float((a - b).norm() / b.norm()) > 0.5


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("heads,vdim", [(3, 10), (4, 64), (1, 256), (5, 24), (2, 264), (2, 520)])
def test_unit_heads_and_gate(device, dtype, heads, vdim):
    g, n = gen(vdim), heads * vdim
    y, z, w = rnd(g, 6, n), rnd(g, 6, n), rnd(g, n)
    y[:, :vdim] *= 8
    yd = y.double().view(6, heads, vdim)
    want = (yd / R.root_mean_square(yd, 1e-5)).view(6, n) * w.double() * torch.sigmoid(z.double())
    got = K.gated_norm(acts(y, device, dtype), acts(z, device, dtype), w.float().to(device), 1e-5, heads, False)
    assert rel(got, want) < tol(dtype, 2e-6, 4e-3)


# ---- whole models through the engine -----------------------------------------------------------------------
WHOLE = [pytest.param("cpu", F32, 5e-5, id="cpu"), pytest.param("cuda", F32, 5e-5, marks=GPU, id="gpu-f32"),
         pytest.param("cuda", BF16, 0.07, marks=GPU, id="gpu-bf16")]
LENS = [(171, 1), (97, 2), (1, 3), (40, 4), (130, 5)]
NAMES = list(CONFIGS)


@pytest.mark.parametrize("device,dtype,t", WHOLE)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_alone_and_together(name, device, dtype, t):
    eng = ZOO.engine(name, device, dtype)
    rp = ZOO.replay(name, eng)
    for key in LENS:
        rp.step({key: key[0]})
    ZOO.check(name, rp, t)
    rp2 = ZOO.replay(name, eng)
    rp2.step({k: k[0] for k in LENS[:4]})
    ZOO.check(name, rp2, t)
    assert eng.blocks.num_free == eng.blocks.num_blocks and (eng.slots is None or len(eng.slots.free) == 4)


@pytest.mark.parametrize("device,dtype,t", WHOLE)
@pytest.mark.parametrize("name", NAMES)
def test_decoding_matches_prefill(name, device, dtype, t):
    """Token by token from the start and after a long prompt."""
    rp = ZOO.replay(name, ZOO.engine(name, device, dtype))
    for _ in range(97):
        rp.step({(97, 2): 1})
    rp.step({(171, 1): 140})
    for _ in range(31):
        rp.step({(171, 1): 1})
    ZOO.check(name, rp, t)


@pytest.mark.parametrize("device,dtype,t", WHOLE)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("sizes", [(2,), (3, 16, 64), (65, 80, 2, 1), (70,)], ids=str)
def test_portions(name, device, dtype, t, sizes):
    rp = ZOO.replay(name, ZOO.engine(name, device, dtype))
    for c in random_portions(171, random.Random(len(sizes)), sizes):
        rp.step({(171, 1): c})
    ZOO.check(name, rp, t)


@pytest.mark.parametrize("device,dtype,t", WHOLE)
@pytest.mark.parametrize("name", NAMES)
def test_mixed_batches_with_pages_and_slots_used_again(name, device, dtype, t):
    """More requests than slots, a pool that only just holds the live ones: everything is handed out several times."""
    eng = ZOO.engine(name, device, dtype, num_blocks=34)
    rp = ZOO.replay(name, eng)
    for st in mixed_schedule(LENS + [(97, 6), (171, 7), (23, 8), (64, 9)], random.Random(5), (2, 3, 16, 29, 64, 70)):
        rp.step(st)
    ZOO.check(name, rp, t)
    assert eng.blocks.num_free == 34


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["wide", "tall"])
def test_absorbed_and_expanded_prompts_agree(name):
    out = []
    for pack in (True, False):
        eng = ZOO.engine(name, "cuda", BF16)
        eng.runner.pack_prompts = pack
        rp = ZOO.replay(name, eng)
        for c in (100, 71):
            rp.step({(171, 1): c, (172, 2): c})
        out.append(torch.cat([rp.logits((171, 1)), rp.logits((172, 2))]))
    e = row_errors(out[0], out[1].double())
    assert e.mean() < 0.03 and int((e > 0.1).sum()) <= 0.02 * len(e) and e.max() < 0.3, e.sort().values[-8:]


@pytest.mark.gpu
def test_long_prompt_and_long_decoding():
    """Beyond the decode kernels' splits and several prompt tiles, portions on top of a long cache."""
    name, n = "wide", 900
    rp = ZOO.replay(name, ZOO.engine(name, "cuda", BF16, num_blocks=80, max_len=1024))
    for c in [600, 100, 2] + [1] * 100 + [98]:
        rp.step({(n, 3): c})
    ZOO.check(name, rp, 0.07)


def _with(st, **edits):
    out = dict(st)
    for k, f in edits.items():
        out[k.replace("__", ".")] = f(out[k.replace("__", ".")])
    return out


MISTAKES = {
    "rotation base": lambda d, w: (d["layers"][0]["mixer"]["rot"].update(base=2e4), w)[1],
    "rotated dims": lambda d, w: (d["layers"][0]["mixer"]["rot"].update(dims=8), w)[1],
    "score scale": lambda d, w: (d["layers"][2]["mixer"].update(scale=0.38), w)[1],
    "gate cap": lambda d, w: (d["layers"][1]["mixer"].update(gate_cap=7.0), w)[1],
    "embedding scale": lambda d, w: (d["embedding"].update(scale=1.6), w)[1],
    "no sink": lambda d, w: _with(w, l2__mix__sink=lambda t: t - 1e4),
    "mix transposed": lambda d, w: _with(w, l1__hc2__mix=lambda t: t.t()),
    "taps reversed": lambda d, w: _with(w, l3__canon1=lambda t: t.flip(1)),
    "powers exchanged": lambda d, w: _with(w, l0__mlp__act=lambda t: t[[0, 2, 1, 3]]),
    "gates exchanged": lambda d, w: {**w, "l3.mix.i.b": w["l3.mix.f.b"], "l3.mix.f.b": w["l3.mix.i.b"]},
}


@pytest.mark.parametrize("what", list(MISTAKES))
def test_a_mistake_shows(what):
    """The comparisons above can fail: the oracle with one detail off is hundreds of fp32 tolerances away."""
    d, _, _, w = ZOO.model("odd")
    d = copy.deepcopy(d)
    bad = R.forward(d, MISTAKES[what](d, w), ZOO.tokens("odd", 171, 1))
    assert row_errors(bad, ZOO.oracle("odd", 171, 1)).max() > 0.01


def test_streams_after_every_layer():
    d, _, _, w = ZOO.model("odd")
    eng = ZOO.engine("odd", "cpu", F32)
    eng.runner.trace = []
    ZOO.replay("odd", eng).step({(40, 4): 40})
    want = []
    R.forward(d, w, ZOO.tokens("odd", 40, 4), want)
    assert len(want) == len(eng.runner.trace) == len(d["layers"])
    for a, b in zip(eng.runner.trace, want):
        assert rel(a, b) < 1e-5


# ---- generation through the scheduler ----------------------------------------------------------------------
@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=GPU)])
@pytest.mark.parametrize("kw", [dict(), dict(prefill_chunk=7), dict(mixed_batches=False), dict(async_scheduling=False)], ids=str)
def test_greedy_generation(device, kw):
    ZOO.check_generation("odd", device, **kw)


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=GPU)])
def test_greedy_generation_with_preemption(device):
    assert ZOO.check_generation("ones", device, num_blocks=6, max_len=128).sched.num_preemptions > 0


@pytest.mark.gpu
def test_bf16_generation_uses_graphs_and_matches_replay():
    """Each generated token is the argmax of the logits that replaying the same tokens gives, up to ties within the rounding of
    the two schedules."""
    from dlti_b200.serve.params import Request, SamplingParams
    eng = ZOO.engine("wide", "cuda", BF16)
    prompts = [ZOO.tokens("wide", n, 40 + n) for n in (90, 7, 130)]
    n0 = _lib.launch_count()
    outs = eng.generate(prompts, SamplingParams(max_tokens=40, temperature=0.0, ignore_eos=True))
    assert eng.graphs and _lib.launch_count() > n0
    for p, o in zip(prompts, outs):
        seq = p + o["token_ids"]
        lg = eng.replay_step([(r := Request("x", [], SamplingParams()), seq[:-1], list(range(len(p) - 1, len(seq) - 1)))])
        eng.replay_end(r)
        gap = lg.max(1).values - lg[torch.arange(40), torch.tensor(o["token_ids"])]
        assert gap.max() < 0.15 * lg.std()


def test_sampling_parameters_reach_the_sampler():
    from dlti_b200.serve.params import SamplingParams
    eng = ZOO.engine("ones", "cpu", F32)
    sp = SamplingParams(max_tokens=12, temperature=1.0, top_k=5, seed=7, ignore_eos=True)
    a, b = (eng.generate([ZOO.tokens("ones", 9, 1)], sp)[0]["token_ids"] for _ in range(2))
    c = eng.generate([ZOO.tokens("ones", 9, 1)], SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True))[0]["token_ids"]
    assert a == b and a != c


# ---- configuration, loading, command line ------------------------------------------------------------------
def test_registry_config_and_checkpoint_round_trip(tmp_path):
    from dlti_b200.models.config import resolve_config
    from dlti_b200.models.registry import family_of
    d, cfg, st, _ = ZOO.model("odd")
    LZ.save_checkpoint(cfg, st, tmp_path)
    c = resolve_config(str(tmp_path))
    assert isinstance(c, LZ.LogozenConfig) and c.layers == cfg.layers and json.load(open(tmp_path / "config.json")) == d
    fam = family_of(c)
    assert fam.name == "Logozen"
    w = fam.load_weights(c, tmp_path, "cpu", F32)
    assert {n for n, _ in LZ.named_tensors(w)} == set(st)
    for name, dst in LZ.named_tensors(w):
        assert torch.equal(dst, st[name].float()), name
    assert c.num_params() >= sum(t.numel() for t in st.values())
    for p in ("logozen-tiny", "logozen-1b"):
        assert isinstance(resolve_config(p), LZ.LogozenConfig)
    assert family_of(resolve_config("sigosun-tiny")).name == "Sigosun"


@pytest.mark.parametrize("edit,msg", [(lambda d: d["layers"][0]["mixer"]["rot"].update(dims=7), "rotary"),
                                      (lambda d: d["layers"][0]["mixer"]["rot"].update(dims=12), "rotary"),
                                      (lambda d: d["layers"][1]["mixer"].update(gate_cap=0), "gate_cap"),
                                      (lambda d: d["canon"].update(taps=0), "taps"), (lambda d: d["layers"][1].update(type="conv"), "mixer type"),
                                      (lambda d: d["layers"][0]["mlp"].update(kind="sparse"), "feed-forward")])
def test_inconsistent_configurations_are_refused(edit, msg):
    d = copy.deepcopy(CONFIGS["odd"])
    edit(d)
    with pytest.raises(ValueError, match=msg):
        LZ.LogozenConfig.from_dict(d)


def test_misfitting_tensors_and_prefix_caching_are_refused():
    _, cfg, st, _ = ZOO.model("odd")
    with pytest.raises(ValueError, match="l0.mix.dkv"):
        LZ.from_state(cfg, {**st, "l0.mix.dkv": st["l0.mix.dkv"][:-1]}, "cpu", F32)
    with pytest.raises(ValueError, match="l1.canon2"):
        LZ.from_state(cfg, {**st, "l1.canon2": st["l1.canon2"][:, :-1]}, "cpu", F32)
    with pytest.raises(ValueError, match="prefix caching"):
        ZOO.engine("odd", "cpu", F32, enable_prefix_caching=True)


def test_cache_holds_latents_and_states_only():
    """One row per token and attention layer for all heads; matrices, normalisers and convolution inputs per slot."""
    eng = ZOO.engine("wide", "cpu", F32)
    for l, k, v, ssm, canon in zip(eng.cfg.layers, eng.kv.k, eng.kv.v, eng.states.ssm, eng.states.canon):
        att = isinstance(l.mixer, LatentAttentionMixer)
        assert (k is not None) == att and (ssm is None) == att and canon.shape[0] == (1 if l.mlp is None else 2)
        if att:
            assert k.shape[2:] == (1, round16(l.mixer.kv_rank) + round16(l.mixer.rot_dim) + 8) and v.numel() == 0


@pytest.mark.parametrize("device,dtype,t", WHOLE)
def test_trace_run_command(tmp_path, device, dtype, t):
    name = "odd"
    _, cfg, st, _ = ZOO.model(name)
    LZ.save_checkpoint(cfg, st, tmp_path / "m")
    a, b = ZOO.tokens(name, 97, 2), ZOO.tokens(name, 40, 4)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [49, 3]}, {"id": "b", "tokens": b[:39], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[39:], "want": [0]}, {"id": "a", "tokens": a[50:90], "want": [0, 39]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[90:91], "want": []}], "end": []},
             {"step": 7, "entries": [{"id": "a", "tokens": a[91:92], "want": [0]}, {"id": "b", "tokens": b[:1], "want": [0]}], "end": ["a", "b"]}]
    args = [os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "bfloat16" if dtype == BF16 else "float32",
            "--out", str(tmp_path / "o"), "--max-tokens", "192", "--device", device]
    p = subprocess.run([sys.executable] + args, input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2", "done 7"]
    read = lambda s: torch.from_numpy(np.fromfile(tmp_path / "o" / f"{s}.f32", dtype="<f4").reshape(-1, cfg.vocab_size))
    wa, wb = ZOO.oracle(name, 97, 2), ZOO.oracle(name, 40, 4)
    for s, want in ((0, wa[[49, 3]]), (1, torch.stack([wb[39], wa[50], wa[89]])), (7, torch.stack([wa[91], wb[0]]))):
        assert row_errors(read(s), want).max() < t
    assert not (tmp_path / "o" / "2.f32").exists()
