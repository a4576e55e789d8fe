"""Latanex against its plain implementation (tests/ref_latanex.py): each mechanism alone, then whole models through the
engine in every kind of schedule. CPU runs use the ops' PyTorch restatements, GPU runs the kernels."""
import copy
import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

from dlti_b200.models import latanex as LX
from dlti_b200.models.stack import AttentionMixer, DeltaMixer, MoeMlp, mixer_sections, mlp_sections, round8
from dlti_b200.ops import _lib
from dlti_b200.ops import delta as D
from dlti_b200.ops import dyt as N
from dlti_b200.ops import moe as M
from dlti_b200.ops import stack as K
from dlti_b200.serve.engine import _pieces, chunk_pieces
from tests import ref_latanex as R
from tests.latanex_util import CONFIGS, ZOO, choice_margin
from tests.stack_util import mixed_schedule, random_portions, row_errors, rows_for

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


def accumulator(x):
    """x as the decode GEMM's fp32 accumulator."""
    out = torch.zeros(x.shape[0], round8(x.shape[1]), device="cuda")
    out[:, :x.shape[1]] = x
    return out


# ---- norms and residual ------------------------------------------------------------------------------------
def _norm(g, d):
    return torch.rand(1, generator=g) + 0.3, torch.randn(d, generator=g), torch.randn(d, generator=g)


def _dd(n, device=None):
    return tuple(t.double() if device is None else t.to(device) for t in n)


def _ref_norm(x, n):
    return R.dynamic_tanh(x, n[0].double(), n[1].double(), n[2].double())


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("T,d", [(5, 100), (1, 8), (3, 1031), (700, 2048), (9, 4096), (130, 2052)])
def test_norms_between_sublayers(device, dtype, T, d):
    g = gen(T * d)
    x, y, post, pre = torch.randn(T, d, generator=g) * 3, rnd(g, T, d), _norm(g, d), _norm(g, d)
    want = x.double() + _ref_norm(y.double(), post)
    t = tol(dtype, 2e-6, 4e-3)
    xd = x.clone().to(device)
    h = N.tanh_between_(xd, acts(y, device, dtype), _dd(post, device), _dd(pre, device), dtype)
    assert rel(xd, want) < tol(dtype, 1e-6, 3e-6) and rel(h, _ref_norm(want, pre)) < t
    idx = torch.tensor([T - 1, 0, T // 2], device=device)
    assert rel(N.tanh_rows(xd, idx, _dd(pre, device), dtype), _ref_norm(want, pre)[idx.cpu()]) < t
    assert N.tanh_between_(xd, acts(y, device, dtype), _dd(post, device), None, dtype) is None
    if device == "cuda" and dtype == BF16:
        acc = accumulator(y.cuda().float())
        xf = x.clone().to(device)
        hf = N.tanh_between_(xf, acc, _dd(post, device), _dd(pre, device), dtype, acc=True)
        assert rel(xf, want) < 3e-6 and torch.equal(hf, h) and not acc.any()


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("T,d,top,shared", [(5, 100, 3, True), (4, 256, 1, False), (600, 512, 7, True), (3, 33, 40, False)])
def test_expert_outputs_are_added_up(device, dtype, T, d, top, shared):
    g = gen(T + d)
    x, rows, w, y, post, pre = torch.randn(T, d, generator=g), rnd(g, T * top, d), torch.randn(T, top, generator=g), rnd(g, T, d), _norm(g, d), _norm(g, d)
    sum_ = (rows.double().view(T, top, d) * w.double()[:, :, None]).sum(1) + (y.double() if shared else 0)
    want = x.double() + _ref_norm(sum_, post)
    xd, counts = x.clone().to(device), torch.full((37,), 5, dtype=torch.int32, device=device)
    e = M.ExpertSum(acts(rows, device, dtype), w.to(device), acts(y, device, dtype) if shared else None, counts)
    h = N.tanh_between_(xd, e, _dd(post, device), _dd(pre, device), dtype)
    assert rel(xd, want) < 4e-6 and rel(h, _ref_norm(want, pre)) < tol(dtype, 4e-6, 4e-3)
    assert device == "cpu" or not counts.any()
    if device == "cuda" and dtype == BF16 and shared:
        xf, acc = x.clone().to(device), accumulator(y.cuda().float())
        hf = N.tanh_between_(xf, M.ExpertSum(e.rows, e.weights, acc, counts), _dd(post, device), _dd(pre, device), dtype, acc=True)
        assert torch.equal(xf, xd) and torch.equal(hf, h) and not acc.any()


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("d", [36, 1024, 1030])
def test_embedding_and_its_norm(device, dtype, d):
    g = gen(d)
    table, n, ids = rnd(g, 11, d), _norm(g, d), torch.tensor([3, 10, 0])
    x, h = N.embed_tanh(ids.to(device), table.to(device, dtype), 1.3, _dd(n, device), dtype)
    want = table.double()[ids] * 1.3
    assert rel(x, want) < 1e-6 and rel(h, _ref_norm(want, n)) < tol(dtype, 2e-6, 4e-3)


# ---- attention ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("H,G,dim,vdim", [(6, 3, 14, 10), (8, 2, 64, 128), (1, 1, 8, 8), (4, 4, 33, 7), (16, 4, 128, 128), (5, 1, 40, 264)])
def test_whole_row_norm_bias_and_value_mixing(device, dtype, H, G, dim, vdim):
    g, bs = gen(H * dim + vdim), 16
    m = AttentionMixer(H, G, dim, vdim, 1.0, qk_norm=False, head_gate=False, bias=True, row_norm=True, v_mix=True)
    sec = mixer_sections(m)
    rows, nb = rows_for([(17, 1), (0, 9), (30, 4)], 1, bs, device)
    T = rows.pos.numel()
    rows.slots[3] = -1                                            # a row that is not cached
    proj = torch.zeros(T, sec.total)
    lw = {"b_in": torch.zeros(sec.total), "q_norm": torch.randn(H * dim, generator=g), "k_norm": torch.randn(G * dim, generator=g),
          "v_mix": torch.tensor([0.3])}
    for s, (o, n) in sec.at.items():
        proj[:, o:o + n], lw["b_in"][o:o + n] = rnd(g, T, n).float() * 2, torch.randn(n, generator=g)
    first = rnd(g, T, G * vdim)
    cut = lambda s: (proj + lw["b_in"]).double()[:, sec[s]:sec[s] + sec.at[s][1]]
    q, k, v = (cut(s) for s in "qkv")
    q, k = R.whole_norm(q, lw["q_norm"].double(), 1e-4), R.whole_norm(k, lw["k_norm"].double(), 1e-4)
    t = tol(dtype, 2e-6, 4e-3)
    lwd = {n: x.to(device) for n, x in lw.items()}
    for have in (None, first):
        mixed = v if have is None else R.mix_values(v, first.double(), 0.3)
        for acc in ((False, True) if device == "cuda" and dtype == BF16 else (False,)):
            kc = torch.full((nb, bs, G, round8(dim)), 9.0, dtype=dtype, device=device)
            vc = torch.full((nb, bs, G, round8(vdim)), 9.0, dtype=dtype, device=device)
            p = accumulator(proj.cuda()) if acc else acts(proj, device, dtype)
            got, own = K.qkv_rows(p, sec, m, lwd, 1e-4, rows, None if have is None else acts(first, device, dtype), kc, vc, dtype, acc=acc)
            assert not acc or not p.any()
            assert rel(got.reshape(T, H, -1)[..., :dim].flatten(1), q) < t
            assert (own is None) == (have is not None) and (own is None or rel(own, v) < t)
            ok = rows.slots >= 0
            assert rel(kc.view(-1, G, round8(dim))[rows.slots[ok], :, :dim].flatten(1), k[ok.cpu()]) < t
            assert rel(vc.view(-1, G, round8(vdim))[rows.slots[ok], :, :vdim].flatten(1), mixed[ok.cpu()]) < t
            assert int((kc == 9).all(-1).sum()) >= (nb * bs - int(ok.sum())) * G          # nothing else was written


class AttentionCase:
    """One attention layer with its cache: sequences of given q, k, v, fed in portions, beside the oracle."""

    def __init__(self, device, dtype, H, G, dim, vdim, window, cap, lens, bs=16, seed=0, change=None):
        g = gen(H * dim + window + seed)
        self.device, self.dtype, self.bs, self.lens = device, dtype, bs, lens
        self.m = m = AttentionMixer(H, G, dim, vdim, 1.5 * dim ** -0.5, qk_norm=False, head_gate=False, window=window, softcap=cap, sink=True)
        self.sec = mixer_sections(m)
        self.q, self.k, self.v = ([rnd(g, n, h, x) for n in lens] for h, x in ((H, dim), (G, dim), (G, vdim)))
        self.sink = torch.randn(H, generator=g) + 1
        if change:
            change(self)
        self.want = [R.attend(*(x[i].double() for x in (self.q, self.k, self.v)), m.scale, cap, window, self.sink.double()).flatten(1)
                     for i in range(len(lens))]
        need = [-(-n // bs) for n in lens]
        perm, o = torch.randperm(sum(need) + 3, generator=g), 0
        self.tabs = torch.zeros(len(lens), max(need) + 1, dtype=torch.int32)
        for i, x in enumerate(need):
            self.tabs[i, :x] = perm[o:o + x]
            o += x
        new = lambda n: torch.full((sum(need) + 3, bs, G, round8(n)), 9.0, dtype=dtype, device=device)      # leftovers of other sequences
        self.kc, self.vc = new(dim), new(vdim)
        self.at, self.got = [0] * len(lens), [[] for _ in lens]

    def step(self, parts, packed=False):
        """parts: {sequence: next rows}; packed: prompt rows through the varlen kernel."""
        live = sorted(parts, key=lambda s: not (parts[s] == 1 and self.at[s] > 0))
        nd = sum(parts[s] == 1 and self.at[s] > 0 for s in live)
        rows, _ = rows_for([(self.at[s], parts[s]) for s in live], nd, self.bs, "cpu")
        rows.tables = self.tabs[live].contiguous()
        rows.slots = torch.tensor([int(rows.tables[i, p // self.bs]) * self.bs + p % self.bs for i, p in zip(rows.seq.tolist(), rows.pos.tolist())])
        pieces = None
        if packed and len(live) > nd:
            import dlti_b200.serve.engine as E
            keep, E.PACK_FROM = E.PACK_FROM, 1
            arr, n, longest, ext, prefix = chunk_pieces(rows.cu.tolist(), [self.at[s] for s in live[nd:]], rows.tables.tolist()[nd:], self.bs, 0,
                                                        1 << 30, self.m.window)
            E.PACK_FROM = keep
            pieces = _pieces(torch.from_numpy(arr).to(self.device), int(rows.cu[-1]), n, longest, ext, prefix)
        rows = K.Rows(*[t.to(self.device) if torch.is_tensor(t) else t for t in vars(rows).values()])
        T, m = rows.pos.numel(), self.m
        proj = torch.zeros(T, self.sec.total, dtype=self.dtype)
        for s, xs in (("q", self.q), ("k", self.k), ("v", self.v)):
            x = torch.cat([xs[i][self.at[i]:self.at[i] + parts[i]].flatten(1) for i in live])
            proj[:, self.sec[s]:self.sec[s] + x.shape[1]] = x
        q, _ = K.qkv_rows(proj.to(self.device), self.sec, m, {}, 0.0, rows, None, self.kc, self.vc, self.dtype, packed=pieces)
        sink = self.sink.to(self.device)
        if pieces is not None:
            out = K.packed_attention(q, m, rows, pieces, self.kc, self.vc, None, sink=sink)
        else:
            out = K.paged_attention(q, m, rows, self.kc, self.vc, None, sink=sink)
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


SHAPES = [(6, 3, 14, 10), (8, 2, 64, 128), (3, 3, 40, 72), (4, 1, 136, 24), (20, 1, 33, 8), (2, 1, 264, 40)]
REACH = [(0, 0.0), (1, 3.0), (15, 0.0), (16, 8.0), (17, 30.0), (64, 2.0), (65, 0.0), (127, 4.0), (128, 9.0), (129, 5.0), (400, 6.0)]


def _packs(device, dtype, dim, vdim):
    return [False, True] if device == "cuda" and dtype == BF16 and max(dim, vdim) <= 128 and vdim % 8 == 0 else [False]


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("window,cap", REACH)
def test_attention_over_portions(device, dtype, shape, window, cap):
    """Windows, caps and sinks; decode rows beside portions, portions around page borders and window edges."""
    for packed in _packs(device, dtype, *shape[2:]):
        c = AttentionCase(device, dtype, *shape, window, cap, [170, 75, 20, 33])
        for parts in ({0: 64, 1: 2, 2: 16}, {0: 1, 1: 15, 3: 31}, {2: 1, 0: 65, 1: 1}, {3: 2, 0: 1, 1: 1, 2: 1}, {0: 2, 1: 55}, {0: 1, 1: 1, 2: 1}, {0: 36}):
            c.step(parts, packed)
        c.check(tol(dtype, 1e-5, 1.5e-2))


@pytest.mark.gpu
@pytest.mark.parametrize("window", [1, 50, 100, 128, 129, 200, 256, 257, 300, 640, 0])
@pytest.mark.parametrize("cap", [0.0, 7.0])
def test_window_tiles_of_the_prompt_kernel(window, cap):
    """Several tiles of 128 rows, whole prompts and portions on top of cached rows."""
    for cuts in ([600], [130, 300, 170]):
        c = AttentionCase("cuda", BF16, 4, 2, 64, 64, window, cap, [600, 385])
        at = 0
        for x in cuts:
            c.step({0: x, 1: min(x, 385 - c.at[1])} if c.at[1] < 385 and min(x, 385 - c.at[1]) > 1 else {0: x}, packed=True)
            at += x
        c.check(1.5e-2)


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("window", [16, 40, 63, 64, 65, 129])
@pytest.mark.parametrize("shape", [(6, 3, 14, 10), (4, 2, 64, 128)], ids=str)
def test_one_key_stands_out(device, dtype, window, shape):
    """Keys far larger than the others just inside and just outside the window of one query, and right after the query: in prompts,
    portions and decoding."""
    n = 200
    for query in (window - 1, window, 130, 144, 199):
        def spike(c):
            for h in range(shape[0]):
                c.q[0][query, h] = 2
            for x in (query - window, query - window + 1, query + 1):
                if 0 <= x < n:
                    c.k[0][x] = 2.5 if x != query - window + 1 else 2
        for cuts in ([n], [query, 1, n], [max(1, query - 5), 7, n], [max(1, query - 70), n]):
            for packed in _packs(device, dtype, *shape[2:]):
                c = AttentionCase(device, dtype, *shape, window, 25.0, [n], change=spike)
                for x in cuts:
                    if min(x, n - c.at[0]) > 0:
                        c.step({0: min(x, n - c.at[0])}, packed)
                c.check(tol(dtype, 2e-5, 4e-2))


@pytest.mark.gpu
@pytest.mark.parametrize("window", [0, 40, 700])
def test_decode_splits(window):
    g, bs, lens, H, G, dim = gen(window), 16, [(5, 1), (777, 1), (64, 1), (1023, 1), (0, 1)], 8, 2, 72
    rows, nb = rows_for(lens, 5, bs, "cuda")
    m = AttentionMixer(H, G, dim, dim, dim ** -0.5, window=window, softcap=5.0)
    q, kc, vc, sink = rnd(g, 5, H, dim), rnd(g, nb, bs, G, dim), rnd(g, nb, bs, G, dim), torch.randn(H, generator=g)
    want = []
    for i, (s, _) in enumerate(lens):
        j = torch.arange(s + 1)
        sl = rows.tables[i].cpu()[j // bs].long() * bs + j % bs
        k, v = (c.view(-1, G, dim)[sl].double() for c in (kc, vc))
        qq = torch.zeros(s + 1, H, dim, dtype=torch.double)
        qq[-1] = q[i].double()
        want.append(R.attend(qq, k, v, m.scale, 5.0, window, sink.double())[-1].flatten())
    for splits in (1, 2, 5, 32, None):
        out = torch.full((5, H * dim), 7.0, dtype=BF16, device="cuda")
        K.attn_paged_decode(q.flatten(1).cuda(), m, rows, kc.cuda(), vc.cuda(), None, out, splits=splits, sink=sink.cuda())
        assert rel(out, torch.stack(want)) < 4e-3


# ---- feed-forwards -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("T,ff,limit", [(5, 61, 0.0), (300, 128, 0.0), (3, 264, 0.7), (700, 37, 1.5), (2, 2056, 2.0), (2000, 1024, 0.0)])
def test_gated_activations(device, dtype, T, ff, limit):
    g, d = gen(ff), 72
    h, w = rnd(g, T, d), rnd(g, 2, ff, d) * 0.2
    merged = torch.zeros(2 * round8(ff), d, dtype=dtype, device=device)
    merged[:ff], merged[round8(ff):round8(ff) + ff] = w[0], w[1]
    p = {"gate": w[0].double(), "up": w[1].double(), "down": torch.eye(ff, dtype=torch.double)}
    want = R.clipped_expert(h.double(), p, "", limit) if limit else R.swiglu(h.double(), p)
    hd = acts(h, device, dtype)
    if not limit:
        assert rel(M.swiglu(hd, merged, ff, dtype), want) < tol(dtype, 3e-6, 8e-3)
    z = K.linear(hd, merged)
    assert rel(M.gated_act(z, 0, round8(ff), ff, limit, dtype), want) < tol(dtype, 3e-6, 8e-3)
    if device == "cuda" and dtype == BF16 and T <= 256:
        from dlti_b200.ops.gemm import gemm_skinny_acc
        acc = gemm_skinny_acc(hd, merged)
        assert rel(M.gated_act(acc, 0, round8(ff), ff, limit, dtype, acc=True), want) < 8e-3 and not acc.any()


ROUTERS = [(10, 3, 5, 2, 1.7), (8, 2, 1, 1, 1.0), (12, 4, 3, 2, 2.5), (64, 8, 8, 4, 2.5), (1, 1, 1, 1, 0.5), (6, 6, 3, 3, 1.0), (256, 33, 16, 5, 1.0),
           (7, 3, 7, 4, 1.0), (100, 1, 2, 1, 3.0)]


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=GPU)])
@pytest.mark.parametrize("E,top,groups,keep,scale", ROUTERS)
def test_routing(device, E, top, groups, keep, scale):
    """Groups by their two best, corrections that make choice scores negative, weights without the correction."""
    g, T = gen(E + top), 75
    e = MoeMlp(E, top, 8, 1.0, groups, keep, scale)
    z, corr = torch.randn(T, E, generator=g) * 2, torch.randn(E, generator=g) - 1
    cfg = {"groups": {"count": groups, "keep": keep}, "top": top}
    clear = choice_margin(z.double(), corr.double(), cfg) > 1e-5
    assert clear.float().mean() > 0.9
    if device == "cpu":
        idx, w = M.route_ref(z, corr, e)
    else:
        wide = torch.full((T, E + 11), 7.0, device="cuda")
        wide[:, 5:5 + E] = z
        w, lists, counts = M._route(None, wide, 5, corr.cuda(), e)
        assert int(counts.sum()) == T * top
        idx = torch.full((T * top,), -1)
        for j in range(E):
            idx[lists[j, :int(counts[j])].long().cpu()] = j
        counts.zero_()
        idx = idx.view(T, top)
    for t in clear.nonzero()[:, 0].tolist():
        want = R.route(z[t].double(), corr.double(), top, groups, keep, scale)
        got = {int(a): float(b) for a, b in zip(idx[t], w[t].cpu())}
        assert set(got) == {a for a, _ in want}
        assert all(abs(got[a] - float(b)) < 2e-6 * scale for a, b in want)


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("T", [1, 3, 40, 257, 700])
@pytest.mark.parametrize("d,e", [(100, MoeMlp(10, 3, 21, 0.6, 5, 2, 1.7, 37, 0.9)), (72, MoeMlp(7, 2, 30, 1.1)), (264, MoeMlp(12, 4, 136, 1.5, 3, 2, 2.5, 128, 2.0)),
                                 (520, MoeMlp(3, 1, 264, 1.0, 1, 1, 1.0, 8, 0.3)), (64, MoeMlp(40, 6, 8, 0.8, 8, 4, 2.0))], ids=str)
def test_mixture_of_experts(device, dtype, T, d, e):
    """Lists of every length, also empty ones and ones of several tiles."""
    g = gen(T + d)
    sec, ffr = mlp_sections(e), round8(e.ff)
    shared = {"shared": {"ff": e.shared_ff, "limit": e.shared_limit}} if e.shared_ff else {}
    cfg = {"router": {"experts": e.experts, "top": e.top, "scale": e.scale, "groups": {"count": e.groups, "keep": e.keep}},
           "expert": {"limit": e.limit}, **shared}
    h = rnd(g, T, d)
    h[:, 0] = 1                                                   # a favourite: its list spans several tiles
    p = {"router": (rnd(g, e.experts, d) * d ** -0.5), "correction": torch.randn(e.experts, generator=g) * 0.2 - 0.5}
    p["router"][e.experts // 2, 0] += 4
    for j in [f"e{i}." for i in range(e.experts)] + (["shared."] if e.shared_ff else []):
        ff = e.shared_ff if j == "shared." else e.ff
        p |= {j + "gate": rnd(g, ff, d) * d ** -0.5, j + "up": rnd(g, ff, d) * d ** -0.5, j + "down": rnd(g, d, ff) * ff ** -0.5}
    new = lambda *s: torch.zeros(*s, dtype=dtype, device=device)
    lw = {"w_up": new(sec.total, round8(d))[:, :d], "e_up": new(e.experts, round8(2 * e.ff), round8(d))[..., :d], "e_down": new(e.experts, round8(d), ffr)[..., :e.ff],
          "correction": p["correction"].to(device), "w_down": new(round8(d), round8(e.shared_ff or 8))[:, :e.shared_ff or 8]}
    lw["w_up"][sec["router"]:sec["router"] + e.experts] = p["router"]
    for i in range(e.experts):
        lw["e_up"][i, 0:2 * e.ff:2], lw["e_up"][i, 1:2 * e.ff:2], lw["e_down"][i, :d] = (p[f"e{i}.{s}"] for s in ("gate", "up", "down"))
    if e.shared_ff:
        lw["w_up"][sec["gate"]:sec["gate"] + e.shared_ff], lw["w_up"][sec["up"]:sec["up"] + e.shared_ff] = p["shared.gate"], p["shared.up"]
        lw["w_down"][:d] = p["shared.down"]
    pd = {k: v.double() for k, v in p.items()}
    clear = choice_margin(h.double() @ pd["router"].t(), pd["correction"], cfg["router"]) > 1e-4
    want = R.experts(h.double(), pd, cfg)
    for acc in ((False, True) if device == "cuda" and dtype == BF16 and T <= 256 else (False,)):
        from dlti_b200.ops.gemm import gemm_skinny_acc
        out = M.moe(acts(h, device, dtype), e, lw, dtype, gemm_skinny_acc if acc else K.linear, acc=acc)
        got = out.value(d).double().cpu()
        if acc and out.shared is not None:
            out.shared.zero_()
        if out.counts is not None:
            assert int(out.counts.sum()) == T * e.top
            out.counts.zero_()
        assert float((got - want)[clear].norm() / want[clear].norm()) < tol(dtype, 3e-6, 8e-3)


@pytest.mark.gpu
@pytest.mark.parametrize("T,skew", [(1, 0), (16, 0), (64, 3), (300, 0), (300, 4), (2500, 1)])
def test_expert_gemms_with_long_rows(T, skew):
    """Dozens of k blocks, lists from none to thousands of rows: the stages of the kernels go round many times while some of their
    warps have nothing to copy."""
    g, E, top, d, ff = torch.Generator("cuda").manual_seed(T), 48, 4, 1544, 200
    e = MoeMlp(E, top, ff, 2.0, 4, 3)
    rnd_ = lambda *s: torch.randn(*s, device="cuda", generator=g).to(BF16)
    h, wu, wd = rnd_(T, d), rnd_(E, 2 * ff, d) * d ** -0.5, rnd_(E, d, ff) * ff ** -0.5
    z = torch.randn(T, E, device="cuda", generator=g) + skew * torch.randn(E, device="cuda", generator=g)
    _, lists, counts = M._route(None, z, 0, torch.zeros(E, device="cuda"), e)
    for _ in range(3):
        a, out = K.act(T * top, ff, BF16, "cuda"), torch.full((T * top, d), 9.0, dtype=BF16, device="cuda")
        M.grouped_gemm(h, wu, lists, counts, a, rows=ff, pairs_per_row=top, up=True, limit=2.0)
        M.grouped_gemm(a, wd, lists, counts, out, rows=d, pairs_per_row=1)
        o = 0
        for j in range(E):
            pair = lists[j, :int(counts[j])].long().cpu()
            x = h[(pair // top).cuda()].double().cpu()
            p = {"gate": wu[j, 0::2].double().cpu(), "up": wu[j, 1::2].double().cpu(), "down": torch.eye(ff, dtype=torch.double)}
            if len(pair):
                mid = a[o:o + len(pair)].cpu()
                assert rel(mid, R.clipped_expert(x, p, "", 2.0)) < 6e-3
                assert rel(out[pair.cuda()], mid.double() @ wd[j].double().cpu().t()) < 6e-3
            o += len(pair)
        assert o == T * top
    counts.zero_()


# ---- delta rule --------------------------------------------------------------------------------------------
def _delta_case(device, dtype, heads, groups, N_, P, cuts, A_log, dt_bias, seed=0, t=None, change=None):
    g = gen(N_ + P + seed)
    data, want = [], []
    for c in cuts:
        T = sum(c)
        q, k, v, z = rnd(g, T, groups, N_), rnd(g, T, groups, N_) + 0.5, rnd(g, T, heads, P), rnd(g, T, 2 * heads).float() * 2
        if change:
            change(q, k, v, z)
        data.append((q, k, v, z))
        rep = lambda x: x.repeat_interleave(heads // groups, 1)
        want.append(R.delta_rule(rep(R.unit(q.double()) * N_ ** -0.5), rep(R.unit(k.double())), v.double(), R.sigmoid(z[:, heads:].double()),
                                 R.step_decay(z[:, :heads].double(), A_log.double(), dt_bias.double())))
    ssm = torch.full((len(cuts) + 1, heads, N_, P), 3.0, device=device)    # slots hold leftovers
    slot = list(range(len(cuts), 0, -1))
    at, got = [0] * len(cuts), [[] for _ in cuts]
    for i in range(max(map(len, cuts))):
        live = [s for s in range(len(cuts)) if i < len(cuts[s])]
        live.sort(key=lambda s: not (cuts[s][i] == 1 and at[s] > 0))
        nd = sum(cuts[s][i] == 1 and at[s] > 0 for s in live)
        rows, _ = rows_for([(at[s], cuts[s][i]) for s in live], nd, 16, device)
        rows.state = torch.tensor([slot[s] for s in live], dtype=torch.int32, device=device)
        q, k, v, z = (torch.cat([data[s][x][at[s]:at[s] + cuts[s][i]] for s in live]).flatten(1) for x in range(4))
        out = D.delta_scan(acts(q, device, dtype), acts(k, device, dtype), acts(v, device, dtype), acts(z, device, F32), A_log.to(device),
                           dt_bias.to(device), ssm, rows, heads, groups, N_, P)
        o = 0
        for s in live:
            got[s].append(out[o:o + cuts[s][i]].cpu())
            o += cuts[s][i]
            at[s] += cuts[s][i]
    for a, b in zip(got, want):
        a = torch.cat(a).double().view(b.shape)
        e = (a - b).norm(dim=2) / b.square().sum(2).mean(0).sqrt()         # a head has its own size
        assert e.max() < (t or tol(dtype, 2e-5, 1e-2)), (int(e.argmax()), float(e.max()))
    assert bool((ssm[0] == 3).all())                                       # a slot nobody holds stays as it was


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("heads,groups,N_,P", [(4, 2, 20, 12), (3, 3, 72, 40), (4, 1, 128, 96), (2, 1, 256, 8), (1, 1, 300, 4), (1, 1, 8, 8), (5, 5, 18, 70),
                                               (2, 2, 64, 64)])
def test_delta_rule_over_portions(device, dtype, heads, groups, N_, P):
    """Long and short memories, portions around the 64-token chunk of the prompt kernel, states carried through slots."""
    cuts = [[64, 1, 1, 63, 17, 2], [130, 1, 40, 1], [1, 1, 2, 65]]
    _delta_case(device, dtype, heads, groups, N_, P, cuts, torch.linspace(-4, 1, heads), torch.linspace(-5, 2, heads))


@pytest.mark.parametrize("device,dtype", MODES)
def test_delta_rule_keeps_and_replaces(device, dtype):
    """No decay and full steps: what was stored for a key far back comes out unchanged, and is replaced when its key returns. The
    same key in every place of a chunk makes the chunk's system as coupled as it gets."""
    def change(q, k, v, z):
        T = q.shape[0]
        z[:, :1], z[:, 1:] = -20, 12
        k[:], q[:] = 0, 0
        k[torch.arange(T), 0, 2 + torch.arange(T) % 5] = 1       # keys come back every five tokens ...
        k[0] = 0
        k[0, 0, 0] = 1                                           # ... but the first one does not
        q[:, 0, 0] = 1
        q[1::2] = 0
        q[1::2, 0, 3] = 1
    _delta_case(device, dtype, 1, 1, 24, 16, [[150, 1, 1, 70, 2]], torch.tensor([0.0]), torch.tensor([-9.0]), t=tol(dtype, 2e-5, 6e-3), change=change)
    same = lambda q, k, v, z: (k.copy_(k[:1].expand_as(k)), q.copy_(k))
    _delta_case(device, dtype, 2, 1, 64, 32, [[200, 1, 64]], torch.tensor([-6.0, 0.0]), torch.tensor([-6.0, 0.0]), change=same)


@pytest.mark.parametrize("device,dtype", MODES)
def test_long_memory(device, dtype):
    """Slow decays over many tokens, half of them decoded one by one: rounding must not add up."""
    _delta_case(device, dtype, 2, 1, 16, 8, [[300] + [1] * 200], torch.tensor([-6.0, -4.0]), torch.tensor([-4.0, -3.0]), t=tol(dtype, 5e-5, 1e-2))


@pytest.mark.gpu
@pytest.mark.parametrize("lens", [[1000, 3, 64, 129], [17] * 9, [2048]], ids=str)
def test_chunked_delta_rule_agrees_with_tokens(lens):
    """Many chunks of unequal prompts: the prompt kernels against the token kernel."""
    g, heads, groups, N_, P = gen(len(lens)), 4, 2, 128, 64
    rows, _ = rows_for([(0, n) for n in lens], 0, 16, "cuda")
    T = sum(lens)
    q, k, v, z = rnd(g, T, groups * N_).cuda(), rnd(g, T, groups * N_).cuda(), rnd(g, T, heads * P).cuda(), torch.randn(T, 2 * heads, generator=g).cuda()
    A_log, bias = torch.linspace(-3, 2, heads).cuda(), torch.linspace(-6, 0, heads).cuda()
    out = []
    for limit in (16, 1 << 30):
        D._CHUNKED_FROM, keep = limit, D._CHUNKED_FROM
        ssm = torch.full((len(lens), heads, N_, P), 3.0, device="cuda")
        out.append((D.delta_scan(q, k, v, z, A_log, bias, ssm, rows, heads, groups, N_, P), ssm))
        D._CHUNKED_FROM = keep
    assert rel(out[0][0], out[1][0].double().cpu()) < 4e-3 and rel(out[0][1], out[1][1].double().cpu()) < 1e-4


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("C,taps", [(20, 3), (64, 4), (13, 1), (136, 2), (1032, 5)])
def test_short_convolution_over_portions(device, dtype, C, taps):
    g, cuts = gen(C), [1, 1, 2, 30, 1, 3, 70]
    m = DeltaMixer(1, 1, 8, 8, taps)
    x, w = rnd(g, sum(cuts), C), rnd(g, C, taps)
    want = R.silu(R.causal_conv(x.double(), w.double()))
    wt = torch.zeros(taps, round8(C))
    wt[:, :C] = w.t()
    state = torch.full((1, taps - 1, round8(C)), 5.0, dtype=dtype, device=device) if m.conv > 1 else None
    ssm, at, got = torch.zeros(1, 1, 8, 8, device=device), 0, []
    for c in cuts:
        rows, _ = rows_for([(at, c)], int(c == 1 and at > 0), 16, device)
        rows.state = torch.zeros(1, dtype=torch.int32, device=device)
        proj = torch.zeros(c, round8(C) + 8, dtype=dtype)
        proj[:, :C] = x[at:at + c]
        proj = proj.to(device)
        y, _ = K.short_conv(proj, 0, round8(C), wt.to(device), torch.zeros(round8(C), device=device), state, rows, dtype)
        z = torch.zeros(c, 8, dtype=dtype, device=device)
        D.delta_scan(z, z, z, torch.zeros(c, 2, device=device), torch.zeros(1, device=device), torch.zeros(1, device=device), ssm, rows, 1, 1, 8, 8,
                     conv_src=proj, conv_col=0, conv_state=state)          # renews the state
        got.append(y[:, :C].cpu())
        at += c
    assert rel(torch.cat(got), want) < tol(dtype, 2e-6, 5e-3)


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("heads,vdim", [(3, 10), (4, 64), (1, 256), (5, 24), (2, 264), (2, 520)])
def test_head_norm_with_a_silu_gate(device, dtype, heads, vdim):
    g, n = gen(vdim), heads * vdim
    y, z, w = rnd(g, 6, n), rnd(g, 6, n), rnd(g, vdim)
    y[:, :vdim] *= 8
    yd = y.double().view(6, heads, vdim)
    want = (yd / R.root_mean_square(yd, 1e-5) * w.double()).view(6, n) * R.silu(z.double())
    got = K.gated_norm(acts(y, device, dtype), acts(z, device, dtype), w.float().repeat(heads).to(device), 1e-5, heads, False, silu=True)
    assert rel(got, want) < tol(dtype, 2e-6, 4e-3)


# ---- whole models through the engine -----------------------------------------------------------------------
WHOLE = [pytest.param("cpu", F32, 5e-5, id="cpu"), pytest.param("cuda", F32, 5e-5, marks=GPU, id="gpu-f32"),
         pytest.param("cuda", BF16, 0.02, marks=GPU, id="gpu-bf16")]
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
    assert eng.blocks.num_free == eng.blocks.num_blocks and len(eng.slots.free) == 4


@pytest.mark.parametrize("device,dtype,t", WHOLE)
@pytest.mark.parametrize("name", NAMES)
def test_decoding_matches_prefill(name, device, dtype, t):
    """Token by token from the start and after a long prompt."""
    rp = ZOO.replay(name, ZOO.engine(name, device, dtype))
    for _ in range(97):
        rp.step({(97, 2): 1})
    rp.step({(171, 1): 120})
    for _ in range(51):
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
def test_packed_and_paged_prompts_agree():
    out = []
    for pack in (True, False):
        eng = ZOO.engine("wide", "cuda", BF16)
        eng.runner.pack_prompts = pack
        rp = ZOO.replay("wide", eng)
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
    ZOO.check(name, rp, 0.02)


def _mlp(d, i, **kw):
    d["layers"][i]["mlp"]["router"].update(kw)


def _edit(w, **edits):
    return {**w, **{k.replace("__", "."): f(w[k.replace("__", ".")]) for k, f in edits.items()}}


MISTAKES = {
    "window one longer": lambda d, w: (d["layers"][1]["mixer"]["mask"].update(size=24), w)[1],
    "window one shorter": lambda d, w: (d["layers"][3]["mixer"]["mask"].update(size=64), w)[1],
    "no cap": lambda d, w: (d["layers"][1]["mixer"].update(softcap=0.0), w)[1],
    "no sink": lambda d, w: _edit(w, l2__mix__sink=lambda t: t - 1e4),
    "values not mixed": lambda d, w: _edit(w, l3__mix__vmix=lambda t: t * 0),
    "another first layer": lambda d, w: (d["layers"][1]["mixer"].update(v_mix=False), w)[1],
    "score scale": lambda d, w: (d["layers"][2]["mixer"].update(scale=0.45), w)[1],
    "logit scale": lambda d, w: (d.update(logit_scale=0.33), w)[1],
    "embedding scale": lambda d, w: (d["embedding"].update(scale=1.6), w)[1],
    "one group more": lambda d, w: (_mlp(d, 0, groups={"count": 5, "keep": 3}), w)[1],
    "router scale": lambda d, w: (_mlp(d, 0, scale=1.5), w)[1],
    "no correction": lambda d, w: _edit(w, l0__mlp__correction=lambda t: t * 0),
    "expert limit": lambda d, w: (d["layers"][2]["mlp"]["expert"].update(limit=1.0), w)[1],
    "shared limit": lambda d, w: (d["layers"][0]["mlp"]["shared"].update(limit=0.8), w)[1],
    "taps reversed": lambda d, w: _edit(w, l0__mix__k__conv=lambda t: t.flip(1)),
    "decay": lambda d, w: _edit(w, l4__mix__A_log=lambda t: t + 0.1),
    "no bias": lambda d, w: _edit(w, l1__mix__k__b=lambda t: t * 0),
    "norms exchanged": lambda d, w: {**w, "l2.norm1": w["l2.norm1b"], "l2.norm1b": w["l2.norm1"]},
}


@pytest.mark.parametrize("what", list(MISTAKES))
def test_a_mistake_shows(what):
    """The comparisons above can fail: the oracle with one detail off is many fp32 tolerances away."""
    d, _, _, w = ZOO.model("odd")
    d = copy.deepcopy(d)
    bad = R.forward(d, MISTAKES[what](d, w), ZOO.tokens("odd", 171, 1))
    assert row_errors(bad, ZOO.oracle("odd", 171, 1)).max() > 0.005


def test_residual_after_every_layer():
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
    LX.save_checkpoint(cfg, st, tmp_path)
    c = resolve_config(str(tmp_path))
    assert isinstance(c, LX.LatanexConfig) and c.layers == cfg.layers and json.load(open(tmp_path / "config.json")) == d
    fam = family_of(c)
    assert fam.name == "Latanex"
    w = fam.load_weights(c, tmp_path, "cpu", F32)
    assert {n for n, _ in LX.named_tensors(w)} == set(st)
    for name, dst in LX.named_tensors(w):
        assert torch.equal(dst, st[name].float().reshape(dst.shape)), name
    assert c.num_params() >= sum(t.numel() for t in st.values())
    for p in ("latanex-tiny", "latanex-3b"):
        assert isinstance(resolve_config(p), LX.LatanexConfig)
    assert family_of(resolve_config("logozen-tiny")).name == "Logozen"


def test_optional_entries_of_the_configuration():
    """Entries that mean "none" when absent or null; the first mixing layer's unused share may be stored."""
    d = copy.deepcopy(CONFIGS["odd"])
    for e in d["layers"][2]["mixer"], d["layers"][3]["mixer"]:
        e["mask"], e["softcap"], e["v_mix"] = None, None, False
    del d["layers"][1]["mixer"]["mask"], d["layers"][2]["mlp"]["router"]["groups"]
    d["layers"][2]["mlp"]["shared"] = None
    cfg = LX.LatanexConfig.from_dict(d)
    a, e = cfg.layers[2].mixer, cfg.layers[2].mlp
    assert (a.window, a.softcap, a.v_mix, cfg.layers[1].mixer.window) == (0, 0.0, False, 0) and (e.groups, e.keep, e.shared_ff) == (1, 1, 0)
    st = LX.random_state(cfg)
    assert "l1.mix.vmix" not in st and not any("shared" in k for k in st if k.startswith("l2."))
    LX.from_state(cfg, {**st, "l1.mix.vmix": torch.tensor(0.5)}, "cpu", F32)
    eng = ZOO.engine("odd", "cpu", F32)
    eng2 = type(eng)(cfg, LX.from_state(cfg, st, "cpu", F32), eng.tp, eng.tokenizer, num_blocks=32, max_model_len=128, max_num_seqs=4)
    rp = ZOO.replay("odd", eng2)
    rp.step({(97, 2): 97})
    want = R.forward(d, {k: v.double() for k, v in st.items()}, ZOO.tokens("odd", 97, 2))
    assert row_errors(rp.logits((97, 2)), want).max() < 5e-5


@pytest.mark.parametrize("edit,msg", [(lambda d: d["layers"][0]["mlp"]["router"].update(groups={"count": 4, "keep": 2}), "groups"),
                                      (lambda d: d["layers"][0]["mlp"]["router"].update(top=5), "experts"),
                                      (lambda d: d["layers"][1]["mixer"].update(kv_heads=4), "query heads"),
                                      (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "query/key heads"),
                                      (lambda d: d["layers"][3]["mixer"].update(vdim=12), "mixed"),
                                      (lambda d: d["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
                                      (lambda d: d["layers"][1].update(type="conv"), "mixer type"),
                                      (lambda d: d["layers"][1]["mlp"].update(kind="sparse"), "feed-forward")])
def test_inconsistent_configurations_are_refused(edit, msg):
    d = copy.deepcopy(CONFIGS["odd"])
    edit(d)
    with pytest.raises(ValueError, match=msg):
        LX.LatanexConfig.from_dict(d)


def test_misfitting_tensors_and_prefix_caching_are_refused():
    _, cfg, st, _ = ZOO.model("odd")
    with pytest.raises(ValueError, match="l0.mlp.e3.up"):
        LX.from_state(cfg, {**st, "l0.mlp.e3.up": st["l0.mlp.e3.up"][:-1]}, "cpu", F32)
    with pytest.raises(ValueError, match="l0.mix.v.conv"):
        LX.from_state(cfg, {**st, "l0.mix.v.conv": st["l0.mix.v.conv"][:, :-1]}, "cpu", F32)
    with pytest.raises(ValueError, match="prefix caching"):
        ZOO.engine("odd", "cpu", F32, enable_prefix_caching=True)


@pytest.mark.parametrize("device,dtype,t", WHOLE)
def test_trace_run_command(tmp_path, device, dtype, t):
    name = "odd"
    _, cfg, st, _ = ZOO.model(name)
    LX.save_checkpoint(cfg, st, tmp_path / "m")
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
