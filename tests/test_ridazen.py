"""Ridazen against its plain implementation (tests/ref_ridazen.py): each mechanism alone, then whole models through the
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

from dlti_b200.models import ridazen as RZ
from dlti_b200.models.stack import AttentionMixer, DistanceBias, MoeMlp, QueryTemp, mixer_sections, mlp_sections, round8
from dlti_b200.ops import _lib
from dlti_b200.ops import moe as M
from dlti_b200.ops import prenorm as P
from dlti_b200.ops import stack as K
from dlti_b200.serve.engine import _pieces, chunk_pieces
from tests import ref_ridazen as R
from tests.ridazen_util import CONFIGS, ZOO, choice_margin
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
@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("T,d", [(5, 100), (1, 8), (3, 1031), (700, 2048), (9, 4096), (130, 2052), (2, 8200)])
def test_norms_between_sublayers(device, dtype, T, d):
    """A finished output with a factor, plain and normed; the embedding on top; the next input normed and as it is."""
    g, eps = gen(T * d), 1e-4
    x, y, post, pre = torch.randn(T, d, generator=g) * 3, rnd(g, T, d), torch.randn(d, generator=g), torch.randn(d, generator=g)
    table, ids = rnd(g, 7, d), torch.randint(0, 7, (T,), generator=g)
    t = tol(dtype, 2e-6, 4e-3)
    dev = lambda v: v.to(device)
    for p, again in ((None, False), (post, False), (None, True), (post, True)):
        add = y.double() if p is None else R.rms_norm(y.double(), p.double(), eps)
        want = x.double() + 0.37 * add + (1.7 * table.double()[ids] if again else 0)
        kw = dict(mult=0.37, post=None if p is None else dev(p), embed=(dev(ids), table.to(device, dtype), 1.7) if again else None)
        xd = x.clone().to(device)
        h = P.between_(xd, acts(y, device, dtype), dev(pre), eps, dtype, **kw)
        assert rel(xd, want) < 2e-6 and rel(h, R.rms_norm(want, pre.double(), eps)) < t
        xc = x.clone().to(device)
        hc = P.between_(xc, acts(y, device, dtype), None, eps, dtype, copy=True, **kw)
        assert torch.equal(xc, xd) and torch.equal(hc, xd.to(dtype))
        assert P.between_(x.clone().to(device), acts(y, device, dtype), None, eps, dtype, **kw) is None
        if device == "cuda" and dtype == BF16:
            acc, xf = accumulator(y.cuda().float()), x.clone().to(device)
            hf = P.between_(xf, acc, dev(pre), eps, dtype, acc=True, **kw)
            assert torch.equal(xf, xd) and torch.equal(hf, h) and not acc.any()
    x0 = torch.full((T, d), 5.0, device=device)
    h = P.between_(x0, None, dev(pre), eps, dtype, embed=(dev(ids), table.to(device, dtype), 1.0), fresh=True)
    assert rel(x0, table.double()[ids]) < 1e-7 and rel(h, R.rms_norm(table.double()[ids], pre.double(), eps)) < t


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("T,d,top,shared", [(5, 100, 3, True), (4, 256, 1, False), (600, 512, 7, True), (3, 33, 40, False), (2, 2048, 8, True)])
def test_expert_outputs_are_added_up(device, dtype, T, d, top, shared):
    g, eps = gen(T + d), 1e-5
    x, rows, w, y, s, pre = (torch.randn(T, d, generator=g), rnd(g, T * top, d), torch.randn(T, top, generator=g), rnd(g, T, d),
                             torch.rand(T, generator=g), torch.randn(d, generator=g))
    sum_ = (rows.double().view(T, top, d) * w.double()[:, :, None]).sum(1) + (y.double() * s.double()[:, None] if shared else 0)
    want = x.double() + 0.6 * sum_
    xd, counts = x.clone().to(device), torch.full((37,), 5, dtype=torch.int32, device=device)
    e = M.ExpertSum(acts(rows, device, dtype), w.to(device), acts(y, device, dtype) if shared else None, counts, s.to(device) if shared else None)
    h = P.between_(xd, e, pre.to(device), eps, dtype, mult=0.6)
    assert rel(xd, want) < 4e-6 and rel(h, R.rms_norm(want, pre.double(), eps)) < tol(dtype, 4e-6, 4e-3)
    assert device == "cpu" or not counts.any()
    if device == "cuda" and dtype == BF16 and shared:
        xf, acc = x.clone().to(device), accumulator(y.cuda().float())
        hf = P.between_(xf, M.ExpertSum(e.rows, e.weights, acc, counts, e.share), pre.to(device), eps, dtype, mult=0.6, acc=True)
        assert torch.equal(xf, xd) and torch.equal(hf, h) and not acc.any()


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("T,n,col,width", [(5, 13, 26, 39), (300, 24, 24, 72), (1, 1, 2, 5), (64, 128, 0, 1536)])
def test_token_inputs(device, dtype, T, n, col, width):
    g = gen(n)
    u, table, ids = rnd(g, T, n) * 2, rnd(g, 11, width), torch.randint(0, 11, (T,), generator=g)
    want = R.gelu_tanh(u.double()) * table.double()[ids][:, col:col + n]
    got = P.token_gate(acts(u, device, dtype), ids.to(device), table.to(device, dtype), col, n, dtype)
    assert rel(got, want) < tol(dtype, 2e-6, 4e-3)
    if device == "cuda" and dtype == BF16:
        acc = accumulator(u.cuda().float())
        assert torch.equal(P.token_gate(acc, ids.cuda(), table.cuda(), col, n, dtype, acc=True), got) and not acc.any()


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("T", [1, 30, 300])
@pytest.mark.parametrize("scale,cap", [(1.0, 0.0), (0.7, 0.0), (1.0, 4.0), (0.3, 2.5)])
def test_logits_are_scaled_and_capped(device, dtype, T, scale, cap):
    g = gen(T)
    h, w = rnd(g, T, 72), rnd(g, 104, 72)
    z = h.double() @ w.double().t() * scale
    got = K.linear_f32(acts(h, device, dtype), w.to(device, dtype), scale, cap)
    assert got.dtype == F32 and rel(got, R.softcap(z, cap) if cap else z) < tol(dtype, 2e-6, 2e-6 if T <= 256 else 5e-6)


# ---- attention ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows,far", [(16, 128), (32, 128), (2, 2), (12, 70), (8, 31), (20, 4000), (4, 3), (64, 33), (10, 6)])
def test_distance_buckets(rows, far):
    b = DistanceBias(rows, far)
    want = [R.distance_bucket(n, rows, far) for n in range(3 * far)]
    assert [b.bucket(n) for n in range(3 * far)] == want
    assert want == sorted(want) and want[far:] == [rows - 1] * (2 * far)
    assert b.buckets == want[:want.index(rows - 1)]


def test_query_factors():
    t = K.temp_table(500, QueryTemp(0.35, 64), "cpu")
    assert torch.allclose(t.double(), torch.tensor([R.query_factor(p, 0.35, 64) for p in range(500)], dtype=torch.double), rtol=1e-7)
    assert t[62] == 1 and t[63] > 1.2 and t[63] == t[126] and t[127] > t[126]


class AttentionCase:
    """One attention layer with its cache and convolution state: sequences of given projections, fed in portions, beside the oracle."""

    def __init__(self, device, dtype, shape, taps, temp, bias, lens, bs=16, seed=0, change=None):
        H, G, dim, vdim = shape
        g = gen(H * dim + taps + seed)
        self.device, self.dtype, self.bs, self.lens = device, dtype, bs, lens
        self.m = m = AttentionMixer(H, G, dim, vdim, 1.5 * dim ** -0.5, head_gate=False, conv=taps, q_temp=QueryTemp(*temp) if temp else None,
                                    bias_by=DistanceBias(*bias) if bias else None, out_gate=True)
        self.sec = sec = mixer_sections(m)
        self.width = dict(q=H * dim, k=G * dim, v=G * vdim, g=H * vdim)
        self.u = {s: [rnd(g, n, w) for n in lens] for s, w in self.width.items()}
        self.norm = {s: torch.randn(dim, generator=g) * 0.3 + 1 for s in "qk"}
        self.conv = {s: rnd(g, self.width[s], taps) for s in "qkv"} if taps else None
        self.table = rnd(g, bias[0], H) * 2 if bias else None
        self.factor = (lambda p: R.query_factor(p, *temp)) if temp else (lambda p: 1.0)
        if change:
            change(self)
        self.want = [self.oracle(i) for i in range(len(lens))]
        self.lw = {"q_norm": self.norm["q"].to(device), "k_norm": self.norm["k"].to(device)}
        if taps:
            w = torch.zeros(taps, sec["g"])
            for s in "qkv":
                w[:, sec[s]:sec[s] + self.width[s]] = self.conv[s].t()
            self.lw["conv"] = w.to(device)
        self.bias = None
        if bias:
            t = self.table.float()
            self.bias = (t[m.bias_by.buckets] - t[-1]).t().contiguous().to(device)
        self.factors = K.temp_table(max(lens) + 1, m.q_temp, device) if temp else None
        # slots and pages hold leftovers of other sequences
        self.state = torch.full((len(lens) + 1, taps - 1, sec["g"]), 9.0, dtype=dtype, device=device) if taps > 1 else None
        need = [-(-n // bs) for n in lens]
        perm, o = torch.randperm(sum(need) + 3, generator=g), 0
        self.tabs = torch.zeros(len(lens), max(need) + 1, dtype=torch.int32)
        for i, x in enumerate(need):
            self.tabs[i, :x] = perm[o:o + x]
            o += x
        new = lambda n: torch.full((sum(need) + 3, bs, G, round8(n)), 9.0, dtype=dtype, device=device)
        self.kc, self.vc = new(dim), new(vdim)
        self.at, self.got = [0] * len(lens), [[] for _ in lens]

    def oracle(self, i):
        m, n = self.m, self.lens[i]
        q, k, v = (self.u[s][i].double() if self.conv is None else R.causal_conv(self.u[s][i].double(), self.conv[s].double()) for s in "qkv")
        q = R.rms_norm(q.view(n, m.heads, m.dim), self.norm["q"].double(), 1e-5)
        k = R.rms_norm(k.view(n, m.kv_heads, m.dim), self.norm["k"].double(), 1e-5)
        q = q * torch.tensor([self.factor(p) for p in range(n)], dtype=torch.double)[:, None, None]
        bias = None
        if self.table is not None:
            b = m.bias_by
            bias = self.table.double()[[R.distance_bucket(x, b.rows, b.far) for x in range(n)]]
        o = R.attend(q, k, v.view(n, m.kv_heads, m.vdim), m.scale, bias).flatten(1)
        return o * R.sigmoid(self.u["g"][i].double())

    def step(self, parts, packed=False, acc=False):
        """parts: {sequence: next rows}; packed: prompt rows through the varlen kernel; acc: the projection as an accumulator."""
        live = sorted(parts, key=lambda s: not (parts[s] == 1 and self.at[s] > 0))
        nd = sum(parts[s] == 1 and self.at[s] > 0 for s in live)
        rows, _ = rows_for([(self.at[s], parts[s]) for s in live], nd, self.bs, "cpu")
        rows.tables = self.tabs[live].contiguous()
        rows.slots = torch.tensor([int(rows.tables[i, p // self.bs]) * self.bs + p % self.bs for i, p in zip(rows.seq.tolist(), rows.pos.tolist())])
        rows.state = torch.tensor([len(self.lens) - s for s in live], dtype=torch.int32)
        pieces = None
        if packed and len(live) > nd:
            import dlti_b200.serve.engine as E
            keep, E.PACK_FROM = E.PACK_FROM, 1
            arr, n, longest, ext, prefix = chunk_pieces(rows.cu.tolist(), [self.at[s] for s in live[nd:]], rows.tables.tolist()[nd:], self.bs, 0, 1 << 30)
            E.PACK_FROM = keep
            pieces = _pieces(torch.from_numpy(arr).to(self.device), int(rows.cu[-1]), n, longest, ext, prefix)
        rows = K.Rows(*[t.to(self.device) if torch.is_tensor(t) else t for t in vars(rows).values()])
        T, m = rows.pos.numel(), self.m
        proj = torch.zeros(T, self.sec.total, dtype=F32 if acc else self.dtype)
        for s, xs in self.u.items():
            proj[:, self.sec[s]:self.sec[s] + self.width[s]] = torch.cat([xs[i][self.at[i]:self.at[i] + parts[i]] for i in live])
        proj = proj.to(self.device)
        q, gate = K.conv_qkv(proj, self.sec, m, self.lw, self.factors, 1e-5, rows, self.state, self.kc, self.vc, self.dtype, packed=pieces, acc=acc)
        assert not acc or not proj.any()
        attend = K.paged_attention if pieces is None else lambda q, m, rows, *a, **kw: K.packed_attention(q, m, rows, pieces, *a, **kw)
        out = attend(q, m, rows, self.kc, self.vc, None, bias=self.bias, out_gate=gate)
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
        if self.state is not None:
            assert bool((self.state[0] == 9).all())                       # a slot nobody holds stays as it was


def _packs(device, dtype, dim, vdim):
    return [False, True] if device == "cuda" and dtype == BF16 and max(dim, vdim) <= 128 and vdim % 8 == 0 else [False]


SHAPES = [(6, 3, 14, 10), (8, 2, 64, 64), (4, 4, 128, 128), (3, 3, 40, 72), (2, 1, 256, 256), (20, 1, 33, 8), (2, 1, 264, 40), (4, 1, 64, 128)]
KINDS = [(3, (0.4, 17), (12, 70)), (4, (0.2, 50), (32, 128)), (1, (0.1, 1), (2, 2)), (2, None, (64, 40)), (0, (0.3, 64), None), (6, None, (16, 300)),
         (0, None, None)]


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("taps,temp,bias", KINDS, ids=str)
def test_attention_over_portions(device, dtype, shape, taps, temp, bias):
    """Decode rows beside portions, portions around page borders and shorter than the convolution, states carried through slots."""
    for packed in _packs(device, dtype, *shape[2:]):
        c = AttentionCase(device, dtype, shape, taps, temp, bias, [170, 75, 20, 33])
        for parts in ({0: 64, 1: 2, 2: 16}, {0: 1, 1: 15, 3: 31}, {2: 1, 0: 65, 1: 1}, {3: 2, 0: 1, 1: 1, 2: 1}, {0: 2, 1: 55}, {0: 1, 1: 1, 2: 1}, {0: 36}):
            c.step(parts, packed)
        # one tap alone makes heavy-tailed heads: sharper scores
        c.check(tol(dtype, 1e-5, 2.5e-2 if taps == 1 else 1.5e-2))


@pytest.mark.gpu
@pytest.mark.parametrize("shape", SHAPES, ids=str)
@pytest.mark.parametrize("taps,temp,bias", KINDS, ids=str)
def test_decoding_from_accumulators(shape, taps, temp, bias):
    """Decode steps that consume the GEMM's accumulator, from the first token on; a prompt's portion between them."""
    c = AttentionCase("cuda", BF16, shape, taps, temp, bias, [40, 33, 9])
    c.step({0: 7})                                        # longer than one convolution, then decoded
    for _ in range(8):
        c.step({1: 1}, acc=c.at[1] > 0)                   # from its first token on
    for i in range(20):
        c.step({0: 1, 1: 1, **({2: 1} if 0 < c.at[2] < 9 else {})}, acc=True) if i != 5 else c.step({0: 1, 1: 1, 2: 2})
    c.check(1.5e-2)


@pytest.mark.gpu
@pytest.mark.parametrize("rows,far", [(2, 2), (8, 5), (32, 100), (32, 127), (16, 128), (32, 129), (16, 200), (32, 256), (12, 257), (20, 700), (64, 4000)])
def test_biased_tiles_of_the_prompt_kernel(rows, far):
    """Several tiles of 128 rows, whole prompts and portions on top of cached rows; biases of neighbouring buckets far apart."""
    def alternate(c):
        c.table = ((-1.0) ** torch.arange(rows)[:, None] * 3 + rnd(gen(far), rows, 4)).to(BF16)
    for cuts in ([600], [130, 300, 170]):
        c = AttentionCase("cuda", BF16, (4, 2, 64, 64), 3, (0.2, 100), (rows, far), [600, 385], change=alternate)
        at = 0
        for x in cuts:
            y = min(x, 385 - c.at[1])
            c.step({0: x, 1: y} if y > 1 else {0: x}, packed=True)
            at += x
        c.check(1.5e-2)


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("shape", [(6, 3, 14, 10), (4, 2, 64, 64)], ids=str)
@pytest.mark.parametrize("far", [16, 63, 64, 129])
def test_one_distance_stands_out(device, dtype, far, shape):
    """The bucket that holds the last distances before `far`, or the first bucket beyond all others, outweighs everything: a distance
    that falls into the wrong bucket shows. In prompts, portions and decoding; pages and tiles end on either side."""
    n, rows = 200, 12
    edges = [R.distance_bucket(x, rows, far) for x in range(n)]
    for b in (0, rows // 2 - 1, rows // 2, edges[far - 1], rows - 1):
        def spike(c):
            c.table[b] = 14
        for cuts in ([n], [far, 1, n], [max(1, far - 5), 7, n], [max(1, far + 3), n]):
            for packed in _packs(device, dtype, *shape[2:]):
                c = AttentionCase(device, dtype, shape, 2, (0.3, 50), (rows, far), [n], change=spike)
                for x in cuts:
                    if min(x, n - c.at[0]) > 0:
                        c.step({0: min(x, n - c.at[0])}, packed)
                for i in range(3):
                    if c.at[0] < n:
                        c.step({0: 1})
                c.check(tol(dtype, 2e-5, 2e-2))


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("shape", [(6, 3, 14, 10), (4, 2, 64, 64)], ids=str)
@pytest.mark.parametrize("query,key", [(199, 0), (199, 1), (150, 16), (144, 15), (130, 2), (64, 63), (65, 0), (16, 15)])
def test_one_far_key_stands_out(device, dtype, shape, query, key):
    """One key that looks like one query, far back among many others, right at page borders and at the first tokens."""
    def spike(c):
        H, G, dim, _ = shape
        c.u["q"][0][query] = c.u["k"][0][key].view(G, 1, dim).expand(G, H // G, dim).flatten() * 4
        c.norm["q"], c.norm["k"] = c.norm["q"] * 0 + 3, c.norm["k"] * 0 + 1.5
    for cuts in ([200], [query, 1, 200], [key + 1, 200], [max(1, query - 5), 7, 200]):
        for packed in _packs(device, dtype, *shape[2:]):
            c = AttentionCase(device, dtype, shape, 0, (0.3, 64), (12, 70), [200], change=spike)
            for x in cuts:
                if min(x, 200 - c.at[0]) > 0:
                    c.step({0: min(x, 200 - c.at[0])}, packed)
            c.check(tol(dtype, 4e-5, 5e-2))


@pytest.mark.gpu
@pytest.mark.parametrize("far", [7, 70, 900])
@pytest.mark.parametrize("H,G,dim", [(8, 2, 72), (20, 1, 64), (4, 4, 128)])
def test_decode_splits(far, H, G, dim):
    g, bs, lens, nb = gen(far), 16, [(5, 1), (777, 1), (64, 1), (1023, 1), (0, 1)], 12
    rows, pages = rows_for(lens, 5, bs, "cuda")
    m = AttentionMixer(H, G, dim, dim, dim ** -0.5, head_gate=False, bias_by=DistanceBias(nb, far), out_gate=True)
    q, kc, vc, z, table = rnd(g, 5, H, dim), rnd(g, pages, bs, G, dim), rnd(g, pages, bs, G, dim), rnd(g, 5, H * dim), rnd(g, nb, H) * 2
    want = []
    for i, (s, _) in enumerate(lens):
        j = torch.arange(s + 1)
        sl = rows.tables[i].cpu()[j // bs].long() * bs + j % bs
        k, v = (c.view(-1, G, dim)[sl].double() for c in (kc, vc))
        qq = torch.zeros(s + 1, H, dim, dtype=torch.double)
        qq[-1] = q[i].double()
        o = R.attend(qq, k, v, m.scale, table.double()[[R.distance_bucket(x, nb, far) for x in range(s + 1)]])[-1].flatten()
        want.append(o * R.sigmoid(z[i].double()))
    bias = (table.float()[m.bias_by.buckets] - table.float()[-1]).t().contiguous().cuda()
    for splits in (1, 2, 5, 32, None):
        out = torch.full((5, H * dim), 7.0, dtype=BF16, device="cuda")
        K.attn_paged_decode(q.flatten(1).cuda(), m, rows, kc.cuda(), vc.cuda(), None, out, splits=splits, bias=bias, out_gate=z.cuda())
        assert rel(out, torch.stack(want)) < 5e-3


# ---- feed-forwards -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=GPU)])
@pytest.mark.parametrize("E,top", [(10, 3), (1, 1), (64, 8), (6, 6), (256, 33), (100, 1), (12, 2)])
def test_routing(device, E, top):
    """The largest biased logits, weighed by their softmax among themselves; large logits do not overflow."""
    g, T = gen(E + top), 75
    e = MoeMlp(E, top, 8, act="relu2", score="softmax")
    z, b = torch.randn(T, E, generator=g) * 3, torch.randn(E, generator=g)
    z[:5] += 200
    z[5:9] -= 200
    clear = choice_margin(z.double() + b.double(), top) > 1e-4
    assert clear.float().mean() > 0.9
    if device == "cpu":
        idx, w = M.route_ref(z, b, e)
    else:
        wide = torch.full((T, E + 11), 7.0, device="cuda")
        wide[:, 5:5 + E], wide[:, 2] = z, z[:, 0]
        share = torch.zeros(T, device="cuda")
        w, lists, counts = M._route(None, wide, 5, b.cuda(), e, share=(2, share))
        assert rel(share, R.sigmoid(z[:, 0].double())) < 1e-6
        assert int(counts.sum()) == T * top
        idx = torch.full((T * top,), -1)
        for j in range(E):
            idx[lists[j, :int(counts[j])].long().cpu()] = j
        counts.zero_()
        idx = idx.view(T, top)
    for t in clear.nonzero()[:, 0].tolist():
        want = R.route((z[t] + b).double(), top)
        got = {int(a): float(x) for a, x in zip(idx[t], w[t].cpu())}
        assert set(got) == {a for a, _ in want} and all(abs(got[a] - x) < 3e-6 for a, x in want)


def _experts(*a, shared=0):
    return MoeMlp(*a, act="relu2", score="softmax", shared_ff=shared, shared_gate=shared > 0)


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("T", [1, 3, 40, 257, 700])
@pytest.mark.parametrize("d,e", [(100, _experts(10, 3, 21, shared=37)), (72, _experts(7, 2, 30)), (264, _experts(12, 4, 136, shared=128)),
                                 (520, _experts(3, 1, 264, shared=8)), (64, _experts(40, 6, 8)), (192, _experts(5, 5, 600, shared=2056))], ids=str)
def test_mixture_of_experts(device, dtype, T, d, e):
    """Lists of every length, also empty ones and ones of several tiles."""
    g = gen(T + d)
    sec, ffr = mlp_sections(e), round8(e.ff)
    cfg = {"router": {"experts": e.experts, "top": e.top}, **({"shared": {"ff": e.shared_ff}} if e.shared_ff else {})}
    h = rnd(g, T, d)
    h[:, 0] = 1                                                   # a favourite: its list spans several tiles
    p = {"router": (rnd(g, e.experts, d) * d ** -0.5), "router.b": torch.randn(e.experts, generator=g) * 0.2}
    p["router"][e.experts // 2, 0] += 4
    for j in [f"e{i}." for i in range(e.experts)] + (["shared."] if e.shared_ff else []):
        ff = e.shared_ff if j == "shared." else e.ff
        p |= {j + "up": rnd(g, ff, d) * d ** -0.5, j + "down": rnd(g, d, ff) * ff ** -0.5}
    new = lambda *s: torch.zeros(*s, dtype=dtype, device=device)
    lw = {"w_up": new(sec.total, round8(d))[:, :d], "e_up": new(e.experts, ffr, round8(d))[..., :d], "e_down": new(e.experts, round8(d), ffr)[..., :e.ff],
          "correction": p["router.b"].to(device), "w_down": new(round8(d), round8(e.shared_ff or 8))[:, :e.shared_ff or 8]}
    lw["w_up"][sec["router"]:sec["router"] + e.experts] = p["router"]
    for i in range(e.experts):
        lw["e_up"][i, :e.ff], lw["e_down"][i, :d] = p[f"e{i}.up"], p[f"e{i}.down"]
    if e.shared_ff:
        p["shared.sg"] = rnd(g, 1, d) * d ** -0.5
        lw["w_up"][sec["up"]:sec["up"] + e.shared_ff], lw["w_up"][sec["sg"]], lw["w_down"][:d] = p["shared.up"], p["shared.sg"][0], p["shared.down"]
    pd = {k: v.double() for k, v in p.items()}
    clear = choice_margin(h.double() @ pd["router"].t() + pd["router.b"], e.top) > 1e-4
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


# ---- whole models through the engine -----------------------------------------------------------------------
WHOLE = [pytest.param("cpu", F32, 5e-5, id="cpu"), pytest.param("cuda", F32, 5e-5, marks=GPU, id="gpu-f32"),
         pytest.param("cuda", BF16, 0.03, marks=GPU, id="gpu-bf16")]
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
    ZOO.check(name, rp, 0.03)


def _mixer(d, i, **kw):
    d["layers"][i]["mixer"].update(kw)


def _edit(w, **edits):
    return {**w, **{k.replace("__", "."): f(w[k.replace("__", ".")]) for k, f in edits.items()}}


MISTAKES = {
    "buckets end farther out": lambda d, w: (_mixer(d, 0, bias_max=75), w)[1],
    "one bucket fewer": lambda d, w: _edit(w, l1__mix__rel=lambda t: torch.cat([t[:-2], t[-1:]])),
    "no bias": lambda d, w: _edit(w, l2__mix__rel=lambda t: t * 0),
    "score scale": lambda d, w: (_mixer(d, 2, scale=0.21), w)[1],
    "scaled bias": lambda d, w: _edit(w, l0__mix__rel=lambda t: t * d["layers"][0]["mixer"]["scale"]),
    "no query factor": lambda d, w: (_mixer(d, 0, q_temp=None), w)[1],
    "query factor a position late": lambda d, w: (_mixer(d, 3, q_temp={"coef": 0.5, "every": 2}), w)[1],
    "taps reversed": lambda d, w: _edit(w, l0__mix__k__conv=lambda t: t.flip(1)),
    "no convolution on v": lambda d, w: _edit(w, l1__mix__v__conv=lambda t: torch.cat([t[:, :-1] * 0, t[:, -1:]], 1)),
    "no output gate": lambda d, w: _edit(w, l2__mix__g=lambda t: t * 0),
    "no router bias": lambda d, w: _edit(w, **{"l0__mlp__router__b": lambda t: t * 0}),
    "one expert more": lambda d, w: (d["layers"][0]["mlp"]["router"].update(top=4), w)[1],
    "shared expert's gate": lambda d, w: _edit(w, l3__mlp__shared__sg=lambda t: t * 0),
    "token input of another layer": lambda d, w: {**w, "side.embed": w["side.embed"].roll(d["token_side"]["dim"], 1)},
    "no token input": lambda d, w: _edit(w, l1__side__norm=lambda t: t * 0),
    "one pass fewer": lambda d, w: (d["loop"].update(times=2), w)[1],
    "loop begins later": lambda d, w: (d["loop"].update(start=2), w)[1],
    "residual factor": lambda d, w: (d.update(residual_mult=0.61), w)[1],
    "logit scale": lambda d, w: (d.update(logit_scale=1.32), w)[1],
    "no cap": lambda d, w: (d.update(logit_softcap=0.0), w)[1],
}


@pytest.mark.parametrize("what", list(MISTAKES))
def test_a_mistake_shows(what):
    """The comparisons above can fail: the oracle with one detail off is many fp32 tolerances away."""
    d, _, _, w = ZOO.model("odd")
    d = copy.deepcopy(d)
    bad = R.forward(d, MISTAKES[what](d, w), ZOO.tokens("odd", 171, 1))
    assert row_errors(bad, ZOO.oracle("odd", 171, 1)).max() > 0.004


def test_the_embedding_is_added_before_each_pass_but_the_first():
    order = R.running_order(4, {"start": 1, "stop": 3, "times": 3})
    cfg = RZ.RidazenConfig.from_dict(CONFIGS["odd"])
    assert cfg.runs == [i for i, _ in order] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert cfg.restarts == {r for r, (_, again) in enumerate(order) if again} == {3, 5}


def test_residual_after_every_run():
    d, _, _, w = ZOO.model("odd")
    eng = ZOO.engine("odd", "cpu", F32)
    eng.runner.trace = []
    ZOO.replay("odd", eng).step({(40, 4): 40})
    want = []
    R.forward(d, w, ZOO.tokens("odd", 40, 4), want)
    assert len(want) == len(eng.runner.trace) == 8
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
    RZ.save_checkpoint(cfg, st, tmp_path)
    c = resolve_config(str(tmp_path))
    assert isinstance(c, RZ.RidazenConfig) and c.layers == cfg.layers and json.load(open(tmp_path / "config.json")) == d
    fam = family_of(c)
    assert fam.name == "Ridazen"
    w = fam.load_weights(c, tmp_path, "cpu", F32)
    assert {n for n, _ in RZ.named_tensors(w)} == set(st)
    for name, dst in RZ.named_tensors(w):
        assert torch.equal(dst, st[name].float()), name
    assert c.num_params() >= sum(t.numel() for t in st.values())
    for p in ("ridazen-tiny", "ridazen-3b"):
        assert isinstance(resolve_config(p), RZ.RidazenConfig)


def test_bucket_counts_come_from_the_checkpoint(tmp_path):
    """config.json need not say how many distance buckets a layer has: the stored tables do, layer by layer."""
    d, cfg, st, _ = ZOO.model("odd")
    RZ.save_checkpoint(cfg, st, tmp_path)
    plain = copy.deepcopy(d)
    for l in plain["layers"]:
        l["mixer"].pop("bias_rows", None)
    json.dump(plain, open(tmp_path / "config.json", "w"))
    assert RZ.RidazenConfig.load(tmp_path).layers == cfg.layers
    os.remove(tmp_path / "model.safetensors")
    assert RZ.RidazenConfig.load(tmp_path).layers[0].mixer.bias_by.rows == RZ.BIAS_ROWS


def test_optional_entries_of_the_configuration():
    """Entries that mean "none" when absent or null."""
    d = copy.deepcopy(CONFIGS["odd"])
    del d["loop"], d["token_side"], d["residual_mult"], d["layers"][0]["mlp"]["shared"]
    d["logit_softcap"], d["layers"][1]["mlp"] = None, None
    for k in ("conv", "q_temp", "bias_max"):
        d["layers"][0]["mixer"][k] = None
    cfg = RZ.RidazenConfig.from_dict(d)
    a, e = cfg.layers[0].mixer, cfg.layers[0].mlp
    assert (a.conv, a.q_temp, a.bias_by, e.shared_ff, e.shared_gate) == (0, None, None, 0, False) and cfg.runs == [0, 1, 2, 3]
    assert (cfg.residual_mult, cfg.token_side, cfg.logit_softcap) == (1.0, 0, 0.0)
    st = RZ.random_state(cfg)
    assert not any("side" in k or k.startswith("l0.mix.rel") or "l0.mlp.shared" in k for k in st)
    eng = ZOO.engine("odd", "cpu", F32)
    eng2 = type(eng)(cfg, RZ.from_state(cfg, st, "cpu", F32), eng.tp, eng.tokenizer, num_blocks=32, max_model_len=128, max_num_seqs=4)
    rp = ZOO.replay("odd", eng2)
    rp.step({(97, 2): 60})
    rp.step({(97, 2): 37})
    want = R.forward(d, {k: v.double() for k, v in st.items()}, ZOO.tokens("odd", 97, 2))
    assert row_errors(rp.logits((97, 2)), want).max() < 5e-5


@pytest.mark.parametrize("edit,msg", [(lambda d: d["layers"][0]["mlp"]["router"].update(top=11), "experts"),
                                      (lambda d: d["layers"][1]["mixer"].update(kv_heads=3), "query heads"),
                                      (lambda d: d["layers"][1]["mixer"].update(bias_max=4), "distance buckets"),
                                      (lambda d: d["layers"][0]["mixer"]["q_temp"].update(every=0), "query temperature"),
                                      (lambda d: d["layers"][0]["mixer"].update(conv=-1), "taps"),
                                      (lambda d: d["loop"].update(stop=5), "cannot run"),
                                      (lambda d: d["loop"].update(start=3), "cannot run"),
                                      (lambda d: d["loop"].update(times=0), "cannot run"),
                                      (lambda d: d["layers"][1].update(type="conv"), "mixer type"),
                                      (lambda d: d["layers"][1]["mlp"].update(kind="sparse"), "feed-forward")])
def test_inconsistent_configurations_are_refused(edit, msg):
    d = copy.deepcopy(CONFIGS["odd"])
    edit(d)
    with pytest.raises(ValueError, match=msg):
        RZ.RidazenConfig.from_dict(d)


def test_misfitting_tensors_and_prefix_caching_are_refused():
    _, cfg, st, _ = ZOO.model("odd")
    for name in ("l0.mlp.e3.up", "l1.mix.rel", "side.embed", "l3.side.proj"):
        with pytest.raises(ValueError, match=name):
            RZ.from_state(cfg, {**st, name: st[name][:-1]}, "cpu", F32)
    with pytest.raises(ValueError, match="l0.mix.v.conv"):
        RZ.from_state(cfg, {**st, "l0.mix.v.conv": st["l0.mix.v.conv"][:, :-1]}, "cpu", F32)
    with pytest.raises(ValueError, match="prefix caching"):
        ZOO.engine("odd", "cpu", F32, enable_prefix_caching=True)


@pytest.mark.parametrize("device,dtype,t", WHOLE)
def test_trace_run_command(tmp_path, device, dtype, t):
    name = "odd"
    _, cfg, st, _ = ZOO.model(name)
    RZ.save_checkpoint(cfg, st, tmp_path / "m")
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
