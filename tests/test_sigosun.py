"""Sigosun against its plain implementation (tests/ref_sigosun.py): each mechanism alone, then whole models through the
engine in every kind of schedule. CPU runs use the ops' PyTorch restatements, GPU runs the kernels."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from dlti_b200.models.stack import AttentionMixer, Rope, Sections, round8
from dlti_b200.ops import _lib
from tests.sigosun_util import (CONFIGS, K, R, SG, ZOO, Replay, check, engine, mixed_schedule, model, mutated, oracle, random,
                                random_portions, row_errors, rows_for, tokens)

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


def rnd(g, *s, dtype=BF16):
    """Random values that every compute dtype represents."""
    return torch.randn(*s, generator=g).to(dtype)


def acts(x, device, dtype):
    """x as an activation view (row pitch a multiple of 8)."""
    out = K.act(x.shape[0], x.shape[1], dtype, device)
    out.copy_(x)
    return out


# ---- mechanisms alone --------------------------------------------------------------------------------------
@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("d", [100, 136, 1031, 4096])
def test_norm_and_residual(device, dtype, d):
    g = gen(d)
    y, x, w = rnd(g, 5, d), torch.randn(5, d, generator=g), rnd(g, d) * 0.3
    want = x.double() + R.rms_norm(y.double(), w.double(), 1e-3, one_plus=True)
    xd = x.to(device)
    xa = K.post_norm_add_(acts(y, device, dtype), xd, w.float().to(device), 1e-3, True, dtype)
    assert rel(xd, want) < 1e-6 and rel(xa, want) < tol(dtype, 1e-6, 4e-3)
    idx = torch.tensor([4, 0, 4], device=device)
    out = K.rms_rows(xd, idx, w.float().to(device), 1e-3, True, dtype)
    assert rel(out, R.rms_norm(want[[4, 0, 4]], w.double(), 1e-3, one_plus=True)) < tol(dtype, 1e-6, 4e-3)


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("ff", [1, 61, 264])
def test_squared_relu(device, dtype, ff):
    u = rnd(gen(ff), 7, ff)
    assert rel(K.relu2(acts(u, device, dtype), ff, dtype), torch.relu(u.double()).square()) < tol(dtype, 1e-6, 4e-3)


@pytest.mark.gpu
@pytest.mark.parametrize("M,ff,K", [(2048, 2048, 264), (2100, 2051, 136), (16384, 200, 64)])
def test_squared_relu_in_the_gemm_epilogue(M, ff, K):
    from dlti_b200.ops.gemm import gemm, gemm_relu2
    g = gen(M)
    x, w = rnd(g, M, K).cuda(), torch.zeros(round8(ff), K, dtype=BF16)
    w[:ff] = rnd(g, ff, K) * 0.1
    h = gemm_relu2(x, w.cuda(), ff)
    want = torch.relu(gemm(x, w.cuda()).float()[:, :ff]).square().to(BF16)
    assert h.shape == (M, ff) and float((h.float() - want.float()).abs().max()) <= 0.02 * float(want.float().abs().max())
    assert rel(h, torch.relu(x.double().cpu() @ w.double().t()[:, :ff]).square()) < 6e-3
    assert gemm_relu2(x[:300], w.cuda(), ff) is None


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("n,groups", [(48, 1), (48, 3), (60, 5), (96, 4), (2048, 1), (1040, 2)])
def test_gated_norms(device, dtype, n, groups):
    g = gen(n)
    y, z, w = rnd(g, 6, n), rnd(g, 6, n) * 2, rnd(g, n)
    y[:, :n // groups] *= 8                                       # parts of unequal size: each has its own mean square
    yd, zd, wd = y.double(), z.double(), w.double()
    v = (yd * R.silu(zd)).view(6, groups, -1)
    first = (v / torch.sqrt((v * v).mean(-1, keepdim=True) + 1e-5)).view(6, n) * wd
    dev = lambda t: acts(t, device, dtype)
    assert rel(K.gated_norm(dev(y), dev(z), w.float().to(device), 1e-5, groups, True), first) < tol(dtype, 2e-6, 4e-3)
    if groups == 1:
        last = R.rms_norm(yd, wd, 1e-5) * torch.sigmoid(zd)
        assert rel(K.gated_norm(dev(y), dev(z), w.float().to(device), 1e-5, 1, False), last) < tol(dtype, 2e-6, 4e-3)


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("dim,vdim,rot,own", [(22, 18, 10, True), (64, 64, 64, True), (64, 64, 20, True), (128, 128, 128, True),
                                              (256, 256, 128, True), (40, 24, 40, True), (128, 128, 32, False), (22, 18, 22, False)])
def test_head_norm_rotation_and_cache_write(device, dtype, dim, vdim, rot, own):
    H, G, bs, eps = 6, 2, 16, 1e-4
    m = AttentionMixer(H, G, dim, vdim, 1.0, Rope(rot, 3e4), kv_from=None if own else 0)
    rows, nb = rows_for([(700, 1), (33, 40), (0, 3)], 1, bs, device)
    T, g = rows.pos.numel(), gen(dim)
    sec = Sections(q=H * dim, **({"k": G * dim, "v": G * vdim} if own else {}), g=H)
    x = torch.zeros(T, sec.total, dtype=BF16)
    for k, (o, n) in sec.at.items():
        x[:, o:o + n] = rnd(g, T, n)
    qn, kn = rnd(g, dim), rnd(g, dim)
    kc = torch.zeros(nb, bs, G, round8(dim), dtype=dtype, device=device)
    vc = torch.zeros(nb, bs, G, round8(vdim), dtype=dtype, device=device)
    before = kc.clone()
    q, gate = K.qk_norm_rope_cache(x.to(device, dtype), sec, m, qn.float().to(device), kn.float().to(device) if own else None, eps, rows,
                                   K.rope_tables(800, rot, 3e4, device), kc, vc, dtype)
    xd, pos = x.double(), rows.pos.cpu()
    prep = lambda s, h, w: R.rotate_pairs(R.rms_norm(xd[:, sec[s]:sec[s] + h * dim].view(T, h, dim), w.double(), eps), pos, 3e4, rot)
    t = tol(dtype, 2e-6, 4e-3)
    assert rel(q.view(T, H, -1)[..., :dim], prep("q", H, qn)) < t
    assert rel(gate, torch.sigmoid(xd[:, sec["g"]:sec["g"] + H])) < 1e-6
    if own:
        sl = rows.slots.cpu()
        kf, vf = kc.cpu().view(-1, G, kc.shape[3]), vc.cpu().view(-1, G, vc.shape[3])
        assert rel(kf[sl][..., :dim], prep("k", G, kn)) < t
        assert torch.equal(vf[sl][..., :vdim].double(), xd[:, sec["v"]:sec["v"] + G * vdim].view(T, G, vdim))
        untouched = torch.ones(nb * bs, dtype=torch.bool)
        untouched[sl] = False
        assert not kf[untouched].any() and not kf[..., dim:].any()
    else:
        assert torch.equal(kc, before)


def _attention_case(device, dtype, H, G, dim, vdim, chunk, lens, nd, spike=None, bs=16):
    """Paged attention over lens = [(start, n)] beside the oracle on whole sequences. spike(q, k): makes scores stand out."""
    rows, nb = rows_for(lens, nd, bs, device)
    g = gen(H * dim + chunk)
    m = AttentionMixer(H, G, dim, vdim, dim ** -0.5, None, chunk)
    kc = torch.full((nb, bs, G, round8(dim)), 7.0)               # pages hold leftovers of other sequences
    vc = torch.full((nb, bs, G, round8(vdim)), -9.0)
    qs, wants = [], []
    tabs = rows.tables.cpu()
    for i, (s, n) in enumerate(lens):
        L = s + n
        q, k, v = rnd(g, L, H, dim), rnd(g, L, G, dim), rnd(g, L, G, vdim)
        if spike:
            spike(q, k)
        j = torch.arange(L)
        sl = tabs[i, j // bs].long() * bs + j % bs
        kc.view(-1, G, kc.shape[3])[sl, :, :dim] = k.float()
        vc.view(-1, G, vc.shape[3])[sl, :, :vdim] = v.float()
        qs.append(q[s:])
        wants.append(R.softmax_attention(q.double(), k.double(), v.double(), m.scale, chunk or None)[s:])
    kc[..., dim:], vc[..., vdim:] = 0, 0
    q = torch.cat(qs)
    T = q.shape[0]
    qb = torch.zeros(T, H, round8(dim), dtype=dtype)
    qb[..., :dim] = q
    gate = torch.rand(T, H, generator=g)
    out = K.paged_attention(qb.view(T, -1).to(device), m, rows, kc.to(device, dtype), vc.to(device, dtype), gate.to(device))
    want = (torch.cat(wants) * gate.double()[:, :, None]).reshape(T, -1)
    e = (out.double().cpu() - want).norm(dim=1) / want.norm(dim=1)
    assert e.max() < tol(dtype, 1e-5, 6e-3), (float(e.max()), int(e.argmax()))


SHAPES = [(6, 2, 22, 18), (4, 2, 64, 64), (3, 3, 128, 72), (5, 1, 40, 136), (2, 1, 256, 200)]


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("H,G,dim,vdim", SHAPES)
@pytest.mark.parametrize("chunk", [0, 1, 37, 64])
def test_paged_attention(device, dtype, H, G, dim, vdim, chunk):
    _attention_case(device, dtype, H, G, dim, vdim, chunk, [(130, 1), (0, 1), (63, 1), (64, 1), (0, 75), (60, 9), (15, 2), (36, 3)], 4)


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("key,query", [(0, 63), (0, 64), (63, 64), (64, 127), (64, 130), (127, 128), (15, 16), (5, 130), (129, 130), (128, 140)])
def test_one_key_stands_out(device, dtype, key, query):
    """Chunks of 64: one query / key pair has a score far above the others, so seeing a key too many or too few shows."""
    def spike(q, k):
        if query < q.shape[0]:
            k[key, :, 0] = 30
            q[query, :, 0] = 30
    n = 141
    for chunk in (64, 0):
        _attention_case(device, dtype, 4, 2, 64, 64, chunk, [(query, 1), (0, n), (query - query % 16, n - query + query % 16)], 1, spike)


@pytest.mark.gpu
@pytest.mark.parametrize("H,G,rep_dim", [(48, 1, 64), (20, 2, 128)])
def test_decode_splits_and_many_heads_on_one_key_head(H, G, rep_dim):
    bs = 16
    lens = [(5, 1), (777, 1), (64, 1), (1023, 1)]
    rows, nb = rows_for(lens, 4, bs, "cuda")
    m = AttentionMixer(H, G, rep_dim, rep_dim, rep_dim ** -0.5, None, 500)
    g = gen(H)
    q, kc, vc = (rnd(g, *s).cuda() for s in ((4, H * rep_dim), (nb, bs, G, rep_dim), (nb, bs, G, rep_dim)))
    want = K.paged_attention_ref(q.cpu().float(), m, K.Rows(*[t.cpu() if torch.is_tensor(t) else t for t in vars(rows).values()]),
                                 kc.cpu().float(), vc.cpu().float(), None)
    for splits in (1, 2, 5, 32):
        out = K.attn_paged_decode(q, m, rows, kc, vc, None, K.act(4, H * rep_dim, BF16, "cuda"), splits=splits)
        assert rel(out, want.double()) < 4e-3


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("C,taps", [(20, 3), (64, 4), (13, 1), (136, 2), (40, 6)])
def test_convolution_over_portions(device, dtype, C, taps):
    """Inputs of earlier portions come from the state; portions shorter than the taps keep older ones."""
    g = gen(C)
    cuts = [[1, 1, 1, 2, 30, 1, 3, 70], [40, 2, 2, 1, 1, 60], [3, 1, 1]]
    col, w, b = 8, rnd(g, C, taps), rnd(g, C)
    xs = [rnd(g, sum(c), C) for c in cuts]
    want = [R.silu(R.causal_conv(x.double(), w.double(), b.double())) for x in xs]
    wt = torch.zeros(taps, round8(C))
    wt[:, :C] = w.t().float()
    bt = torch.zeros(round8(C))
    bt[:C] = b.float()
    conv = torch.full((len(cuts), taps - 1, C), 5.0, dtype=dtype, device=device) if taps > 1 else None
    ssm = torch.zeros(len(cuts), 1, 8, 8, device=device)
    at, got = [0] * len(cuts), [[] for _ in cuts]
    for i in range(max(map(len, cuts))):
        live = [s for s in range(len(cuts)) if i < len(cuts[s])]
        live.sort(key=lambda s: not (cuts[s][i] == 1 and at[s] > 0))
        nd = sum(cuts[s][i] == 1 and at[s] > 0 for s in live)
        rows, _ = rows_for([(at[s], cuts[s][i]) for s in live], nd, 16, device)
        rows.state = torch.tensor(live, dtype=torch.int32, device=device)
        x = torch.cat([xs[s][at[s]:at[s] + cuts[s][i]] for s in live])
        proj = torch.full((x.shape[0], round8(col + C + 3)), 2.0, dtype=dtype, device=device)
        proj[:, col:col + C] = x.to(device, dtype)
        out, _ = K.short_conv(proj, col, C, wt.to(device), bt.to(device), conv, rows, dtype)
        z = torch.zeros(x.shape[0], 8, dtype=dtype, device=device)
        K.linear_scan(z, z, z, K.Decay(const=torch.ones(1, device=device)), ssm, rows, 1, 1, 8, 8, conv_src=proj, conv_col=col, conv_state=conv)
        o = 0
        for s in live:
            got[s].append(out[o:o + cuts[s][i]].cpu())
            o += cuts[s][i]
            at[s] += cuts[s][i]
    for a, b_ in zip(got, want):
        assert rel(torch.cat(a), b_) < tol(dtype, 2e-6, 5e-3)


@pytest.mark.parametrize("device,dtype", MODES)
@pytest.mark.parametrize("heads,groups,N,P", [(4, 2, 20, 12), (6, 3, 72, 40), (2, 2, 128, 64), (3, 1, 256, 8), (1, 1, 300, 4)])
@pytest.mark.parametrize("kind", ["mamba2", "lightning"])
def test_recurrence_over_portions(device, dtype, heads, groups, N, P, kind):
    """Long and short memories, portions around the 64-token chunk of the prefill kernel, states carried through slots."""
    if kind == "lightning" and groups != heads:
        pytest.skip("lightning heads have their own keys")
    g = gen(N + P)
    cuts = [[64, 1, 1, 63, 17, 2], [130, 1, 40, 1], [1, 1, 2, 65]]
    data = []
    for c in cuts:
        T = sum(c)
        q, k, v = rnd(g, T, groups, N), (rnd(g, T, groups, N).float() * 0.2).bfloat16(), rnd(g, T, heads, P)
        data.append((q, k, v, rnd(g, T, heads)))
    bias, A_log, D = torch.linspace(-6, 0.5, heads), torch.linspace(-0.5, 2.5, heads), rnd(g, heads)
    decay = torch.tensor([0.3, 0.999, 0.9, 0.97, 0.5, 0.99][:heads])
    want = []
    for q, k, v, dt in data:
        if kind == "mamba2":
            step = torch.logaddexp(dt.double() + bias.double(), torch.zeros(1, dtype=torch.float64))
            want.append(R.ssd_recurrence(v.double(), k.double(), q.double(), step, A_log.double(), D.double()))
        else:
            f = lambda x: R.silu(x.double())
            want.append(R.decay_recurrence(f(q), f(k), f(v), decay.double()))
    ssm = torch.full((4, heads, N, P), 3.0, device=device)       # slots hold leftovers
    at, got = [0] * 3, [[] for _ in cuts]
    for i in range(max(map(len, cuts))):
        live = [s for s in range(3) if i < len(cuts[s])]
        live.sort(key=lambda s: not (cuts[s][i] == 1 and at[s] > 0))
        nd = sum(cuts[s][i] == 1 and at[s] > 0 for s in live)
        rows, _ = rows_for([(at[s], cuts[s][i]) for s in live], nd, 16, device)
        rows.state = torch.tensor([(3, 1, 0)[s] for s in live], dtype=torch.int32, device=device)
        part = [torch.cat([data[s][x][at[s]:at[s] + cuts[s][i]] for s in live]).flatten(1) for x in range(4)]
        q, k, v, dt = (acts(x, device, dtype) for x in part)
        dec = K.Decay(const=decay.to(device)) if kind == "lightning" else K.Decay(dt=dt, dt_bias=bias.to(device), A_log=A_log.to(device),
                                                                                 D=D.float().to(device))
        out = K.linear_scan(q, k, v, dec, ssm, rows, heads, groups, N, P, silu=kind == "lightning")
        o = 0
        for s in live:
            got[s].append(out[o:o + cuts[s][i]].cpu())
            o += cuts[s][i]
            at[s] += cuts[s][i]
    for a, b in zip(got, want):
        e = (torch.cat(a).double() - b.flatten(1)).norm(dim=1) / b.flatten(1).norm(dim=1).square().mean().sqrt()
        assert e.max() < tol(dtype, 1e-5, 2e-2), (int(e.argmax()), float(e.max()))
    assert bool((ssm[2] == 3).all())                             # a slot nobody holds stays as it was


# ---- whole models through the engine -----------------------------------------------------------------------
WHOLE = [pytest.param("cpu", F32, 5e-5, id="cpu"), pytest.param("cuda", F32, 5e-5, marks=GPU, id="gpu-f32"),
         pytest.param("cuda", BF16, 0.07, marks=GPU, id="gpu-bf16")]
LENS = [(171, 1), (97, 2), (1, 3), (40, 4), (130, 5)]


@pytest.mark.parametrize("device,dtype,t", WHOLE)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_alone_and_together(name, device, dtype, t):
    eng = engine(name, device, dtype)
    rp = Replay(name, eng)
    for key in LENS:
        rp.step({key: key[0]})
    check(name, rp, t)
    rp2 = Replay(name, eng)
    rp2.step({k: k[0] for k in LENS[:4]})
    check(name, rp2, t)
    assert eng.blocks.num_free == eng.blocks.num_blocks and (eng.slots is None or len(eng.slots.free) == 4)


@pytest.mark.parametrize("device,dtype,t", WHOLE)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_decoding_matches_prefill(name, device, dtype, t):
    """Token by token from the start (across chunk edges) and after a long prompt."""
    eng = engine(name, device, dtype)
    rp = Replay(name, eng)
    for _ in range(97):
        rp.step({(97, 2): 1})
    rp.step({(171, 1): 140})
    for _ in range(31):
        rp.step({(171, 1): 1})
    check(name, rp, t)


@pytest.mark.parametrize("device,dtype,t", WHOLE)
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("sizes", [(2,), (3, 16, 64), (65, 80, 2, 1), (70,)], ids=str)
def test_portions(name, device, dtype, t, sizes):
    eng = engine(name, device, dtype)
    rp = Replay(name, eng)
    for c in random_portions(171, random.Random(len(sizes)), sizes):
        rp.step({(171, 1): c})
    check(name, rp, t)


@pytest.mark.parametrize("device,dtype,t", WHOLE)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_mixed_batches_with_pages_and_slots_used_again(name, device, dtype, t):
    """More requests than slots, a pool that only just holds the live ones: everything is handed out several times."""
    eng = engine(name, device, dtype, num_blocks=34)
    rp = Replay(name, eng)
    keys = LENS + [(97, 6), (171, 7), (23, 8), (64, 9)]
    for st in mixed_schedule(keys, random.Random(5), (2, 3, 16, 29, 64, 70)):
        rp.step(st)
    check(name, rp, t)
    assert eng.blocks.num_free == 34


@pytest.mark.gpu
@pytest.mark.parametrize("name", list(CONFIGS))
def test_packed_and_paged_prompt_attention_agree(name):
    out = []
    for pack in (True, False):
        eng = engine(name, "cuda", BF16)
        eng.runner.pack_prompts = pack
        rp = Replay(name, eng)
        for c in (100, 71):
            rp.step({(171, 1): c, (172, 2): c})
        out.append(torch.cat([rp.logits((171, 1)), rp.logits((172, 2))]))
    assert row_errors(out[0], out[1].double()).max() < 0.05


@pytest.mark.parametrize("name,edit", [("odd", dict(layer=0, mask={"size": 38})), ("odd", dict(layer=0, mask={"size": 36})),
                                       ("odd", dict(layer=2, mask={"size": 37})), ("odd", dict(layer=0, rot={"base": 1e4, "dims": 12})),
                                       ("odd", dict(layer=1, norm_groups=1)), ("odd", dict(layer=3, decay=[0.4, 0.93, 0.99])),
                                       ("wide", dict(layer=2, scale=0.1)), ("wide", dict(layer=4, mask={"size": 112}))])
def test_a_wrong_constant_shows(name, edit):
    """The comparisons above can fail: the oracle with one constant off is thousands of fp32 tolerances away."""
    _, _, _, w = model(name)
    bad = R.forward(mutated(name, **edit), w, tokens(name, 171, 1))
    assert row_errors(bad, oracle(name, 171, 1)).max() > 0.05


def test_residual_stream_after_every_layer():
    d, _, _, w = model("odd")
    eng = engine("odd", "cpu", F32)
    eng.runner.trace = []
    Replay("odd", eng).step({(40, 4): 40})
    want = []
    R.forward(d, w, tokens("odd", 40, 4), want)
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
    eng = ZOO.check_generation("ones", device, num_blocks=6, max_len=128)
    assert eng.sched.num_preemptions > 0


@pytest.mark.gpu
def test_bf16_generation_uses_graphs_and_matches_replay():
    """Sampling bf16 logits: each generated token is the argmax of the logits that replaying the same tokens gives, up to
    ties within the rounding of the two schedules."""
    from dlti_b200.serve.params import SamplingParams
    name = "wide"
    eng = engine(name, "cuda", BF16)
    prompts = [tokens(name, n, 40 + n) for n in (90, 7, 130)]
    n0 = _lib.launch_count()
    outs = eng.generate(prompts, SamplingParams(max_tokens=40, temperature=0.0, ignore_eos=True))
    assert eng.graphs and _lib.launch_count() > n0
    from dlti_b200.serve.params import Request
    for p, o in zip(prompts, outs):
        seq = p + o["token_ids"]
        lg = eng.replay_step([(r := Request("x", [], SamplingParams()), seq[:-1], list(range(len(p) - 1, len(seq) - 1)))])
        eng.replay_end(r)
        gap = lg.max(1).values - lg[torch.arange(40), torch.tensor(o["token_ids"])]
        assert gap.max() < 0.15 * lg.std()


def test_sampling_parameters_reach_the_sampler():
    from dlti_b200.serve.params import SamplingParams
    eng = engine("ones", "cpu", F32)
    sp = SamplingParams(max_tokens=12, temperature=1.0, top_k=5, seed=7, ignore_eos=True)
    a, b = (eng.generate([tokens("ones", 9, 1)], sp)[0]["token_ids"] for _ in range(2))
    c = eng.generate([tokens("ones", 9, 1)], SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True))[0]["token_ids"]
    assert a == b and a != c


# ---- configuration, loading, command line ------------------------------------------------------------------
def test_registry_config_and_checkpoint_round_trip(tmp_path):
    from dlti_b200.models.config import LlamaConfig, resolve_config
    from dlti_b200.models.registry import family_of
    d, cfg, st, _ = model("odd")
    SG.save_checkpoint(cfg, st, tmp_path)
    c = resolve_config(str(tmp_path))
    assert isinstance(c, SG.SigosunConfig) and c.layers == cfg.layers and json.load(open(tmp_path / "config.json")) == d
    fam = family_of(c)
    w = fam.load_weights(c, tmp_path, "cpu", F32)
    for name, dst in SG.named_tensors(w):
        got = torch.cat(dst) if isinstance(dst, list) else dst
        assert torch.equal(got, st[name].float()), name
    assert c.num_params() >= sum(t.numel() for t in st.values())
    assert isinstance(resolve_config("tiny"), LlamaConfig) and family_of(resolve_config("tiny")).name == "LlamaForCausalLM"
    assert isinstance(resolve_config("sigosun-tiny"), SG.SigosunConfig)


@pytest.mark.parametrize("edit,msg", [(dict(layer=2, kv_from=1), "kv_from"), (dict(layer=0, kv_heads=4), "query heads"),
                                      (dict(layer=0, rot={"base": 1e4, "dims": 24}), "rotary"), (dict(layer=1, norm_groups=7), "norm_groups"),
                                      (dict(layer=3, decay=[0.5]), "decays")])
def test_inconsistent_configurations_are_refused(edit, msg):
    with pytest.raises(ValueError, match=msg):
        SG.SigosunConfig.from_dict(mutated("odd", **edit))


def test_misfitting_tensor_and_unknown_family_are_refused(tmp_path):
    from dlti_b200.models.config import resolve_config
    _, cfg, st, _ = model("odd")
    with pytest.raises(ValueError, match="l0.mix.k"):
        SG.from_state(cfg, {**st, "l0.mix.k": st["l0.mix.k"][:-1]}, "cpu", F32)
    (tmp_path / "config.json").write_text('{"architecture": "Nothing"}')
    with pytest.raises(ValueError, match="Nothing"):
        resolve_config(str(tmp_path))
    with pytest.raises(ValueError, match="float32"):
        SG.from_state(cfg, st, "cpu", torch.float16)
    with pytest.raises(ValueError, match="prefix caching"):
        engine("odd", "cpu", F32, enable_prefix_caching=True)


def test_prefix_caching_is_open_to_stateless_stacks():
    """A model of this family without recurrent layers may share pages of a common prefix."""
    from dlti_b200.serve.params import SamplingParams
    eng = engine("tall", "cpu", F32, enable_prefix_caching=True)
    p = tokens("tall", 50, 3)
    sp = SamplingParams(max_tokens=4, temperature=0.0, ignore_eos=True)
    want = ZOO.greedy("tall", p, 4)
    assert eng.generate([p], sp)[0]["token_ids"] == want and eng.generate([p], sp)[0]["token_ids"] == want
    assert eng.blocks.hits >= 48


def test_replay_refuses_what_does_not_fit():
    from dlti_b200.serve.params import Request, SamplingParams
    eng = engine("ones", "cpu", F32, num_blocks=4, max_len=64)
    r = Request("a", [], SamplingParams())
    with pytest.raises(ValueError, match="vocabulary"):
        eng.replay_step([(r, [1, 96], [])])
    with pytest.raises(ValueError, match="longer"):
        eng.replay_step([(r, [1] * 65, [])])
    eng.replay_step([(r, [1] * 60, [])])
    with pytest.raises(RuntimeError, match="pages"):
        eng.replay_step([(Request("b", [], SamplingParams()), [1, 2], [])])


@pytest.mark.parametrize("device,dtype,t", WHOLE)
def test_trace_run_command(tmp_path, device, dtype, t):
    name = "odd"
    _, cfg, st, _ = model(name)
    SG.save_checkpoint(cfg, st, tmp_path / "m")
    a, b = tokens(name, 97, 2), tokens(name, 40, 4)
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
    wa, wb = oracle(name, 97, 2), oracle(name, 40, 4)
    for s, want in ((0, wa[[49, 3]]), (1, torch.stack([wb[39], wa[50], wa[89]])), (7, torch.stack([wa[91], wb[0]]))):
        assert row_errors(read(s), want).max() < t
    assert not (tmp_path / "o" / "2.f32").exists()


def test_trace_run_replays_llama_too(tmp_path):
    """The runner picks the family by config.json: the same steps through a Llama checkpoint, cut in two ways."""
    from dlti_b200.models.config import PRESETS
    from dlti_b200.models.hf_io import resident_state_dict, save_hf_checkpoint
    from dlti_b200.models.llama import ResidentWeights
    from dlti_b200.serve.replay import build_engine, run
    cfg = PRESETS["tiny-gqa"]
    save_hf_checkpoint(cfg, resident_state_dict(ResidentWeights.random_init(cfg, "cpu", F32, seed=1)), tmp_path)
    toks, out = list(range(5, 45)), []
    for cuts in ([40], [13, 1, 20, 1, 5]):
        eng = build_engine(str(tmp_path), "float32", 128, "cpu")
        a, steps = 0, []
        for i, c in enumerate(cuts):
            steps.append(json.dumps({"step": i, "entries": [{"id": "x", "tokens": toks[a:a + c], "want": list(range(c))}], "end": []}))
            a += c
        seen = []
        run(eng, steps, str(tmp_path), seen.append)
        assert seen == [f"done {i}" for i in range(len(cuts))]
        out.append(np.concatenate([np.fromfile(tmp_path / f"{i}.f32", dtype="<f4") for i in range(len(cuts))]))
    assert np.abs(out[0] - out[1]).max() < 1e-4
