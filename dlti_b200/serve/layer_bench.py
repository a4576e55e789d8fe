"""Serving throughput of a layer-stack family beside the closest other family at equal size, and the time of each kernel of
the two against its roofline: Sigosun beside Llama (`bench.py --workload sigosun`), Logozen and Latanex beside Sigosun
(`--workload logozen`, `--workload latanex`), Ridazen beside Latanex (`--workload ridazen`). Random weights; layer sizes of real models. A mixture of experts counts with
the parameters that a token uses, a layer that runs several times with those of every run.

Steps go through LLMEngine.pack_step / _run_step (packing, host-to-device copy, forward, sampling; decode steps replay
CUDA graphs), timed with CUDA events. Kernels are timed one call at a time with the L2 overwritten before each."""
from __future__ import annotations

import json
import statistics
from dataclasses import replace

import torch

from ..models.config import LlamaConfig
from ..models.registry import family_of
from ..models.latanex import LatanexConfig
from ..models.logozen import LogozenConfig
from ..models.ridazen import RidazenConfig
from ..models.sigosun import SigosunConfig
from ..models.stack import (AttentionMixer, DeltaMixer, DenseMlp, DistanceBias, LatentAttentionMixer, Layer, LightningMixer, Loop, Mamba2Mixer,
                            MLstmMixer, MoeMlp, QueryTemp, Rope, StackWeights, mixer_sections, mlp_sections, round8)
from ..ops import _lib
from ..ops import attention as A
from ..ops import delta as DR
from ..ops import dyt as TN
from ..ops import elementwise as E
from ..ops import latent as LA
from ..ops import moe as ME
from ..ops import prenorm as PN
from ..ops import serving as S
from ..ops import stack as K
from ..ops import streams as HS
from ..ops.gemm import gemm, gemm_relu2, gemm_skinny, gemm_skinny_acc
from .engine import LLMEngine, _pieces, chunk_pieces
from .model_runner import TPContext
from .tokenizer import ByteTokenizer


def _sigosun(width: int, blocks: int) -> SigosunConfig:
    heads = width // 128
    att = AttentionMixer(heads=heads, kv_heads=max(1, heads // 4), dim=128, vdim=128, scale=128 ** -0.5, rope=Rope(128, 5e5), chunk=2048)
    mam = Mamba2Mixer(heads=width // 32, vdim=64, state=128, groups=1, conv=4, norm_groups=1)
    lig = LightningMixer(heads=heads, dim=128, vdim=128, decay=tuple(1 - 2.0 ** (-4 - h * 5 / heads) for h in range(heads)))
    ff = DenseMlp(4 * width)
    layers = []
    for b in range(blocks):
        layers += [Layer(att, ff), Layer(replace(att, kv_from=4 * b), ff), Layer(mam, None), Layer(lig, None)]
    return SigosunConfig(hidden_size=width, vocab_size=32000, norm_eps=1e-6, layers=layers, name=f"sigosun-{width}x{4 * blocks}")


def _logozen(width: int, params: int) -> LogozenConfig:
    """Pairs of layers (mLSTM, latent attention), each with a feed-forward, that together hold about `params` parameters."""
    heads = width // 128
    att = LatentAttentionMixer(heads=heads, dim=64, rot_dim=64, vdim=128, kv_rank=512, scale=128 ** -0.5, rope=Rope(64, 1e6))
    mem = MLstmMixer(heads=heads // 2, dim=128, vdim=256, gate_cap=15.0)
    ff = DenseMlp(4 * width, act="polynorm")

    def cfg(n):
        return LogozenConfig(hidden_size=width, vocab_size=32000, norm_eps=1e-6, norm_one_plus=False, streams=4, canon=4, embed_scale=45.0,
                             layers=[Layer(mem, ff), Layer(att, ff)] * n, name=f"logozen-{width}x{2 * n}")
    one = cfg(2).num_params() - cfg(1).num_params()
    return cfg(max(1, round(params / one)))


def _latanex(width: int, params: int) -> LatanexConfig:
    """Pairs of layers (delta rule, windowed attention), each with a mixture of experts, of which a token uses about `params`
    parameters."""
    heads = width // 128
    att = AttentionMixer(heads=heads, kv_heads=max(1, heads // 4), dim=128, vdim=128, scale=128 ** -0.5, qk_norm=False, head_gate=False,
                         window=2048, softcap=30.0, sink=True, bias=True, row_norm=True, v_mix=True)
    mem = DeltaMixer(heads=heads, kv_heads=heads, dim=128, vdim=128, conv=4)
    moe = MoeMlp(experts=64, top=8, ff=width // 4, limit=7.0, groups=8, keep=4, scale=2.5, shared_ff=width // 2, shared_limit=7.0)

    def cfg(n):
        return LatanexConfig(hidden_size=width, vocab_size=32000, norm_eps=1e-6, norm_one_plus=False, tanh_norms=True, embed_scale=4.0,
                             logit_scale=0.5, layers=[Layer(mem, moe), Layer(att, moe)] * n, name=f"latanex-{width}x{2 * n}")
    one = active_params(cfg(2)) - active_params(cfg(1))
    return cfg(max(1, round(params / one)))


def _ridazen(width: int, params: int) -> RidazenConfig:
    """Attention layers with mixtures of experts, the second and third of them run twice; a token uses about `params` parameters."""
    heads = width // 128
    att = AttentionMixer(heads=heads, kv_heads=max(1, heads // 4), dim=128, vdim=128, scale=128 ** -0.5, head_gate=False, conv=4,
                         q_temp=QueryTemp(0.1, 1024), bias_by=DistanceBias(32, 128), out_gate=True)
    moe = MoeMlp(experts=64, top=8, ff=width // 4, act="relu2", score="softmax", shared_ff=width // 2, shared_gate=True)

    def cfg(n):
        return RidazenConfig(hidden_size=width, vocab_size=32000, norm_eps=1e-6, norm_one_plus=False, pre_norm=True, residual_mult=0.7, token_side=128,
                             loop=Loop(1, 3, 2), logit_scale=0.5, logit_softcap=30.0, layers=[Layer(att, moe)] * n, name=f"ridazen-{width}x{n}")
    one = active_params(cfg(5)) - active_params(cfg(4))
    return cfg(max(4, 4 + round((params - active_params(cfg(4)) + 2 * 32000 * width) / one)))


def active_params(cfg) -> int:
    """Parameters that one token uses, those of a layer once per run."""
    layers = getattr(cfg, "layers", [])
    idle = [(e.experts - e.top) * (3 if e.gated else 2) * e.ff * cfg.hidden_size if isinstance(e := l.mlp, MoeMlp) else 0 for l in layers]
    n = cfg.num_params() - sum(idle)
    if layers and (cfg.loop is not None or cfg.token_side):
        w = StackWeights(cfg, "meta", torch.bfloat16)
        n -= 0 if w.side_embed is None else w.side_embed.numel() - w.side_embed.shape[1]
        own = [sum(t.numel() for t in lw.values()) - x for lw, x in zip(w.layers, idle)]
        n += sum(own[j] for j in cfg.runs) - sum(own)
    return n


def experts_hit(e: MoeMlp, rows: int) -> float:
    """Experts that `rows` tokens reach when all are equally likely."""
    return e.experts * (1 - (1 - e.top / e.experts) ** rows)


def _llama(width: int, params: int) -> LlamaConfig:
    """The Llama of the same width whose layers hold about `params` parameters (same key/value head ratio)."""
    heads = width // 128
    c = LlamaConfig(hidden_size=width, intermediate_size=round(width * 2.6875 / 256) * 256, num_attention_heads=heads,
                    num_key_value_heads=max(1, heads // 4), num_hidden_layers=1, max_position_embeddings=16384)
    n = max(1, round(params / c.params_per_layer()))
    return replace(c, num_hidden_layers=n, name=f"llama-{width}x{n}")


def _engine(cfg, max_len: int, seqs: int):
    w = family_of(cfg).random_weights(cfg, "cuda", torch.bfloat16, 0)
    return LLMEngine(cfg, w, TPContext(), ByteTokenizer(cfg.vocab_size), num_blocks=seqs * (max_len // 16) + 64, max_num_seqs=seqs,
                     max_num_batched_tokens=16384, max_model_len=max_len)


def _time(fn, warmup: int, iters: int) -> float:
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    for _ in range(iters):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / iters


def _greedy(n: int):
    return ([0.0] * n, [0] * n, [1.0] * n, [0] * n)


def prefill_ms(eng: LLMEngine, nseq: int, length: int, warmup: int, iters: int) -> float:
    bs = eng.blocks.block_size
    per = -(-length // bs)
    T = nseq * length
    ids = torch.randint(3, eng.cfg.vocab_size, (T,)).tolist()
    pos = list(range(length)) * nseq
    slots = [(i * per) * bs + p for i in range(nseq) for p in range(length)]
    tabs = [list(range(i * per, (i + 1) * per)) for i in range(nseq)]
    cu = [i * length for i in range(nseq + 1)]
    full = eng.per_sequence
    step = lambda: eng.pack_step(0, ids, pos, slots, [length] * nseq if full else [], tabs if full else [], cu, length, _greedy(nseq),
                                 sslots=list(range(nseq)), starts=[0] * nseq)
    return _time(lambda: eng._run_step(step()), warmup, iters)


def decode_ms(eng: LLMEngine, batch: int, ctx: int, warmup: int, iters: int) -> float:
    bs = eng.blocks.block_size
    per = -(-(ctx + 1) // bs)
    ids = torch.randint(3, eng.cfg.vocab_size, (batch,)).tolist()
    tabs = [list(range(i * per, (i + 1) * per)) for i in range(batch)]
    slots = [t[ctx // bs] * bs + ctx % bs for t in tabs]
    step = lambda: eng.pack_step(batch, ids, [ctx] * batch, slots, [ctx + 1] * batch, tabs, [], 0, _greedy(batch),
                                 sslots=list(range(batch)))
    return _time(lambda: eng._run_step(step()), warmup, iters)


def step_bytes(eng: LLMEngine, batch: int, ctx: int) -> int:
    """What a decode step must move: every matrix that the rows reach once, the visible keys and values, recurrent states read and
    written."""
    cfg, w = eng.cfg, eng.w
    size = lambda t: t.numel() * t.element_size()
    runs = cfg.runs if eng.per_sequence else range(len(w.layers))
    n = sum(size(t) for j in runs for t in w.layers[j].values()) + size(w.lm_head)
    if not eng.per_sequence:
        return n + 2 * 2 * cfg.num_hidden_layers * batch * (ctx + 1) * w.KV * cfg.head_dim
    for i, j in enumerate(runs):
        l = cfg.layers[j]
        m = l.mixer
        if isinstance(l.mlp, MoeMlp):
            n -= int((1 - experts_hit(l.mlp, batch) / l.mlp.experts) * (size(w.layers[j]["e_up"]) + size(w.layers[j]["e_down"])))
        if eng.states is not None and eng.states.canon[i] is not None:
            n += 2 * batch * size(eng.states.canon[i][:, 0])
        if isinstance(m, LatentAttentionMixer):
            n += 2 * batch * (ctx + 1) * m.cols
        elif isinstance(m, AttentionMixer):
            seen = ctx + 1 - (ctx // m.chunk * m.chunk if m.chunk else max(0, ctx + 1 - m.window) if m.window else 0)
            n += 2 * batch * seen * m.kv_heads * (m.dim + m.vdim)
            if m.conv > 1:
                n += 2 * 2 * batch * eng.states.conv[i][0].numel()
        else:
            n += 2 * batch * 4 * (eng.states.ssm[i][0].numel() + (0 if eng.states.vec[i] is None else eng.states.vec[i][0].numel()))
    return n


# ---- kernels -----------------------------------------------------------------------------------------------
class _Kernels:
    def __init__(self, peaks: dict, iters: int):
        self.hbm, self.flops, self.iters = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12, iters
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
        self.rows: list[dict] = []

    def run(self, model: str, phase: str, name: str, fn, nbytes: float, flops: float = 0.0):
        for _ in range(3):
            fn()
        ts = []
        for _ in range(self.iters):
            self.flush.fill_(1)
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            ts.append(e0.elapsed_time(e1) * 1e3)
        us = statistics.median(ts)
        roof = max(nbytes / self.hbm, flops / self.flops) * 1e6
        self.rows.append({"model": model, "phase": phase, "kernel": name, "us": round(us, 2), "roof_us": round(roof, 2),
                          "frac_of_roof": round(roof / us, 3), "bound": "flops" if flops / self.flops > nbytes / self.hbm else "bytes"})


def _rows(lens, nd, tables, slots, max_ctx):
    i32 = dict(dtype=torch.int32, device="cuda")
    cu = [0]
    for s, n in lens[nd:]:
        cu.append(cu[-1] + n)
    return K.Rows(torch.cat([torch.arange(s, s + n) for s, n in lens]).to(**i32),
                  torch.cat([torch.full((n,), i) for i, (s, n) in enumerate(lens)]).to(**i32), slots,
                  torch.tensor([s + n for s, n in lens], **i32), torch.tensor(cu, **i32) if len(cu) > 1 else None, tables,
                  torch.arange(len(lens), **i32), nd, max([n for _, n in lens[nd:]], default=0), max_ctx)


def kernels(width: int, peaks: dict, nseq: int, length: int, batch: int, ctx: int, iters: int) -> list[dict]:
    """Each kernel of a prefill step of nseq prompts of `length` and of a decode step of `batch` rows at context ctx."""
    k = _Kernels(peaks, iters)
    cfg = _sigosun(width, 1)
    att, mam, lig = cfg.layers[0].mixer, cfg.layers[2].mixer, cfg.layers[3].mixer
    ll = _llama(width, 1)
    dev, bf = "cuda", torch.bfloat16
    H, G, hd, d = att.heads, att.kv_heads, 128, width
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=bf)
    T, bs = nseq * length, 16
    per = -(-max(length, ctx + 1) // bs)
    n_all = max(nseq, batch)
    tabs = torch.arange(n_all * per, dtype=torch.int32, device=dev).view(n_all, per)
    kc, vc = rnd(n_all * per, bs, G, hd), rnd(n_all * per, bs, G, hd)
    fa, qn = torch.ones(hd, device=dev), torch.ones(d, device=dev)
    tab_r = K.rope_tables(max(length, ctx + 1), hd, 5e5, dev)
    cos, sin = E.rope_tables(max(length, ctx + 1), hd, 5e5, dev)
    sec = mixer_sections(att)
    pslots = torch.cat([torch.arange(length) + i * per * bs for i in range(nseq)]).to(dev)
    dslots = torch.tensor([i * per * bs + ctx for i in range(batch)], device=dev)
    pr = _rows([(0, length)] * nseq, 0, tabs[:nseq].contiguous(), pslots, length)
    dr = _rows([(ctx, 1)] * batch, batch, tabs[:batch].contiguous(), dslots, ctx + 1)
    seen = ctx + 1 - ctx // att.chunk * att.chunk

    def pairs(n, c):                                        # visible (query, key) pairs of one prompt
        c = min(c or n, n)
        full, rest = divmod(n, c)
        return full * c * (c + 1) // 2 + rest * (rest + 1) // 2

    # attention, whole prompts: the same number of visible pairs for both (Llama sees pieces of `chunk` as prompts)
    cut = [i * length + s for i in range(nseq) for s in range(0, length, att.chunk)] + [T]
    seg = (torch.tensor(cut, dtype=torch.int32, device=dev), min(length, att.chunk))
    pieces = K.Pieces(seg[0], seg[1], T)
    qkv, gate = rnd(T, (H + 2 * G) * hd), torch.rand(T, H, device=dev)
    fl = 4.0 * nseq * pairs(length, att.chunk) * H * hd
    io = T * (2 * H + 2 * G) * hd * 2
    k.run("sigosun", "prefill", "attention (packed)", lambda: K.packed_attention(qkv, att, pr, pieces, kc, vc, gate), io, fl)
    k.run("llama", "prefill", "attention", lambda: A.attention_fwd(qkv, seg[0], seg[1], H, G, hd, want_lse=False), io, fl)
    q = rnd(T, H * hd)
    out = K.act(T, H * hd, bf, dev)
    k.run("sigosun", "prefill", "attention (paged, heads > 128)", lambda: K.attn_paged_prefill(q, att, pr, kc, vc, gate, out), io, fl)
    # the second half of every prompt, its first half cached
    h = length // 2
    own = _rows([(h, length - h)] * nseq, 0, tabs[:nseq].contiguous(), pslots.view(nseq, -1)[:, h:].reshape(-1), length)
    arr, n_p, longest, ext, prefix = chunk_pieces([i * (length - h) for i in range(nseq + 1)], [h] * nseq, tabs[:nseq].tolist(), bs, att.chunk)
    half = _pieces(torch.from_numpy(arr).to(dev), nseq * (length - h), n_p, longest, ext, prefix)
    packed2 = rnd(ext, (H + 2 * G) * hd)
    k.run("sigosun", "prefill", "attention (packed, half cached)", lambda: K.packed_attention(packed2, att, own, half, kc, vc, gate),
          nseq * ((length - h) * 2 * H + length * 2 * G) * hd * 2, fl - 4.0 * nseq * pairs(h, att.chunk) * H * hd)
    del packed2
    # attention, decode
    qd, gd, od = rnd(batch, H * hd), torch.rand(batch, H, device=dev), K.act(batch, H * hd, bf, dev)
    k.run("sigosun", "decode", "attention", lambda: K.attn_paged_decode(qd, att, dr, kc, vc, gd, od), batch * seen * G * hd * 4)
    lens = torch.full((batch,), seen, dtype=torch.int32, device=dev)
    k.run("llama", "decode", "attention", lambda: S.paged_decode(qd, kc, vc, dr.tables, lens, H, G, hd, max_ctx=seen), batch * seen * G * hd * 4)
    # projection rows -> rotated q, cache
    for phase, r, n in (("prefill", pr, T), ("decode", dr, batch)):
        acc = phase == "decode"
        proj = torch.zeros(n, sec.total, device=dev) if acc else rnd(n, sec.total)
        k.run("sigosun", phase, "q/k norm + rope + cache", lambda: K.qk_norm_rope_cache(
            proj, sec, att, fa, fa, 1e-6, r, tab_r, kc, vc, bf, packed=None if acc else pieces, acc=acc),
            n * (sec.total * (8 if acc else 2) + (H + (0 if acc else 2 * G)) * hd * 2 + 2 * G * hd * 2 + 4 * H))
        W = (H + 2 * G) * hd
        if acc:
            accb = torch.zeros(n, W, device=dev)
            k.run("llama", phase, "rope + cache", lambda: S.acc_rope_cache(accb, bf, r.pos, cos, sin, r.slots, kc, vc, H, G, hd),
                  n * (W * 10 + 2 * G * hd * 2))
        else:
            k.run("llama", phase, "rope + cache", lambda: S.rope_cache_(qkv, r.pos, cos, sin, r.slots, kc, vc, H, G, hd),
                  n * ((H + G) * hd * 4 + G * hd * 2 + 2 * G * hd * 2))
        # residual + norm
        x, w16 = torch.randn(n, d, device=dev), torch.ones(d, device=dev, dtype=bf)
        y = torch.zeros(n, d, device=dev) if acc else rnd(n, d)
        k.run("sigosun", phase, "norm + residual", lambda: K.post_norm_add_(y, x, qn, 1e-6, True, bf, acc=acc),
              n * d * ((8 if acc else 2) + 8 + 2))
        res = rnd(n, d)
        if acc:
            k.run("llama", phase, "residual + norm", lambda: E.acc_add_rmsnorm(y, res, w16, 1e-6), n * d * (8 + 4 + 2))
        else:
            k.run("llama", phase, "residual + norm", lambda: E.rmsnorm_fwd(y, w16, 1e-6, residual=res), n * d * (2 + 4 + 2))
        # activation
        ff, lf = cfg.layers[0].mlp.ff, ll.intermediate_size
        u = torch.zeros(n, ff, device=dev) if acc else rnd(n, ff)
        if not acc:
            a, b = rnd(n, d), rnd(ff, d)
            k.run("sigosun", phase, "GEMM up + relu^2", lambda: gemm_relu2(a, b, ff), 2 * (n * d + ff * d + n * ff), 2.0 * n * ff * d)
        k.run("sigosun", phase, "relu^2", lambda: K.relu2(u, ff, bf, acc=acc), n * ff * ((8 if acc else 2) + 2))
        gu = torch.zeros(n, 2 * lf, device=dev) if acc else rnd(n, 2 * lf)
        if acc:
            k.run("llama", phase, "swiglu", lambda: E.acc_swiglu(gu, bf), n * lf * 18)
        else:
            k.run("llama", phase, "swiglu", lambda: E.swiglu_fwd(gu), n * lf * 6)
    del qkv, q, out, u, gu
    # GEMMs (the same kernels in both models)
    for phase, n in (("prefill", T), ("decode", batch)):
        mm = gemm if phase == "prefill" else gemm_skinny_acc
        for model, name, N_, K_ in (("sigosun", "GEMM attention in", sec.total, d), ("llama", "GEMM qkv", (H + 2 * G) * hd, d),
                                    ("sigosun", "GEMM mamba2 in", mixer_sections(mam).total, d),
                                    ("sigosun", "GEMM lightning in", mixer_sections(lig).total, d),
                                    ("sigosun", "GEMM up", 4 * d, d), ("llama", "GEMM gate_up", 2 * ll.intermediate_size, d),
                                    ("sigosun", "GEMM down", d, 4 * d), ("llama", "GEMM down", d, ll.intermediate_size)):
            a, b = rnd(n, K_), rnd(N_, K_)
            k.run(model, phase, name, lambda: mm(a, b), 2 * (n * K_ + N_ * K_) + n * N_ * (2 if phase == "prefill" else 4), 2.0 * n * N_ * K_)
            if phase == "decode":
                gemm_skinny(a, b)                         # leaves the shared accumulator zero
    # recurrent layers
    sm, sl = mixer_sections(mam), mixer_sections(lig)
    inner, gn, C = mam.inner, mam.groups * mam.state, mam.conv_channels
    cw, cb = torch.rand(mam.conv, C, device=dev), torch.zeros(C, device=dev)
    for phase, r, n, ns in (("prefill", pr, T, nseq), ("decode", dr, batch, batch)):
        conv = torch.zeros(ns, mam.conv - 1, C, device=dev, dtype=bf)
        ssm = torch.zeros(ns, mam.heads, mam.state, mam.vdim, device=dev)
        acc = phase == "decode"
        proj = torch.zeros(n, sm.total, device=dev) if acc else rnd(n, sm.total)
        k.run("sigosun", phase, "short conv", lambda: K.short_conv(proj, sm["xbc"], C, cw, cb, conv, r, bf, acc=acc, width=sm.total),
              n * (sm.total * 10 + C * 2 + (mam.conv - 1) * C * 2) if acc else n * C * 4)
        p16, xbc = rnd(n, sm.total), rnd(n, C)
        dec = K.Decay(dt=p16[:, sm["dt"]:sm["dt"] + mam.heads], dt_bias=torch.full((mam.heads,), -4.0, device=dev),
                      A_log=torch.zeros(mam.heads, device=dev), D=torch.ones(mam.heads, device=dev))
        q64 = 64
        work = lambda h, N_, P_: 2.0 * n * h * (q64 * (N_ + P_) / 2 + 2 * N_ * P_) if phase == "prefill" else 4.0 * n * h * N_ * P_
        k.run("sigosun", phase, "mamba2 scan", lambda: K.linear_scan(
            xbc[:, inner + gn:], xbc[:, inner:inner + gn], xbc[:, :inner], dec, ssm, r, mam.heads, mam.groups, mam.state, mam.vdim,
            conv_src=p16, conv_col=sm["xbc"], conv_state=conv),
            n * (C + inner + mam.heads) * 2 + ns * 8 * ssm[0].numel(), work(mam.heads, mam.state, mam.vdim))
        yb = rnd(n, inner)
        k.run("sigosun", phase, "gated norm (mamba2)", lambda: K.gated_norm(yb, p16[:, :inner], torch.ones(inner, device=dev), 1e-6, 1, True),
              n * inner * 6)
        pl = rnd(n, sl.total)
        st = torch.zeros(ns, lig.heads, lig.dim, lig.vdim, device=dev)
        qk, vv = lig.heads * lig.dim, lig.heads * lig.vdim
        dl = K.Decay(const=torch.tensor(lig.decay, device=dev))
        k.run("sigosun", phase, "lightning silu + scan", lambda: K.linear_scan(
            pl[:, :qk], pl[:, sl["k"]:sl["k"] + qk], pl[:, sl["v"]:sl["v"] + vv], dl, st, r, lig.heads, lig.heads, lig.dim, lig.vdim,
            silu=True), n * (2 * qk + 2 * vv) * 2 + ns * 8 * st[0].numel(), work(lig.heads, lig.dim, lig.vdim))
        k.run("sigosun", phase, "gated norm (lightning)", lambda: K.gated_norm(pl[:, :vv], pl[:, sl["g"]:sl["g"] + vv],
                                                                              torch.ones(vv, device=dev), 1e-6, 1, False), n * vv * 6)
    return k.rows


def logozen_kernels(width: int, peaks: dict, nseq: int, length: int, batch: int, ctx: int, iters: int) -> list[dict]:
    """The kernels of Logozen in the same two steps; those of Sigosun come from kernels()."""
    k = _Kernels(peaks, iters)
    cfg = _logozen(width, 1)
    mem, m, d, dev, bf = cfg.layers[0].mixer, cfg.layers[1].mixer, width, "cuda", torch.bfloat16
    w = StackWeights(cfg, dev, bf).finish()
    lw, w_expand = w.layers[1], w.derived[1]["w_expand"]
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=bf)
    for t in (lw["w_uk"], lw["w_uv"], w_expand, *(l[n] for l in w.layers for n in ("w_in", "w_up"))):
        t.normal_(0, 0.04)
    T, bs, heads, R = nseq * length, 16, m.heads, m.kv_rank
    per = -(-max(length, ctx + 1) // bs)
    n_all = max(nseq, batch)
    tabs = torch.arange(n_all * per, dtype=torch.int32, device=dev).view(n_all, per)
    cache = rnd(n_all * per, bs, 1, m.pitch)
    tab_r = K.rope_tables(max(length, ctx + 1), m.rope.dims, m.rope.base, dev)
    pslots = torch.cat([torch.arange(length) + i * per * bs for i in range(nseq)]).to(dev)
    dslots = torch.tensor([i * per * bs + ctx for i in range(batch)], device=dev)
    pr = _rows([(0, length)] * nseq, 0, tabs[:nseq].contiguous(), pslots, length)
    dr = _rows([(ctx, 1)] * batch, batch, tabs[:batch].contiguous(), dslots, ctx + 1)
    pieces = K.Pieces(torch.tensor([i * length for i in range(nseq + 1)], dtype=torch.int32, device=dev), length, T)
    pairs = length * (length + 1) // 2
    hp = m.head_pitch
    buf, gate, out, lat = rnd(T, 3 * heads * hp), torch.rand(T, heads, device=dev), K.act(T, heads * m.vdim, bf, dev), rnd(T, m.pitch)[:, :m.cols]
    run = lambda phase, name, fn, nbytes, flops=0.0: k.run("logozen", phase, name, fn, nbytes, flops)
    run("prefill", "attention (packed)", lambda: K.attn_fwd_split(buf, m, heads, heads, pieces, gate, out, sink=lw["sink"]),
        T * heads * (2 * m.qk_dim + 2 * m.vdim) * 2, 2.0 * nseq * pairs * heads * (m.qk_dim + m.vdim))
    useful = heads * (m.dim + m.vdim)
    run("prefill", "GEMM latents -> keys, values", lambda: gemm(lat, w_expand, out=buf[:, heads * hp:], two_cta=False),
        2 * (T * m.cols + w_expand.numel() + 2 * T * heads * hp), 2.0 * T * useful * R)
    qa, od = rnd(batch, heads * m.pitch), torch.empty(batch, heads * R, device=dev, dtype=bf)
    gd = torch.rand(batch, heads, device=dev)
    run("decode", "attention", lambda: LA.latent_decode(qa, m, dr, cache, gd, lw["sink"], od), batch * (ctx + 1) * m.cols * 2,
        2.0 * batch * (ctx + 1) * heads * (m.cols + R))
    qn, o = rnd(batch, heads * m.dim), torch.empty(batch, heads * m.vdim, device=dev, dtype=bf)
    run("decode", "queries into the latent space", lambda: LA.head_gemm(qn, m.dim, lw["w_uk"], qa, m.pitch, heads, m.dim, R, True),
        2 * (lw["w_uk"].numel() + qn.numel() + batch * heads * R))
    run("decode", "latent outputs to values", lambda: LA.head_gemm(od, R, lw["w_uv"], o, m.vdim, heads, R, m.vdim, False),
        2 * (lw["w_uv"].numel() + od.numel() + o.numel()))
    sec, sm = mixer_sections(m), mixer_sections(mem)
    S, ff = cfg.streams, cfg.layers[0].mlp.ff
    inner, qk = mem.heads * mem.vdim, mem.heads * mem.dim
    for phase, r, n, ns in (("prefill", pr, T, nseq), ("decode", dr, batch, batch)):
        acc = phase == "decode"
        es = 8 if acc else 2                                      # accumulators are read and zeroed
        z = lambda c: torch.zeros(n, c, device=dev) if acc else rnd(n, c)
        proj = z(sec.total)
        run(phase, "latent norm + rope + cache", lambda: LA.latent_prep(proj, sec, m, lw["kv_norm"], 1e-6, r, tab_r, cache, bf, None if acc else pieces, acc),
            n * (sec.total * es + heads * m.qk_dim * 2 + m.pitch * 2 * (1 if acc else 2) + 4 * heads))
        x, y = torch.randn(n, S, d, device=dev), z(d)
        c = w.layers[0]
        state = torch.zeros(ns, cfg.canon - 1, d, device=dev, dtype=bf)
        run(phase, "streams + norm (+ convolution)" if acc else "streams + norm", lambda: HS.hyper_(
            x, y, c["hc1.mix"], c["hc1.out"], c["hc1.in"], c["norm1"], 1e-6, bf, conv=(c["canon1"], state, r) if acc else None, acc=acc),
            n * d * (es + 8 * S + 2 + (4 * (cfg.canon - 1) if acc else 0)))
        if not acc:
            h = rnd(n, d)
            run(phase, "input convolution", lambda: HS.canon(h, c["canon1"], state, r), n * d * 4)
        u = z(ff)
        run(phase, "PolyNorm", lambda: HS.poly_norm(u, ff, c["act"], 1e-6, bf, acc=acc), n * ff * (es + 2))
        ssm = torch.zeros(ns, mem.heads, mem.dim, mem.vdim, device=dev)
        vec = torch.zeros(ns, mem.heads, K.mlstm_vec(mem.dim, mem.vdim), device=dev)
        p, g = rnd(n, sm["gates"]), torch.randn(n, 2 * mem.heads, device=dev)
        bias = torch.full((2 * mem.heads,), 3.0, device=dev)
        work = 2.0 * n * mem.heads * (32 * (mem.dim + mem.vdim) + 2 * mem.dim * mem.vdim) if not acc else 4.0 * n * mem.heads * mem.dim * mem.vdim
        run(phase, "mLSTM scan", lambda: K.mlstm_scan(p[:, :qk], p[:, sm["k"]:sm["k"] + qk], p[:, sm["v"]:sm["v"] + inner], g, bias, 15.0, ssm, vec, r,
                                                      mem.heads, mem.dim, mem.vdim),
            n * (2 * qk + 2 * inner) * 2 + n * 8 * mem.heads + ns * 8 * (ssm[0].numel() + vec[0].numel()), work)
        yb = rnd(n, inner)
        run(phase, "unit heads + gate", lambda: K.gated_norm(yb, p[:, sm["g"]:sm["g"] + inner], c["norm"], 1e-6, mem.heads, False), n * inner * 6)
        a = rnd(n, d)
        split = lambda q, t: HS.linear_split(q, t, sm["gates"])
        for name, wt, fn in (("GEMM latent attention in", w.layers[1]["w_in"], None), ("GEMM mLSTM in, gates fp32", w.layers[0]["w_in"], split),
                             ("GEMM up", w.layers[0]["w_up"], None)):
            N_, K_ = wt.shape
            mm = fn or (gemm_skinny_acc if acc else gemm)
            run(phase, name, lambda: mm(a, wt), 2 * (n * K_ + N_ * K_) + n * N_ * (4 if acc else 2), 2.0 * n * N_ * K_)
            if acc and fn is None:
                gemm_skinny(a, wt)                                # leaves the shared accumulator zero
    return k.rows


def latanex_kernels(width: int, peaks: dict, nseq: int, length: int, batch: int, ctx: int, iters: int) -> list[dict]:
    """The kernels of Latanex in the same two steps; those of Sigosun come from kernels()."""
    k = _Kernels(peaks, iters)
    cfg = _latanex(width, 1)
    mem, m, e, d, dev, bf = cfg.layers[0].mixer, cfg.layers[1].mixer, cfg.layers[1].mlp, width, "cuda", torch.bfloat16
    w = StackWeights(cfg, dev, bf).finish()
    lw, lm = w.layers[1], w.layers[0]
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=bf)
    for t in [x[n] for x in w.layers for n in ("w_in", "w_up", "e_up", "e_down", "w_down")]:
        t.normal_(0, d ** -0.5)
    T, bs, H, G, hd = nseq * length, 16, m.heads, m.kv_heads, 128
    per = -(-max(length, ctx + 1) // bs)
    n_all = max(nseq, batch)
    tabs = torch.arange(n_all * per, dtype=torch.int32, device=dev).view(n_all, per)
    kc, vc = rnd(n_all * per, bs, G, hd), rnd(n_all * per, bs, G, hd)
    pslots = torch.cat([torch.arange(length) + i * per * bs for i in range(nseq)]).to(dev)
    dslots = torch.tensor([i * per * bs + ctx for i in range(batch)], device=dev)
    pr = _rows([(0, length)] * nseq, 0, tabs[:nseq].contiguous(), pslots, length)
    dr = _rows([(ctx, 1)] * batch, batch, tabs[:batch].contiguous(), dslots, ctx + 1)
    pieces = K.Pieces(torch.tensor([i * length for i in range(nseq + 1)], dtype=torch.int32, device=dev), length, T)
    run = lambda phase, name, fn, nbytes, flops=0.0: k.run("latanex", phase, name, fn, nbytes, flops)
    pairs = length * (length + 1) // 2
    sink, qkv, out = lw["sink"], rnd(T, (H + 2 * G) * hd), K.act(T, H * hd, bf, dev)
    io, fl = T * (2 * H + 2 * G) * hd * 2, 4.0 * nseq * pairs * H * hd
    run("prefill", "attention (packed)", lambda: K.packed_attention(qkv, m, pr, pieces, kc, vc, None, sink=sink), io, fl)
    half = replace(m, window=length // 4)
    run("prefill", "attention (packed, window of a quarter)", lambda: K.packed_attention(qkv, half, pr, pieces, kc, vc, None, sink=sink), io,
        4.0 * nseq * (half.window * (half.window + 1) // 2 + (length - half.window) * half.window) * H * hd)
    q = rnd(T, H * hd)
    run("prefill", "attention (paged, heads > 128)", lambda: K.attn_paged_prefill(q, m, pr, kc, vc, None, out, sink=sink), io, fl)
    qd, od = rnd(batch, H * hd), K.act(batch, H * hd, bf, dev)
    run("decode", "attention", lambda: K.attn_paged_decode(qd, m, dr, kc, vc, None, od, sink=sink), batch * min(ctx + 1, m.window) * G * hd * 4)
    sec, sm, su = mixer_sections(m), mixer_sections(mem), mlp_sections(e)
    norms = [(torch.ones(1, device=dev), torch.ones(d, device=dev), torch.zeros(d, device=dev)) for _ in range(2)]
    qk, vv = mem.kv_heads * mem.dim, mem.heads * mem.vdim
    for phase, r, n, ns in (("prefill", pr, T, nseq), ("decode", dr, batch, batch)):
        acc = phase == "decode"
        es = 8 if acc else 2                                      # accumulators are read and zeroed
        z = lambda c: torch.zeros(n, c, device=dev) if acc else rnd(n, c)
        proj, first = z(sec.total), rnd(n, G * hd)
        run(phase, "bias + row norm + values + cache", lambda: K.qkv_rows(proj, sec, m, lw, 1e-6, r, first, kc, vc, bf, None if acc else pieces, acc),
            n * (sec.total * es + G * hd * 2 + (H + (0 if acc else 2 * G)) * hd * 2 + 2 * G * hd * 2))
        x, y, rows_, wt = torch.randn(n, d, device=dev), z(d), rnd(n * e.top, d), torch.rand(n, e.top, device=dev)
        run(phase, "tanh norms + residual", lambda: TN.tanh_between_(x, y, *norms, bf, acc=acc), n * d * (es + 8 + 2))
        ex = ME.ExpertSum(rows_, wt, y)
        run(phase, "sum of experts + tanh norms + residual", lambda: TN.tanh_between_(x, ex, *norms, bf, acc=acc), n * d * (es + 8 + 2 + 2 * e.top))
        del rows_, ex
        h, logits = rnd(n, d), torch.randn(n, round8(e.experts), device=dev)
        counts = ME._counts(torch.device(dev, torch.cuda.current_device()), e.experts)

        def route():
            counts.zero_()
            return ME._route(None, logits, 0, lw["correction"], e)
        run(phase, "routing (and clearing its counters)", route, n * (e.experts * 4 + e.top * 8))
        wgt, lists, cnt = route()
        cnt = cnt.clone()
        counts.zero_()                                            # as the next step wants them
        hit = int((cnt > 0).sum())
        a, rows_ = K.act(n * e.top, e.ff, bf, dev), K.act(n * e.top, d, bf, dev)
        run(phase, "experts in + activation", lambda: ME.grouped_gemm(h, lw["e_up"], lists, cnt, a, rows=e.ff, pairs_per_row=e.top, up=True, limit=e.limit),
            2 * (n * d + hit * 2 * e.ff * d + n * e.top * e.ff), 4.0 * n * e.top * e.ff * d)
        run(phase, "experts out", lambda: ME.grouped_gemm(a, lw["e_down"], lists, cnt, rows_, rows=d, pairs_per_row=1),
            2 * (n * e.top * (e.ff + d) + hit * e.ff * d), 2.0 * n * e.top * e.ff * d)
        del a, rows_
        p = z(su.total)
        hs = K.act(n, e.shared_ff, bf, dev)
        run(phase, "gated activation (shared expert)", lambda: ME._route(p, None, 0, None, None, (su["gate"], su["up"], e.shared_ff, 7.0, hs), acc=acc),
            n * e.shared_ff * (2 * es + 2))
        conv, ssm = torch.zeros(ns, mem.conv - 1, sm["g"], device=dev, dtype=bf), torch.zeros(ns, mem.heads, mem.dim, mem.vdim, device=dev)
        pm, gates = rnd(n, sm["gates"]), torch.randn(n, 2 * mem.heads, device=dev)
        cb, zp = w.derived[0]["conv_b"], torch.zeros(n, sm.total, device=dev) if acc else None
        if acc:
            run(phase, "short conv", lambda: K.short_conv(zp, 0, sm["g"], lm["conv"], cb, conv, r, bf, acc=True, width=sm.total, split=sm["gates"]),
                n * (sm.total * 10 + sm["g"] * 2 + (mem.conv - 1) * sm["g"] * 2))
        else:
            run(phase, "short conv", lambda: K.short_conv(pm, 0, sm["g"], lm["conv"], cb, conv, r, bf), n * sm["g"] * 4)
        # useful work of the chunked form: products with the state (three), scores of keys and queries, the triangular system, its use
        work = 2.0 * n * mem.heads * (3 * mem.dim * mem.vdim + 32 * 2 * mem.dim + 32 * 2 * mem.vdim) if not acc else 6.0 * n * mem.heads * mem.dim * mem.vdim
        run(phase, "delta scan", lambda: DR.delta_scan(pm[:, :qk], pm[:, sm["k"]:sm["k"] + qk], pm[:, sm["v"]:sm["v"] + vv], gates, lm["A_log"], lm["dt_bias"],
                                                       ssm, r, mem.heads, mem.kv_heads, mem.dim, mem.vdim, conv_src=pm, conv_col=0, conv_state=conv),
            n * (2 * qk + 2 * vv) * 2 + n * 8 * mem.heads + ns * 8 * ssm[0].numel(), work)
        yb = rnd(n, vv)
        run(phase, "head norm + gate", lambda: K.gated_norm(yb, pm[:, sm["g"]:sm["g"] + vv], w.derived[0]["norm"], 1e-6, mem.heads, False, silu=True), n * vv * 6)
        for name, wm, fn in (("GEMM attention in", lw["w_in"], None), ("GEMM delta in, gates fp32", lm["w_in"], lambda q, t: HS.linear_split(q, t, sm["gates"])),
                             ("GEMM shared expert, router", lw["w_up"], None)):
            N_, K_ = wm.shape
            mm = fn or (gemm_skinny_acc if acc else gemm)
            run(phase, name, lambda: mm(h, wm), 2 * (n * K_ + N_ * K_) + n * N_ * (4 if acc else 2), 2.0 * n * N_ * K_)
            if acc and fn is None:
                gemm_skinny(h, wm)                                # leaves the shared accumulator zero
    return k.rows


def ridazen_kernels(width: int, peaks: dict, nseq: int, length: int, batch: int, ctx: int, iters: int) -> list[dict]:
    """The kernels of Ridazen in the same two steps; those of Latanex come from latanex_kernels()."""
    k = _Kernels(peaks, iters)
    cfg = _ridazen(width, 1)
    m, e, d, dev, bf, side = cfg.layers[0].mixer, cfg.layers[0].mlp, width, "cuda", torch.bfloat16, cfg.token_side
    w = StackWeights(replace(cfg, layers=cfg.layers[:1], loop=None), dev, bf)
    lw = w.layers[0]
    lw["rel"].normal_()
    bias = w.finish().derived[0]["bias"]
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=bf)
    for n in ("w_in", "w_up", "e_up", "e_down", "w_down", "side_gate", "side_proj"):
        lw[n].normal_(0, d ** -0.5)
    T, bs, H, G, hd = nseq * length, 16, m.heads, m.kv_heads, 128
    per = -(-max(length, ctx + 1) // bs)
    n_all = max(nseq, batch)
    tabs = torch.arange(n_all * per, dtype=torch.int32, device=dev).view(n_all, per)
    kc, vc = rnd(n_all * per, bs, G, hd), rnd(n_all * per, bs, G, hd)
    pslots = torch.cat([torch.arange(length) + i * per * bs for i in range(nseq)]).to(dev)
    dslots = torch.tensor([i * per * bs + ctx for i in range(batch)], device=dev)
    pr = _rows([(0, length)] * nseq, 0, tabs[:nseq].contiguous(), pslots, length)
    dr = _rows([(ctx, 1)] * batch, batch, tabs[:batch].contiguous(), dslots, ctx + 1)
    pieces = K.Pieces(torch.tensor([i * length for i in range(nseq + 1)], dtype=torch.int32, device=dev), length, T)
    run = lambda phase, name, fn, nbytes, flops=0.0: k.run("ridazen", phase, name, fn, nbytes, flops)
    pairs = length * (length + 1) // 2
    sec, su = mixer_sections(m), mlp_sections(e)
    qkv, out, proj = rnd(T, (H + 2 * G) * hd), K.act(T, H * hd, bf, dev), rnd(T, sec.total)
    more = dict(bias=bias, out_gate=proj[:, sec["g"]:sec["g"] + H * hd])
    io, fl = T * (3 * H + 2 * G) * hd * 2, 4.0 * nseq * pairs * H * hd
    run("prefill", "attention (packed)", lambda: K.packed_attention(qkv, m, pr, pieces, kc, vc, None, **more), io, fl)
    q = rnd(T, H * hd)
    run("prefill", "attention (paged, heads > 128)", lambda: K.attn_paged_prefill(q, m, pr, kc, vc, None, out, **more), io, fl)
    qd, od, gd = rnd(batch, H * hd), K.act(batch, H * hd, bf, dev), rnd(batch, H * hd)
    run("decode", "attention", lambda: K.attn_paged_decode(qd, m, dr, kc, vc, None, od, bias=bias, out_gate=gd), batch * (ctx + 1) * G * hd * 4)
    del qkv, out, q, proj
    factors = K.temp_table(max(length, ctx + 1), m.q_temp, dev)
    pre, post = torch.ones(d, device=dev), torch.ones(d, device=dev)
    for phase, r, n, ns in (("prefill", pr, T, nseq), ("decode", dr, batch, batch)):
        acc = phase == "decode"
        es = 8 if acc else 2                                      # accumulators are read and zeroed
        z = lambda c: torch.zeros(n, c, device=dev) if acc else rnd(n, c)
        proj, state = z(sec.total), torch.zeros(ns, m.conv - 1, sec["g"], device=dev, dtype=bf)
        cols = sec.total if acc else sec["g"]                     # prompts leave the gates to the attention kernel
        run(phase, "conv + head norms + cache", lambda: K.conv_qkv(proj, sec, m, lw, factors, 1e-6, r, state, kc, vc, bf, None if acc else pieces, acc),
            n * (cols * es + (H + (H if acc else 2 * G)) * hd * 2 + 2 * G * hd * 2) + ns * state[0].numel() * 4)
        x, y, rows_, wt = torch.randn(n, d, device=dev), z(d), rnd(n * e.top, d), torch.rand(n, e.top, device=dev)
        run(phase, "residual + norm", lambda: PN.between_(x, y, pre, 1e-6, bf, mult=0.7, acc=acc), n * d * (es + 8 + 2))
        run(phase, "norm + residual + norm", lambda: PN.between_(x, y, pre, 1e-6, bf, mult=0.7, post=post, acc=acc), n * d * (es + 8 + 2))
        ex = ME.ExpertSum(rows_, wt, y, share=wt[:, 0].contiguous())
        run(phase, "sum of experts + residual", lambda: PN.between_(x, ex, None, 1e-6, bf, mult=0.7, copy=True, acc=acc),
            n * d * (es + 8 + 2 + 2 * e.top))
        del rows_, ex
        h, logits = rnd(n, d), torch.randn(n, round8(e.experts) + 8, device=dev)
        counts, share = ME._counts(torch.device(dev, torch.cuda.current_device()), e.experts), torch.empty(n, device=dev)

        def route():
            counts.zero_()
            return ME._route(None, logits, 0, lw["correction"], e, share=(round8(e.experts), share))
        run(phase, "routing (and clearing its counters)", route, n * (e.experts * 4 + e.top * 8))
        wgt, lists, cnt = route()
        cnt = cnt.clone()
        counts.zero_()                                            # as the next step wants them
        hit = int((cnt > 0).sum())
        a, rows_ = K.act(n * e.top, e.ff, bf, dev), K.act(n * e.top, d, bf, dev)
        run(phase, "experts in + activation", lambda: ME.grouped_gemm(h, lw["e_up"], lists, cnt, a, rows=e.ff, pairs_per_row=e.top, up=True, act=e.act),
            2 * (n * d + hit * e.ff * d + n * e.top * e.ff), 2.0 * n * e.top * e.ff * d)
        run(phase, "experts out", lambda: ME.grouped_gemm(a, lw["e_down"], lists, cnt, rows_, rows=d, pairs_per_row=1),
            2 * (n * e.top * (e.ff + d) + hit * e.ff * d), 2.0 * n * e.top * e.ff * d)
        del a, rows_
        ids, emb = torch.randint(0, 1000, (n,), device=dev), rnd(1000, side)
        u, hs = z(round8(side)), rnd(n, side)
        run(phase, "token input gate", lambda: PN.token_gate(u, ids, emb, 0, side, bf, acc=acc), n * side * (es + 4))
        if acc:
            p, hu = z(su.total), K.act(n, e.shared_ff, bf, dev)
            run(phase, "relu^2 (shared expert)", lambda: ME._route(p, None, 0, None, None, (-1, su["up"], e.shared_ff, 0.0, hu), acc=True),
                n * e.shared_ff * (es + 2))
        else:
            run(phase, "GEMM shared expert in + relu^2", lambda: gemm_relu2(h, lw["w_up"][:su["router"]], e.shared_ff),
                2 * (n * d + su["router"] * d + n * e.shared_ff), 2.0 * n * su["router"] * d)
            run(phase, "GEMM router", lambda: K.linear(h, lw["w_up"][su["router"]:], out_dtype=torch.float32),
                2 * (n * d + (su.total - su["router"]) * d) + 4 * n * (su.total - su["router"]), 2.0 * n * (su.total - su["router"]) * d)
        for name, a, wm in (("GEMM attention in", h, lw["w_in"]), ("GEMM token input in", h, lw["side_gate"]), ("GEMM token input out", hs, lw["side_proj"]),
                            *((("GEMM shared expert, router", h, lw["w_up"]),) if acc else ())):
            N_, K_ = wm.shape
            mm = gemm_skinny_acc if acc else gemm
            run(phase, name, lambda: mm(a, wm), 2 * (n * K_ + N_ * K_) + n * N_ * (4 if acc else 2), 2.0 * n * N_ * K_)
            if acc:
                gemm_skinny(a, wm)                                # leaves the shared accumulator zero
    return k.rows


def main(steps: int, warmup: int, sizes: str, peaks: dict, sampler, workload: str = "sigosun") -> dict:
    iters, warmup = max(3, steps), max(3, warmup)
    name, other = {"logozen": ("Logozen", "Sigosun"), "latanex": ("Latanex", "Sigosun"),
                   "ridazen": ("Ridazen", "Latanex")}.get(workload, ("Sigosun", "Llama"))
    out = {"metric": f"{name} serving tok/s beside {other} of equal size", "impl": "dlti_b200", "dtype": "bf16",
           "data": "synthetic (random token ids; random-init weights)", "steps": iters, "warmup": warmup, "sizes": [], "kernels": {}}
    _lib.reset_launch_count()
    for spec in sizes.split(","):
        width, blocks = (int(x) for x in spec.split("x"))
        sig = _sigosun(width, blocks)
        params = sig.num_params() - 2 * sig.vocab_size * width
        models = {"logozen": lambda: (_logozen(width, params), sig), "latanex": lambda: (_latanex(width, params), sig),
                  "ridazen": lambda: (_ridazen(width, params), _latanex(width, params)),
                  "sigosun": lambda: (sig, _llama(width, params))}[workload]()
        row = {"width": width, "rows": []}
        for cfg in models:
            eng = _engine(cfg, 8704, 64)
            e = {"model": cfg.name, "layers": cfg.num_hidden_layers, "params_m": round(cfg.num_params() / 1e6), "active_params_m": round(active_params(cfg) / 1e6)}
            for nseq, length in ((1, 8192), (4, 2048), (16, 512)):
                ms = prefill_ms(eng, nseq, length, warmup, iters)
                e[f"prefill {nseq}x{length}"] = {"ms": round(ms, 3), "tok_s": round(nseq * length / ms * 1e3)}
            for batch, ctx in ((1, 1000), (16, 1000), (64, 1000), (64, 8000)):
                ms = decode_ms(eng, batch, ctx, warmup + 2, 4 * iters)
                floor = step_bytes(eng, batch, ctx) / peaks["hbm_gbs"] / 1e6
                e[f"decode {batch}@{ctx}"] = {"ms": round(ms, 3), "tok_s": round(batch / ms * 1e3), "frac_of_byte_floor": round(floor / ms, 3)}
            row["rows"].append(e)
            del eng
            torch.cuda.empty_cache()
        out["sizes"].append(row)
        own = {"sigosun": kernels, "logozen": logozen_kernels, "latanex": latanex_kernels, "ridazen": ridazen_kernels}
        beside = {"sigosun": [], "ridazen": ["latanex"]}.get(workload, ["sigosun"])
        ks = own[workload](width, peaks, 4, 2048, 64, 1000, iters)
        for b in beside:
            ks += [r for r in own[b](width, peaks, 4, 2048, 64, 1000, iters) if r["model"] == b]
        out["kernels"][str(width)] = ks
        torch.cuda.empty_cache()
    out["gpu_launches"] = _lib.launch_count()
    out["clocks"] = sampler.stop()
    out["config"] = {"sizes": sizes, "l2": "steps: weights larger than L2 or streamed once per step; kernels: L2 overwritten before every call",
                     "peaks": {k: peaks[k] for k in ("hbm_gbs", "bf16_tflops")}}
    return out


def print_tables(out: dict, emit=print) -> None:
    for s in out["sizes"]:
        a, b = s["rows"]
        size = lambda e: f"{e['model']} ({e['params_m']} M" + (")" if e["active_params_m"] == e["params_m"] else f", {e['active_params_m']} M a token)")
        emit(f"# {size(a)} | {size(b)}")
        for key in a:
            if isinstance(a[key], dict):
                emit(f"{key:20s} {a[key]['ms']:9.3f} ms {a[key]['tok_s']:9d} tok/s | {b[key]['ms']:9.3f} ms {b[key]['tok_s']:9d} tok/s | "
                     f"{a[key].get('frac_of_byte_floor', '')} {b[key].get('frac_of_byte_floor', '')}")
    for w, rows in out["kernels"].items():
        emit(f"# kernels, width {w}")
        for r in rows:
            emit(f"{r['model']:8s} {r['phase']:8s} {r['kernel']:40s} {r['us']:9.2f} us, roof {r['roof_us']:8.2f} us = {r['frac_of_roof']:.3f} ({r['bound']})")


def run_cli(steps: int, warmup: int, sizes: str, peaks: dict, sampler, workload: str) -> None:
    out = main(steps, warmup, sizes, peaks, sampler, workload)
    import sys
    print_tables(out, lambda s: print(s, file=sys.stderr))
    print(json.dumps(out))
