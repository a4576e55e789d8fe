"""Serving forward pass of the layer-stack models (models/stack.py): softmax attention over the paged cache and
recurrent layers over per-sequence states, on the same engine, scheduler, block manager and sampler as the Llama family.

A step's rows are [decode rows | prompt rows]; a prompt's rows may be any portion of it. A model is a list of sublayers
(mixers and feed-forwards); what lies between two of them — adding an output to the residual, norms, the next sublayer's
input — is one object per kind of residual."""
from __future__ import annotations

import os

import torch

from ..models.stack import (AttentionMixer, DeltaMixer, LatentAttentionMixer, LightningMixer, Mamba2Mixer, MLstmMixer, MoeMlp, StackConfig,
                            StackWeights, conv_span, mixer_sections, round8)
from ..ops import _lib
from ..ops import delta as D
from ..ops import dyt as N
from ..ops import latent as LA
from ..ops import moe as M
from ..ops import prenorm as P
from ..ops import stack as K
from ..ops import streams as H
from ..ops.gemm import gemm_relu2, gemm_skinny_acc
from .kv_cache import KVCache, KVSpec, StateCache, StateSpec


_FUSE_ACC = os.environ.get("DLTI_DECODE_FUSE_ACC", "1") == "1"    # A/B switch: consume the fp32 accumulators directly


class OutputNorms:
    """One residual; norms act on the sublayer outputs only, so every sublayer reads the residual itself: the fp32 stream and,
    for 16-bit compute, its rounded copy that the norm-and-add kernel writes next to it. A sublayer is named (weights, 1 for
    the mixer or 2 for the feed-forward, layer)."""

    def __init__(self, run: "StackRunner", ids, rows: K.Rows, first, acc: bool):
        self.run, self.acc = run, acc
        self.x, self.h = K.embed_rows(ids, run.w.embed)

    def step(self, y, done, then):
        """The output y of the sublayer `done` goes to the residual; returns the input of the sublayer `then` (None: the last)."""
        cfg = self.run.cfg
        self.h = K.post_norm_add_(y, self.x, done[0][f"norm{done[1]}"], cfg.norm_eps, cfg.norm_one_plus, self.run.dtype, acc=self.acc)
        return self.h

    def residual(self):
        return self.x.clone()

    def final(self, idx):
        cfg = self.run.cfg
        return K.rms_rows(self.x, idx, self.run.w.final_norm, cfg.norm_eps, cfg.norm_one_plus, self.run.dtype)


class HyperStreams:
    """Several residual streams around pre-norm sublayers (ops/streams.py): one kernel between two sublayers renews the streams and
    makes the next normed input; the convolution of the input is part of it when every sequence has one row."""

    def __init__(self, run: "StackRunner", ids, rows: K.Rows, first, acc: bool):
        self.run, self.rows, self.acc = run, rows, acc
        self.single = rows.nd == ids.numel()
        self.x = H.embed_streams(ids, run.w.embed, run.cfg.streams, run.cfg.embed_scale)
        self.last = None
        self.h = self._between(None, None, first)

    def _between(self, y, done, then):
        run = self.run
        mix = w_out = w_in = norm = conv = None
        if done is not None:
            mix, w_out = done[0][f"hc{done[1]}.mix"], done[0][f"hc{done[1]}.out"]
        if then is not None:
            lw, q, i = then
            w_in, norm = lw[f"hc{q}.in"], lw[f"norm{q}"]
            conv = (lw[f"canon{q}"], run.states.canon[i][q - 1], self.rows)
        h = H.hyper_(self.x, y, mix, w_out, w_in, norm, run.cfg.norm_eps, run.dtype, conv=conv if self.single else None,
                     acc=self.acc and y is not None)
        return h if self.single or then is None else H.canon(h, *conv)

    def step(self, y, done, then):
        return self._between(y, done, then)

    def residual(self):
        return self.x.sum(1)

    def final(self, idx):
        return H.hyper_(self.x, None, None, None, None, self.run.w.final_norm, self.run.cfg.norm_eps, self.run.dtype, idx=idx)


class TanhNorms:
    """One fp32 residual, a dynamic tanh norm before and after every sublayer (ops/dyt.py): one elementwise kernel between two
    sublayers, which also adds up the outputs of a mixture of experts."""

    def __init__(self, run: "StackRunner", ids, rows: K.Rows, first, acc: bool):
        self.run, self.acc = run, acc
        self.x, self.h = N.embed_tanh(ids, run.w.embed, run.cfg.embed_scale, self._norm(first), run.dtype)

    @staticmethod
    def _norm(part, after=""):
        lw, name = part[0], f"norm{part[1]}{after}"
        return lw[name + ".alpha"], lw[name], lw[name + ".b"]

    def step(self, y, done, then):
        return N.tanh_between_(self.x, y, self._norm(done, "b"), None if then is None else self._norm(then), self.run.dtype, acc=self.acc)

    def residual(self):
        return self.x.clone()

    def final(self, idx):
        w = self.run.w
        return N.tanh_rows(self.x, idx, (w.final_norm_alpha, w.final_norm, w.final_norm_b), self.run.dtype)


class PreNorms:
    """One fp32 residual, RMS norms on the sublayer inputs (ops/prenorm.py): one kernel between two sublayers, which also adds up the
    outputs of a mixture of experts, norms the output of a token input, and adds the embedding where a pass of a loop begins."""

    def __init__(self, run: "StackRunner", ids, rows: K.Rows, first, acc: bool):
        self.run, self.acc, self.again = run, acc, False
        self.embed = (ids, run.w.embed, run.cfg.embed_scale)
        self.x = torch.empty((ids.numel(), run.cfg.hidden_size), dtype=torch.float32, device=run.w.embed.device)
        self.h = P.between_(self.x, None, first[0]["norm1"], run.cfg.norm_eps, run.dtype, embed=self.embed, fresh=True)

    def step(self, y, done, then):
        cfg = self.run.cfg
        self.again = then is not None and then[1] == 1 and then[2] in cfg.restarts
        side = then is not None and then[1] == 3                      # a token input reads the residual itself
        return P.between_(self.x, y, None if then is None or side else then[0][f"norm{then[1]}"], cfg.norm_eps, self.run.dtype,
                          mult=cfg.residual_mult, post=done[0]["norm3"] if done[1] == 3 else None, embed=self.embed if self.again else None,
                          copy=side, acc=self.acc)

    def residual(self):
        ids, table, scale = self.embed
        return self.x - table[ids].float() * scale if self.again else self.x.clone()

    def final(self, idx):
        cfg = self.run.cfg
        return K.rms_rows(self.x, idx, self.run.w.final_norm, cfg.norm_eps, False, self.run.dtype)


class StackRunner:
    per_sequence = True

    @staticmethod
    def cache_specs(cfg: StackConfig, weights: StackWeights):
        """(key/value page specs, recurrent-state specs), one entry per run of a layer. Head rows are padded to 16 bytes."""
        kv, st = [], []
        for l in (cfg.layers[j] for j in cfg.runs):
            m = l.mixer
            if isinstance(m, AttentionMixer):
                kv.append(KVSpec(m.kv_heads, round8(m.dim), round8(m.vdim), m.kv_from))
            else:
                kv.append(KVSpec(1, m.pitch, 0) if isinstance(m, LatentAttentionMixer) else None)
            state = {}
            if isinstance(m, Mamba2Mixer):
                state = dict(heads=m.heads, rows=m.state, cols=m.vdim, conv_rows=m.conv - 1, conv_channels=m.conv_channels if m.conv > 1 else 0)
            elif isinstance(m, AttentionMixer) and m.conv > 1:
                state = dict(conv_rows=m.conv - 1, conv_channels=conv_span(m))
            elif isinstance(m, LightningMixer):
                state = dict(heads=m.heads, rows=m.dim, cols=m.vdim)
            elif isinstance(m, DeltaMixer):
                state = dict(heads=m.heads, rows=m.dim, cols=m.vdim, conv_rows=m.conv - 1, conv_channels=mixer_sections(m)["g"] if m.conv > 1 else 0)
            elif isinstance(m, MLstmMixer):
                state = dict(heads=m.heads, rows=m.dim, cols=m.vdim, vec=K.mlstm_vec(m.dim, m.vdim))
            if cfg.streams:
                state |= dict(canon_parts=1 if l.mlp is None else 2, canon_rows=cfg.canon - 1, canon_channels=cfg.hidden_size)
            st.append(StateSpec(**state) if state else None)
        return kv, st

    def __init__(self, cfg: StackConfig, weights: StackWeights, kv: KVCache, states: StateCache | None, max_len: int):
        self.cfg, self.w, self.kv, self.states = cfg, weights, kv, states
        self.device, self.dtype = weights.device, weights.dtype
        # one entry per run of a layer: caches and states belong to the run, weights to the layer
        self.layers = [cfg.layers[j] for j in cfg.runs]
        self.derived = [weights.derived[j] for j in cfg.runs]
        self.sections = [mixer_sections(l.mixer) for l in self.layers]
        self.ropes = [K.rope_tables(max_len, l.mixer.rope.dims, l.mixer.rope.base, self.device)
                      if getattr(l.mixer, "rope", None) is not None else None for l in self.layers]
        self.temps = [K.temp_table(max_len, l.mixer.q_temp, self.device) if getattr(l.mixer, "q_temp", None) is not None else None
                      for l in self.layers]
        if self.device.type == "cuda" and "DLTI_PDL" not in os.environ:
            # serving weights are static: the decode GEMMs may fetch weight tiles while the previous kernel drains
            _lib.gpu_lib().dlti_set_pdl(2)
        self.pack_prompts = True     # False: all prompt attention reads the pages
        self.trace = None            # set to a list: receives the residual after every layer (debugging)
        self.mixers = {AttentionMixer: self._attention, LatentAttentionMixer: self._latent, Mamba2Mixer: self._mamba2,
                       LightningMixer: self._lightning, MLstmMixer: self._mlstm, DeltaMixer: self._delta}
        # the sublayers in order: (layer weights, 1 mixer | 2 feed-forward | 3 token input, run)
        self.parts = [(weights.layers[j], q, i) for i, j in enumerate(cfg.runs)
                      for q, have in ((1, True), (2, cfg.layers[j].mlp is not None), (3, cfg.token_side > 0)) if have]

    @torch.no_grad()
    def forward(self, input_ids, positions, slots, *, num_decode: int = 0, block_tables=None, ctx_lens=None, cu_seqlens=None,
                max_seqlen: int = 0, last_idx=None, max_ctx: int = 0, state_slots=None, row_seq=None, segs=None) -> torch.Tensor:
        """One pass over T token rows (see ops.stack.Rows for the arguments). segs: (attention chunk size, window) ->
        ops.stack.Pieces of the prompt rows (none: prompt attention reads the pages). Returns fp32 logits of the rows `last_idx`."""
        cfg, w = self.cfg, self.w
        rows = K.Rows(positions, row_seq, slots, ctx_lens, cu_seqlens, block_tables, state_slots, int(num_decode), max_seqlen,
                      max_ctx)
        ids = input_ids.view(-1)
        # decode-sized steps stream the weights through the stream-K GEMM; the next op consumes its fp32 accumulator
        self.acc = _FUSE_ACC and w.embed.is_cuda and self.dtype == torch.bfloat16 and ids.numel() <= 256
        mm = gemm_skinny_acc if self.acc else K.linear
        kind = HyperStreams if cfg.streams else TanhNorms if cfg.tanh_norms else PreNorms if cfg.pre_norm else OutputNorms
        res = kind(self, ids, rows, self.parts[0], self.acc)
        h = res.h
        self.first_v = None          # values of the first layer that mixes values
        for part, then in zip(self.parts, self.parts[1:] + [None]):
            lw, q, i = part
            m = self.layers[i].mixer
            if q == 1:
                y = mm(self.mixers[type(m)](i, m, lw, h, rows, segs), lw["w_out"])
            elif q == 2:
                y = self._mlp(self.layers[i].mlp, lw, h, mm)
            else:
                n = cfg.token_side
                y = mm(P.token_gate(mm(h, lw["side_gate"]), ids, w.side_embed, cfg.runs[i] * n, n, self.dtype, acc=self.acc), lw["side_proj"])
            h = res.step(y, part, then)
            if self.trace is not None and (then is None or then[2] != i):
                self.trace.append(res.residual())
        if last_idx is not None and last_idx.numel() == 0:
            return torch.empty((0, cfg.vocab_size), dtype=torch.float32, device=self.device)
        return K.linear_f32(res.final(last_idx), w.lm_head, cfg.logit_scale, cfg.logit_softcap)[:, :cfg.vocab_size]

    def _mlp(self, mlp, lw, h, mm):
        if isinstance(mlp, MoeMlp):
            return M.moe(h, mlp, lw, self.dtype, mm, acc=self.acc)
        if mlp.act == "polynorm":
            u = H.poly_norm(mm(h, lw["w_up"]), mlp.ff, lw["act"], self.cfg.norm_eps, self.dtype, acc=self.acc)
        elif mlp.act == "swiglu":
            u = M.swiglu(h, lw["w_up"], mlp.ff, self.dtype, acc=self.acc)
        else:
            u = gemm_relu2(h, lw["w_up"], mlp.ff) if h.is_cuda and not self.acc else None  # activation in the GEMM
            u = K.relu2(mm(h, lw["w_up"]), mlp.ff, self.dtype, acc=self.acc) if u is None else u
        return mm(u, lw["w_down"])

    def _attention(self, i, m: AttentionMixer, lw, xa, rows: K.Rows, segs):
        # prompts with heads of up to 128: the varlen tcgen05 kernel on rows cut at the chunk edges; everything else
        # (short portions, larger heads, fp32) reads the pages
        packed = None
        if (xa.is_cuda and self.dtype == torch.bfloat16 and 32 < max(m.dim, m.vdim) <= K.PACKED_HD and m.vdim % 8 == 0
                and self.pack_prompts):
            packed = (segs or {}).get(m.reach)
        # the convolutions of prompt rows read their neighbours' inputs: conv_qkv takes the accumulators of decode steps only
        acc = self.acc and (not m.conv_heads or rows.nd == xa.shape[0])
        proj = gemm_skinny_acc(xa, lw["w_in"]) if acc else K.linear(xa, lw["w_in"])
        sink, bias, out_gate = lw.get("sink"), self.derived[i].get("bias"), None
        if bias is not None and bias.shape[1] > K.PACKED_BIAS:
            packed = None
        if m.conv_heads:
            state = self.states.conv[i] if m.conv > 1 else None
            q, out_gate = K.conv_qkv(proj, self.sections[i], m, lw, self.temps[i], self.cfg.norm_eps, rows, state, self.kv.k[i], self.kv.v[i],
                                     self.dtype, packed=packed, acc=acc)
            gate = None
        elif m.whole_rows:
            q, own = K.qkv_rows(proj, self.sections[i], m, lw, self.cfg.norm_eps, rows, self.first_v, self.kv.k[i], self.kv.v[i], self.dtype,
                                packed=packed, acc=acc)
            self.first_v = own if own is not None else self.first_v
            gate = None
        else:
            q, gate = K.qk_norm_rope_cache(proj, self.sections[i], m, lw.get("q_norm"), lw.get("k_norm"), self.cfg.norm_eps, rows,
                                           self.ropes[i], self.kv.k[i], self.kv.v[i], self.dtype, packed=packed, acc=acc)
        more = dict(sink=sink, bias=bias, out_gate=out_gate)
        if packed is not None:
            return K.packed_attention(q, m, rows, packed, self.kv.k[i], self.kv.v[i], gate, **more)
        return K.paged_attention(q, m, rows, self.kv.k[i], self.kv.v[i], gate, **more)

    def _mamba2(self, i, m: Mamba2Mixer, lw, xa, rows: K.Rows, segs):
        s, st = self.sections[i], self.states
        inner, gn = m.inner, m.groups * m.state
        acc = self.acc and rows.nd == xa.shape[0]                 # the convolution of prompt rows reads its neighbours' inputs
        proj = gemm_skinny_acc(xa, lw["w_in"]) if acc else K.linear(xa, lw["w_in"])
        xbc, proj = K.short_conv(proj, s["xbc"], m.conv_channels, lw["conv"], lw["conv_b"], st.conv[i], rows, self.dtype, acc=acc,
                                 width=proj.shape[1])
        decay = K.Decay(dt=proj[:, s["dt"]:s["dt"] + m.heads], dt_bias=lw["dt_bias"], A_log=lw["A_log"], D=lw["D"])
        y = K.linear_scan(xbc[:, inner + gn:], xbc[:, inner:inner + gn], xbc[:, :inner], decay, st.ssm[i], rows, m.heads, m.groups,
                          m.state, m.vdim, conv_src=proj, conv_col=s["xbc"], conv_state=st.conv[i])
        return K.gated_norm(y, proj[:, s["z"]:s["z"] + inner], lw["norm"], self.cfg.norm_eps, m.norm_groups, gate_first=True)

    def _lightning(self, i, m: LightningMixer, lw, xa, rows: K.Rows, segs):
        s = self.sections[i]
        proj = K.linear(xa, lw["w_in"])
        qk, vv = m.heads * m.dim, m.heads * m.vdim
        y = K.linear_scan(proj[:, s["q"]:s["q"] + qk], proj[:, s["k"]:s["k"] + qk], proj[:, s["v"]:s["v"] + vv],
                          K.Decay(const=lw["decay"]), self.states.ssm[i], rows, m.heads, m.heads, m.dim, m.vdim, silu=True)
        return K.gated_norm(y, proj[:, s["g"]:s["g"] + vv], lw["norm"], self.cfg.norm_eps, 1, gate_first=False)

    def _latent(self, i, m: LatentAttentionMixer, lw, xa, rows: K.Rows, segs):
        proj = gemm_skinny_acc(xa, lw["w_in"]) if self.acc else K.linear(xa, lw["w_in"])
        return LA.latent_attention(proj, self.sections[i], m, lw, self.derived[i].get("w_expand"), self.cfg.norm_eps, rows, self.ropes[i],
                                   self.kv.k[i], self.dtype, (segs or {}).get(m.reach) if self.pack_prompts else None, acc=self.acc)

    def _mlstm(self, i, m: MLstmMixer, lw, xa, rows: K.Rows, segs):
        s, st = self.sections[i], self.states
        qk, vv = m.heads * m.dim, m.heads * m.vdim
        proj, gates = H.linear_split(xa, lw["w_in"], s["gates"])
        y = K.mlstm_scan(proj[:, s["q"]:s["q"] + qk], proj[:, s["k"]:s["k"] + qk], proj[:, s["v"]:s["v"] + vv], gates, lw["gate_b"], m.gate_cap,
                         st.ssm[i], st.vec[i], rows, m.heads, m.dim, m.vdim)
        return K.gated_norm(y, proj[:, s["g"]:s["g"] + vv], lw["norm"], self.cfg.norm_eps, m.heads, gate_first=False)

    def _delta(self, i, m: DeltaMixer, lw, xa, rows: K.Rows, segs):
        s, st, der = self.sections[i], self.states, self.derived[i]
        qk, vv = m.kv_heads * m.dim, m.heads * m.vdim
        if self.acc and rows.nd == xa.shape[0]:                   # the convolution of prompt rows reads its neighbours' inputs
            proj = gemm_skinny_acc(xa, lw["w_in"])
            x, proj, gates = K.short_conv(proj, 0, s["g"], lw["conv"], der["conv_b"], st.conv[i], rows, self.dtype, acc=True, width=proj.shape[1],
                                          split=s["gates"])
        else:
            proj, gates = H.linear_split(xa, lw["w_in"], s["gates"])
            x, proj = K.short_conv(proj, 0, s["g"], lw["conv"], der["conv_b"], st.conv[i], rows, self.dtype)
        y = D.delta_scan(x[:, :qk], x[:, s["k"]:s["k"] + qk], x[:, s["v"]:s["v"] + vv], gates, lw["A_log"], lw["dt_bias"], st.ssm[i], rows, m.heads,
                         m.kv_heads, m.dim, m.vdim, conv_src=proj, conv_col=0, conv_state=st.conv[i])
        return K.gated_norm(y, proj[:, s["g"]:s["g"] + vv], der["norm"], self.cfg.norm_eps, m.heads, gate_first=False, silu=True)
