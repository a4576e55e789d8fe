"""Serving forward pass of the layer-stack models (models/stack.py): softmax attention over the paged cache and
recurrent layers over per-sequence states, on the same engine, scheduler, block manager and sampler as the Llama family.

A step's rows are [decode rows | prompt rows]; a prompt's rows may be any portion of it. Norms act on the sublayer
outputs only, so every sublayer reads the residual itself: the fp32 stream and, for 16-bit compute, its rounded copy that
the norm-and-add kernel writes next to it."""
from __future__ import annotations

import os

import torch

from ..models.stack import AttentionMixer, LightningMixer, Mamba2Mixer, StackConfig, StackWeights, mixer_sections, round8
from ..ops import _lib
from ..ops import stack as K
from ..ops.gemm import gemm_relu2, gemm_skinny_acc
from .kv_cache import KVCache, KVSpec, StateCache, StateSpec


_FUSE_ACC = os.environ.get("DLTI_DECODE_FUSE_ACC", "1") == "1"    # A/B switch: consume the fp32 accumulators directly


class StackRunner:
    per_sequence = True

    @staticmethod
    def cache_specs(cfg: StackConfig, weights: StackWeights):
        """(key/value page specs, recurrent-state specs), one entry per layer. Head rows are padded to 16 bytes."""
        kv, st = [], []
        for l in cfg.layers:
            m = l.mixer
            kv.append(KVSpec(m.kv_heads, round8(m.dim), round8(m.vdim), m.kv_from) if isinstance(m, AttentionMixer) else None)
            if isinstance(m, Mamba2Mixer):
                st.append(StateSpec(m.heads, m.state, m.vdim, m.conv - 1, m.conv_channels if m.conv > 1 else 0))
            elif isinstance(m, LightningMixer):
                st.append(StateSpec(m.heads, m.dim, m.vdim))
            else:
                st.append(None)
        return kv, st

    def __init__(self, cfg: StackConfig, weights: StackWeights, kv: KVCache, states: StateCache | None, max_len: int):
        self.cfg, self.w, self.kv, self.states = cfg, weights, kv, states
        self.device, self.dtype = weights.device, weights.dtype
        self.sections = [mixer_sections(l.mixer) for l in cfg.layers]
        self.ropes = [K.rope_tables(max_len, l.mixer.rope.dims, l.mixer.rope.base, self.device)
                      if isinstance(l.mixer, AttentionMixer) and l.mixer.rope is not None else None for l in cfg.layers]
        if self.device.type == "cuda" and "DLTI_PDL" not in os.environ:
            # serving weights are static: the decode GEMMs may fetch weight tiles while the previous kernel drains
            _lib.gpu_lib().dlti_set_pdl(2)
        self.pack_prompts = True     # False: all prompt attention reads the pages
        self.trace = None            # set to a list: receives the residual stream after every layer (debugging)

    @torch.no_grad()
    def forward(self, input_ids, positions, slots, *, num_decode: int = 0, block_tables=None, ctx_lens=None, cu_seqlens=None,
                max_seqlen: int = 0, last_idx=None, max_ctx: int = 0, state_slots=None, row_seq=None, segs=None) -> torch.Tensor:
        """One pass over T token rows (see ops.stack.Rows for the arguments). segs: attention chunk size ->
        ops.stack.Pieces of the prompt rows (none: prompt attention reads the pages). Returns fp32 logits of the rows `last_idx`."""
        cfg, w = self.cfg, self.w
        rows = K.Rows(positions, row_seq, slots, ctx_lens, cu_seqlens, block_tables, state_slots, int(num_decode), max_seqlen,
                      max_ctx)
        x, xa = K.embed_rows(input_ids.view(-1), w.embed)
        # decode-sized steps stream the weights through the stream-K GEMM; the next op consumes its fp32 accumulator
        self.acc = acc = _FUSE_ACC and x.is_cuda and self.dtype == torch.bfloat16 and x.shape[0] <= 256
        mm = gemm_skinny_acc if acc else K.linear
        for i, (l, lw) in enumerate(zip(cfg.layers, w.layers)):
            m = l.mixer
            if isinstance(m, AttentionMixer):
                y = self._attention(i, m, lw, xa, rows, segs)
            elif isinstance(m, Mamba2Mixer):
                y = self._mamba2(i, m, lw, xa, rows)
            else:
                y = self._lightning(i, m, lw, xa, rows)
            xa = self._close(mm(y, lw["w_out"]), x, lw["norm1"])
            if l.mlp is not None:
                h = gemm_relu2(xa, lw["w_up"], l.mlp.ff) if x.is_cuda and not acc else None      # activation in the GEMM
                if h is None:
                    h = K.relu2(mm(xa, lw["w_up"]), l.mlp.ff, self.dtype, acc=acc)
                xa = self._close(mm(h, lw["w_down"]), x, lw["norm2"])
            if self.trace is not None:
                self.trace.append(x.clone())
        if last_idx is not None and last_idx.numel() == 0:
            return torch.empty((0, cfg.vocab_size), dtype=torch.float32, device=self.device)
        xn = K.rms_rows(x, last_idx, w.final_norm, cfg.norm_eps, cfg.norm_one_plus, self.dtype)
        return K.linear_f32(xn, w.lm_head)[:, :cfg.vocab_size]

    def _close(self, y, x, norm):
        """End of a sublayer: x += norm(y); returns the next sublayer's input."""
        return K.post_norm_add_(y, x, norm, self.cfg.norm_eps, self.cfg.norm_one_plus, self.dtype, acc=self.acc)

    def _attention(self, i, m: AttentionMixer, lw, xa, rows: K.Rows, segs):
        # prompts with heads of up to 128: the varlen tcgen05 kernel on rows cut at the chunk edges; everything else
        # (short portions, larger heads, fp32) reads the pages
        packed = None
        if (xa.is_cuda and self.dtype == torch.bfloat16 and 32 < max(m.dim, m.vdim) <= K.PACKED_HD and m.vdim % 8 == 0
                and self.pack_prompts):
            packed = (segs or {}).get(m.chunk)
        proj = gemm_skinny_acc(xa, lw["w_in"]) if self.acc else K.linear(xa, lw["w_in"])
        q, gate = K.qk_norm_rope_cache(proj, self.sections[i], m, lw.get("q_norm"), lw.get("k_norm"), self.cfg.norm_eps, rows,
                                       self.ropes[i], self.kv.k[i], self.kv.v[i], self.dtype, packed=packed, acc=self.acc)
        if packed is not None:
            return K.packed_attention(q, m, rows, packed, self.kv.k[i], self.kv.v[i], gate)
        return K.paged_attention(q, m, rows, self.kv.k[i], self.kv.v[i], gate)

    def _mamba2(self, i, m: Mamba2Mixer, lw, xa, rows: K.Rows):
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

    def _lightning(self, i, m: LightningMixer, lw, xa, rows: K.Rows):
        s = self.sections[i]
        proj = K.linear(xa, lw["w_in"])
        qk, vv = m.heads * m.dim, m.heads * m.vdim
        y = K.linear_scan(proj[:, s["q"]:s["q"] + qk], proj[:, s["k"]:s["k"] + qk], proj[:, s["v"]:s["v"] + vv],
                          K.Decay(const=lw["decay"]), self.states.ssm[i], rows, m.heads, m.heads, m.dim, m.vdim, silu=True)
        return K.gated_norm(y, proj[:, s["g"]:s["g"] + vv], lw["norm"], self.cfg.norm_eps, 1, gate_first=False)
