"""Models described layer by layer: each layer names its token mixer (softmax attention, latent attention, Mamba-2,
lightning attention, mLSTM, gated delta rule) and its feed-forward (dense or a mixture of experts), with every size and
constant a parameter. The model names how sublayers meet the residual and which layers run several times. A design (models/sigosun.py, models/logozen.py,
models/latanex.py, models/ridazen.py) is a parser from its config.json to a `StackConfig` plus its tensor names; the weights container,
the cache layout and the serving forward pass (serve/stack_runner.py) are shared by all of them.

Weights are kept as merged input projections, one GEMM per mixer. Every section of a merged projection and the row
pitch of every matrix is rounded up to 8 elements, so any head count or width meets the 16-byte rules of the TMA
GEMMs; padding rows are zero and padding columns are never read.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from functools import cached_property

import torch


def round8(n: int) -> int:
    return (n + 7) // 8 * 8


def round16(n: int) -> int:
    return (n + 15) // 16 * 16


# ---- layer descriptions ------------------------------------------------------------------------------------
@dataclass(frozen=True)
class Rope:
    dims: int                      # leading dimensions of a head that are rotated
    base: float
    interleaved: bool = True       # pairs (2i, 2i+1); False: (i, i + dims/2)


@dataclass(frozen=True)
class QueryTemp:
    """Queries at position p are multiplied by 1 + coef ln(floor((p + 1) / every) + 1)."""
    coef: float
    every: int


@dataclass(frozen=True)
class DistanceBias:
    """A learned number per head and bucket of the distance n = query position - key position, added to the scores. The first
    rows // 2 buckets are single distances, the others grow evenly in ln n up to `far`; everything beyond is in the last one."""
    rows: int
    far: int

    def bucket(self, n: int) -> int:
        half = self.rows // 2
        if n < half:
            return n
        return min(self.rows - 1, half + math.floor(math.log(n / half) / math.log(self.far / half) * (self.rows - half)))

    @cached_property
    def buckets(self) -> list[int]:
        """The buckets of the distances 0, 1, ... below the first one from which on all are in the last bucket."""
        out = [self.bucket(n) for n in range(self.far + 1)]
        while out and out[-1] == self.rows - 1:
            out.pop()
        return out


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int                       # query / key size of a head
    vdim: int                      # value size of a head
    scale: float
    rope: Rope | None = None
    chunk: int = 0                 # > 0: position i sees only keys of its own chunk of this many positions
    qk_norm: bool = True           # per-head RMS norm on q and k, before the rotation
    head_gate: bool = True         # each head's output times sigmoid of one projected number
    kv_from: int | None = None     # use the cached keys and values of this earlier layer
    window: int = 0                # > 0: position i sees only itself and the window - 1 positions before it
    softcap: float = 0.0           # > 0: scores become softcap * tanh(score / softcap)
    sink: bool = False             # a learned term per head in the softmax denominator
    bias: bool = False             # on the q, k and v projections
    row_norm: bool = False         # RMS norm over all heads of q (and of k) at once
    v_mix: bool = False            # values are mixed with those of the first such layer, by one learned share per layer
    conv: int = 0                  # > 0: taps of a causal convolution on each channel of q, k and v, before the norms
    q_temp: QueryTemp | None = None
    bias_by: DistanceBias | None = None
    out_gate: bool = False         # every output element times sigmoid of its own projected number

    @property
    def reach(self) -> tuple[int, int]:
        return (self.chunk, self.window)

    @property
    def whole_rows(self) -> bool:
        """Queries, keys and values are made from whole projection rows (ops.stack.qkv_rows), not head by head."""
        return self.bias or self.row_norm or self.v_mix

    @property
    def conv_heads(self) -> bool:
        """Queries, keys and values are made head by head by the op that also convolves and scales (ops.stack.conv_qkv)."""
        return self.conv > 0 or self.q_temp is not None or self.out_gate


@dataclass(frozen=True)
class Mamba2Mixer:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int                      # taps of the causal convolution
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_channels(self) -> int:
        return self.inner + 2 * self.groups * self.state


@dataclass(frozen=True)
class LightningMixer:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]       # one factor per head


@dataclass(frozen=True)
class LatentAttentionMixer:
    """Keys and values of all heads are linear in one cached latent per token; a rotated key part is shared by the heads."""
    heads: int
    dim: int                       # unrotated query / key size of a head
    rot_dim: int                   # size of the part that carries the rotation
    vdim: int
    kv_rank: int                   # size of the latent
    scale: float
    rope: Rope | None = None       # on the rot_dim part
    sink: bool = True              # a learned term per head in the softmax denominator
    head_gate: bool = True

    chunk = window = 0             # every earlier position is seen
    reach = (0, 0)
    softcap = 0.0

    @property
    def qk_dim(self) -> int:
        return self.dim + self.rot_dim

    @property
    def rot_at(self) -> int:       # a cache row is [latent, zeros, rotated part, zeros], both parts padded to 16, ...
        return round16(self.kv_rank)

    @property
    def cols(self) -> int:
        return self.rot_at + round16(self.rot_dim)

    @property
    def pitch(self) -> int:        # ... and 8 more: a page copied as it is into shared memory is read without bank conflicts
        return self.cols + 8

    @property
    def head_pitch(self) -> int:
        """Columns of a head when its keys and values are laid out one by one: 128 for the packed layout of the tcgen05
        kernel, else rounded to 16 bytes."""
        n = max(self.qk_dim, self.vdim)
        return 128 if n <= 128 and self.vdim % 8 == 0 else round8(n)


@dataclass(frozen=True)
class MLstmMixer:
    """Matrix memory with exponential gates, a running maximum and a normaliser."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class DeltaMixer:
    """Gated delta rule: a matrix per head that forgets by one factor and replaces, by a share, what it holds for a key. Short
    convolutions on q, k and v, unit queries and keys shared by the heads of a group, a norm and a gate on the outputs."""
    heads: int
    kv_heads: int                  # query / key heads
    dim: int
    vdim: int
    conv: int                      # taps of the causal convolutions


@dataclass(frozen=True)
class DenseMlp:
    ff: int
    act: str = "relu2"             # square of relu; "polynorm": sum of the normed first three powers; "swiglu": silu(gate) * up


@dataclass(frozen=True)
class MoeMlp:
    """Mixture of experts. score "sigmoid": the router's sigmoid scores pick `top` experts by score plus a correction, out of the
    `keep` best of `groups` equal groups; the chosen scores, made to sum to `scale`, weigh the outputs. "softmax": the largest
    logits (the correction is their bias) are picked, and weighed by their softmax among the chosen, times scale."""
    experts: int
    top: int
    ff: int
    limit: float = 0.0             # act "swiglu": gate <= limit, -limit <= up <= limit
    groups: int = 1
    keep: int = 1
    scale: float = 1.0
    shared_ff: int = 0             # > 0: one more expert of this size that runs for every token
    shared_limit: float = 0.0
    shared_gate: bool = False      # the shared expert's output times sigmoid of one projected number per token
    act: str = "swiglu"            # clipped; "relu2": no gate, square of relu
    score: str = "sigmoid"

    @property
    def gated(self) -> bool:
        return self.act == "swiglu"


@dataclass(frozen=True)
class Layer:
    mixer: AttentionMixer | LatentAttentionMixer | Mamba2Mixer | LightningMixer | MLstmMixer | DeltaMixer
    mlp: DenseMlp | MoeMlp | None = None


@dataclass(frozen=True)
class Loop:
    """Layers start ... stop - 1 run `times` times in a row with the same weights, each pass on a cache and states of its own.
    Before each pass but the first the embedding is added to the residual."""
    start: int
    stop: int
    times: int


@dataclass
class StackConfig:
    hidden_size: int
    vocab_size: int
    norm_eps: float
    layers: list[Layer]
    norm_one_plus: bool = True     # layer and final norm weights are stored around zero: 1 + w
    # 0: one residual, RMS norms on the sublayer outputs. n > 0: n residual streams with learned mixing around every
    # sublayer (hyper-connections), a layer norm and a causal convolution of `canon` taps on its input
    streams: int = 0
    canon: int = 0
    tanh_norms: bool = False       # one residual, a dynamic tanh norm before and after every sublayer instead
    pre_norm: bool = False         # one residual, RMS norms on the sublayer inputs instead
    residual_mult: float = 1.0     # pre_norm: on everything that is added to the residual
    # pre_norm, > 0: after each layer, proj(gelu(gate x) * e) with the RMS norm on it, e = this many numbers of the token for the layer
    token_side: int = 0
    loop: Loop | None = None
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    logit_softcap: float = 0.0     # > 0: logits become softcap * tanh(logit / softcap)
    max_position_embeddings: int = 8192        # only a default for the server's max_model_len
    bos_token_id: int = 1
    eos_token_id: int = 2
    torch_dtype: str = "bfloat16"
    name: str = "stack"

    def __post_init__(self):
        for i, l in enumerate(self.layers):
            m = l.mixer
            if isinstance(m, AttentionMixer):
                if m.heads % m.kv_heads:
                    raise ValueError(f"layer {i}: {m.heads} query heads do not divide into {m.kv_heads} key/value heads")
                if m.rope is not None and (m.rope.dims % 2 or m.rope.dims > m.dim):
                    raise ValueError(f"layer {i}: rotary dims {m.rope.dims} must be even and at most {m.dim}")
                if m.kv_from is not None:
                    src = self.layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
                    if not isinstance(src, AttentionMixer) or src.kv_from is not None or \
                            (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
                        raise ValueError(f"layer {i}: kv_from {m.kv_from} is not an earlier attention layer of the same shape")
                if m.chunk and m.window:
                    raise ValueError(f"layer {i}: attention is cut by a chunk or by a window, not by both")
                if m.softcap < 0 or m.window < 0:
                    raise ValueError(f"layer {i}: softcap {m.softcap} and window {m.window} must not be negative")
                if m.whole_rows and (m.rope is not None or m.head_gate or m.kv_from is not None or m.qk_norm):
                    raise ValueError(f"layer {i}: biases, row norms and value mixing do not combine with rotations, head gates, head "
                                     "norms or shared keys")
                if m.conv_heads and (m.whole_rows or m.rope is not None or m.head_gate or m.kv_from is not None):
                    raise ValueError(f"layer {i}: convolutions, query temperatures and output gates do not combine with whole-row "
                                     "projections, rotations, head gates or shared keys")
                if m.bias_by is not None and (m.softcap or m.sink):
                    raise ValueError(f"layer {i}: distance biases do not combine with capped scores or sinks")
                if m.bias_by is not None and not 1 <= m.bias_by.rows // 2 < m.bias_by.far:
                    raise ValueError(f"layer {i}: {m.bias_by.rows} distance buckets up to {m.bias_by.far}")
                if m.q_temp is not None and m.q_temp.every < 1 or m.conv < 0:
                    raise ValueError(f"layer {i}: query temperature {m.q_temp}, convolutions of {m.conv} taps")
                src = self.v_mix_from(i)
                if src is not None and (src.kv_heads, src.vdim) != (m.kv_heads, m.vdim):
                    raise ValueError(f"layer {i}: values are mixed with those of a layer of another shape")
            elif isinstance(m, Mamba2Mixer):
                if m.heads % m.groups or m.inner % m.norm_groups:
                    raise ValueError(f"layer {i}: groups must divide the heads and norm_groups the inner size")
            elif isinstance(m, LatentAttentionMixer):
                if m.rope is not None and (m.rope.dims % 2 or m.rope.dims > m.rot_dim):
                    raise ValueError(f"layer {i}: rotary dims {m.rope.dims} must be even and at most {m.rot_dim}")
            elif isinstance(m, MLstmMixer):
                if not m.gate_cap > 0:
                    raise ValueError(f"layer {i}: gate_cap {m.gate_cap} must be positive")
            elif isinstance(m, DeltaMixer):
                if m.heads % m.kv_heads or m.conv < 1:
                    raise ValueError(f"layer {i}: {m.heads} heads on {m.kv_heads} query/key heads, convolutions of {m.conv} taps")
            elif len(m.decay) != m.heads:
                raise ValueError(f"layer {i}: {len(m.decay)} decays for {m.heads} heads")
            e = l.mlp
            if isinstance(e, MoeMlp):
                if e.experts % e.groups or not 1 <= e.keep <= e.groups or not 1 <= e.top <= e.keep * (e.experts // e.groups):
                    raise ValueError(f"layer {i}: {e.top} of {e.experts} experts from {e.keep} of {e.groups} groups")
                if not self.tanh_norms and not self.pre_norm:
                    raise ValueError(f"layer {i}: mixtures of experts need the tanh norms or pre-norms, which add up their outputs")
                if e.act not in ("swiglu", "relu2") or e.score not in ("sigmoid", "softmax") or e.shared_gate and not e.shared_ff:
                    raise ValueError(f"layer {i}: experts {e.act}, scores {e.score}, gate on a shared expert of {e.shared_ff}")
                if e.score == "softmax" and e.groups > 1:
                    raise ValueError(f"layer {i}: groups of experts need sigmoid scores")
        if self.streams and self.canon < 1:
            raise ValueError(f"canon taps {self.canon}: at least 1")
        if (self.token_side or self.residual_mult != 1.0 or self.loop) and not self.pre_norm:
            raise ValueError("token inputs, residual factors and loops need the pre-norms")
        if self.loop is not None:
            a, b, n = self.loop.start, self.loop.stop, self.loop.times
            if not 0 <= a < b <= len(self.layers) or n < 1:
                raise ValueError(f"layers {a} ... {b - 1} of {len(self.layers)} cannot run {n} times")
            if any(getattr(l.mixer, "kv_from", None) is not None or getattr(l.mixer, "v_mix", False) for l in self.layers):
                raise ValueError("layers on another layer's keys or values do not run in a loop")

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def runs(self) -> list[int]:
        """The layers in the order in which a token passes them; each run has a cache and states of its own."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b = self.loop.start, self.loop.stop
        return [*range(a), *(list(range(a, b)) * self.loop.times), *range(b, n)]

    @property
    def restarts(self) -> set[int]:
        """The runs before which the embedding is added once more."""
        return set() if self.loop is None else {self.loop.start + t * (self.loop.stop - self.loop.start) for t in range(1, self.loop.times)}

    def v_mix_from(self, i: int) -> AttentionMixer | None:
        """The layer whose values layer i mixes into its own (None: it mixes none, or is the first such layer itself)."""
        mixing = [j for j, l in enumerate(self.layers[:i + 1]) if getattr(l.mixer, "v_mix", False)]
        return self.layers[mixing[0]].mixer if len(mixing) > 1 and mixing[-1] == i else None

    @property
    def has_state(self) -> bool:
        """Some layer carries recurrent state (or earlier inputs of a convolution) from token to token."""
        return self.canon > 1 or any(l.mixer.conv > 1 if isinstance(l.mixer, AttentionMixer) else not isinstance(l.mixer, LatentAttentionMixer)
                                     for l in self.layers)

    @property
    def reaches(self) -> list[tuple[int, int]]:
        """The distinct (chunk, window) limits of the attention layers, in order of first use (0 = unlimited)."""
        return list(dict.fromkeys(l.mixer.reach for l in self.layers if isinstance(l.mixer, (AttentionMixer, LatentAttentionMixer))))

    @property
    def pack_prefix(self) -> int:
        """Most cached rows per prompt row that are worth laying out in front of a portion. Latent attention makes their keys
        and values anew by a GEMM, which beats reading the latents once per prompt row at any ratio short of this."""
        return 64 if any(isinstance(l.mixer, LatentAttentionMixer) for l in self.layers) else 4

    def num_params(self) -> int:
        return sum(t.numel() for t in StackWeights(self, "meta", torch.bfloat16).tensors())


# ---- weights -----------------------------------------------------------------------------------------------
class Sections:
    """Row ranges of a merged projection: name -> (offset, rows), every offset a multiple of 8."""

    def __init__(self, **rows: int):
        self.at: dict[str, tuple[int, int]] = {}
        o = 0
        for k, n in rows.items():
            self.at[k] = (o, n)
            o += round8(n)
        self.total = o

    def __getitem__(self, k: str) -> int:
        return self.at[k][0]

    def __contains__(self, k: str) -> bool:
        return k in self.at


def mixer_sections(m) -> Sections:
    if isinstance(m, AttentionMixer):
        s = {"q": m.heads * m.dim}
        if m.kv_from is None:
            s |= {"k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
        if m.head_gate or m.out_gate:
            s["g"] = m.heads * (m.vdim if m.out_gate else 1)
        return Sections(**s)
    if isinstance(m, Mamba2Mixer):
        return Sections(z=m.inner, xbc=m.conv_channels, dt=m.heads)
    if isinstance(m, LatentAttentionMixer):
        return Sections(q=m.heads * m.qk_dim, dkv=m.kv_rank + m.rot_dim, **({"g": m.heads} if m.head_gate else {}))
    if isinstance(m, DeltaMixer):                          # numbers that enter the decay and the step: products stay fp32
        return Sections(q=m.kv_heads * m.dim, k=m.kv_heads * m.dim, v=m.heads * m.vdim, g=m.heads * m.vdim, gates=2 * m.heads)
    if isinstance(m, MLstmMixer):                          # the log gates come last: their products stay fp32
        return Sections(q=m.heads * m.dim, k=m.heads * m.dim, v=m.heads * m.vdim, g=m.heads * m.vdim, gates=2 * m.heads)
    return Sections(q=m.heads * m.dim, k=m.heads * m.dim, v=m.heads * m.vdim, g=m.heads * m.vdim)


def conv_span(m: AttentionMixer) -> int:
    """Columns of the merged projection that the convolutions of an attention layer cover: q, k, v and the padding between them."""
    return sum(round8(n) for n in (m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim))


def mixer_out(m) -> int:
    return m.heads * m.vdim


def mlp_sections(e: DenseMlp | MoeMlp) -> Sections:
    """Rows of a feed-forward's merged input projection (of an MoeMlp: its shared expert and, last, what stays
    fp32: its router and the shared expert's gate)."""
    if isinstance(e, MoeMlp):
        shared = ({"gate": e.shared_ff} if e.gated else {}) | {"up": e.shared_ff}
        return Sections(**(shared if e.shared_ff else {}), router=e.experts, **({"sg": 1} if e.shared_gate else {}))
    return Sections(gate=e.ff, up=e.ff) if e.act == "swiglu" else Sections(up=e.ff)


class StackWeights:
    """Device-resident weights. Matrices are [rows rounded up to 8, cols] views with a row pitch that is a multiple of
    8 elements; norm weights and everything that enters a recurrence are fp32."""

    def __init__(self, cfg: StackConfig, device, dtype: torch.dtype):
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError("layer-stack models run in bfloat16 or float32 (fp16 has no headroom for the recurrent states)")
        self.cfg, self.device, self.dtype = cfg, torch.device(device), dtype
        d = cfg.hidden_size

        def mat(rows, cols):
            return torch.zeros(round8(rows), round8(cols), dtype=dtype, device=device)[:, :cols]

        def vec(n):
            return torch.zeros(n, dtype=torch.float32, device=device)

        self.embed = torch.zeros(cfg.vocab_size, d, dtype=dtype, device=device)
        self.lm_head = mat(cfg.vocab_size, d)
        self.final_norm = vec(d)
        if cfg.tanh_norms:
            self.final_norm_b, self.final_norm_alpha = vec(d), vec(1)
        self.side_embed = torch.zeros(cfg.vocab_size, len(cfg.layers) * cfg.token_side, dtype=dtype, device=device) if cfg.token_side else None
        self.lora = None
        self.layers: list[dict] = []
        for l in cfg.layers:
            m = l.mixer
            w = {"w_in": mat(mixer_sections(m).total, d), "w_out": mat(d, mixer_out(m)), "norm1": vec(d)}
            if isinstance(m, AttentionMixer):
                if m.qk_norm:
                    w["q_norm"] = vec(m.dim)
                    if m.kv_from is None:
                        w["k_norm"] = vec(m.dim)
                if m.row_norm:
                    w |= {"q_norm": vec(m.heads * m.dim), "k_norm": vec(m.kv_heads * m.dim)}
                if m.bias:
                    w["b_in"] = vec(mixer_sections(m).total)
                if m.sink:
                    w["sink"] = vec(m.heads)
                if m.v_mix:
                    w["v_mix"] = vec(1)
                if m.conv:                                 # tap-major, over the convolved sections with the padding between them
                    w["conv"] = torch.zeros(m.conv, conv_span(m), dtype=torch.float32, device=device)
                if m.bias_by is not None:
                    w["rel"] = torch.zeros(m.bias_by.rows, m.heads, dtype=torch.float32, device=device)
            elif isinstance(m, Mamba2Mixer):
                # convolution weights tap-major: one tap's channels are contiguous
                w |= {"conv": torch.zeros(m.conv, round8(m.conv_channels), dtype=torch.float32, device=device),
                      "conv_b": vec(round8(m.conv_channels)), "dt_bias": vec(m.heads), "A_log": vec(m.heads),
                      "D": vec(m.heads), "norm": vec(m.inner)}
            elif isinstance(m, LatentAttentionMixer):
                w |= {"kv_norm": vec(m.kv_rank), "w_uk": mat(m.heads * m.dim, m.kv_rank), "w_uv": mat(m.heads * m.vdim, m.kv_rank)}
                if m.sink:
                    w["sink"] = vec(m.heads)
            elif isinstance(m, MLstmMixer):
                w |= {"gate_b": vec(2 * m.heads), "norm": vec(mixer_out(m))}
            elif isinstance(m, DeltaMixer):
                span = mixer_sections(m)["g"]              # the convolved sections, with the padding between them
                w |= {"conv": torch.zeros(m.conv, span, dtype=torch.float32, device=device), "A_log": vec(m.heads), "dt_bias": vec(m.heads),
                      "norm": vec(m.vdim)}
            else:
                w |= {"decay": torch.tensor(m.decay, dtype=torch.float32).to(device),
                      "norm": vec(mixer_out(m))}
            e = l.mlp
            if e is not None:
                w |= {"w_up": mat(mlp_sections(e).total, d), "norm2": vec(d)}
            if isinstance(e, MoeMlp):
                def stack(rows, cols):
                    return torch.zeros(e.experts, round8(rows), round8(cols), dtype=dtype, device=device)[:, :, :cols]
                # gate and up rows of an expert alternate
                w |= {"correction": vec(e.experts), "e_up": stack((2 if e.gated else 1) * e.ff, d), "e_down": stack(d, e.ff)}
                if e.shared_ff:
                    w["w_down"] = mat(d, e.shared_ff)
            elif e is not None:
                w["w_down"] = mat(d, e.ff)
                if e.act == "polynorm":
                    w["act"] = vec(4)
            if cfg.tanh_norms:
                w |= {k: t for q in ((1, 2) if e is not None else (1,)) for n in (f"norm{q}", f"norm{q}b")
                      for k, t in ((n, vec(d)), (n + ".b", vec(d)), (n + ".alpha", vec(1)))}
            if cfg.token_side:
                w |= {"side_gate": mat(cfg.token_side, d), "side_proj": mat(d, cfg.token_side), "norm3": vec(d)}
            if cfg.streams:
                for q in (1, 2) if l.mlp is not None else (1,):
                    w |= {f"hc{q}.in": vec(cfg.streams), f"hc{q}.out": vec(cfg.streams),
                          f"hc{q}.mix": torch.zeros(cfg.streams, cfg.streams, dtype=torch.float32, device=device),
                          f"canon{q}": torch.zeros(cfg.canon, round8(d), dtype=torch.float32, device=device)}      # tap-major
            self.layers.append(w)
        self.derived: list[dict] = [{} for _ in cfg.layers]      # rearranged copies of weights, made by finish()

    def tensors(self):
        yield from (self.embed, self.lm_head, self.final_norm)
        if self.cfg.tanh_norms:
            yield from (self.final_norm_b, self.final_norm_alpha)
        if self.side_embed is not None:
            yield self.side_embed
        for w in self.layers:
            yield from w.values()

    def section(self, i: int, name: str, of: str = "w_in") -> torch.Tensor:
        """Rows of layer i's merged input projection (of = "b_in": entries of its bias) that belong to `name`."""
        o, n = mixer_sections(self.cfg.layers[i].mixer).at[name]
        return self.layers[i][of][o:o + n]

    def mlp_section(self, i: int, name: str) -> torch.Tensor:
        """The same of its feed-forward's input projection."""
        o, n = mlp_sections(self.cfg.layers[i].mlp).at[name]
        return self.layers[i]["w_up"][o:o + n]

    def fill(self, named, get) -> "StackWeights":
        """Copy the checkpoint tensor get(name) to every (name, destination) of `named`; a list of destinations takes its
        rows one after the other."""
        for name, dst in named:
            src, parts = get(name), dst if isinstance(dst, list) else [dst]
            src = src.reshape(1) if src.dim() == 0 else src              # single numbers
            if sum(p.shape[0] for p in parts) != src.shape[0] or src.shape[1:] != parts[0].shape[1:]:
                raise ValueError(f"tensor {name} has shape {tuple(src.shape)}, which does not fit the configuration")
            o = 0
            for p in parts:
                p.copy_(src[o:o + p.shape[0]])
                o += p.shape[0]
        return self.finish()

    def finish(self) -> "StackWeights":
        """Weights that the kernels want in another arrangement."""
        for i, (l, w) in enumerate(zip(self.cfg.layers, self.layers)):
            m = l.mixer
            if isinstance(m, AttentionMixer) and m.bias_by is not None:
                # per head and distance, less that of the last bucket: softmax does not change, and keys beyond need nothing
                self.derived[i]["bias"] = (w["rel"][m.bias_by.buckets] - w["rel"][-1]).t().contiguous()
            elif isinstance(m, LatentAttentionMixer) and self.device.type == "cuda" and self.dtype != torch.float32:
                # cache row -> [keys | values] of all heads; an identity block hands the rotated part to every head's key
                H, hp = m.heads, m.head_pitch
                e = torch.zeros(2, H, hp, m.cols, dtype=self.dtype, device=self.device)
                e[0, :, :m.dim, :m.kv_rank] = w["w_uk"][:H * m.dim].view(H, m.dim, m.kv_rank)
                e[0, :, m.dim:m.qk_dim, m.rot_at:m.rot_at + m.rot_dim] = torch.eye(m.rot_dim, dtype=self.dtype, device=self.device)
                e[1, :, :m.vdim, :m.kv_rank] = w["w_uv"][:H * m.vdim].view(H, m.vdim, m.kv_rank)
                self.derived[i]["w_expand"] = e.view(2 * H * hp, m.cols)
            elif isinstance(m, DeltaMixer):
                self.derived[i]["norm"] = w["norm"].repeat(m.heads)
                self.derived[i]["conv_b"] = torch.zeros(w["conv"].shape[1], dtype=torch.float32, device=self.device)
        return self
