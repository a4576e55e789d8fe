"""Models described layer by layer: each layer names its token mixer (softmax attention, Mamba-2, lightning attention)
and its feed-forward, with every size and constant a parameter. A design (models/sigosun.py) is a parser from its
config.json to a `StackConfig` plus its tensor names; the weights container, the cache layout and the serving forward
pass (serve/stack_runner.py) are shared by all of them.

Weights are kept as merged input projections, one GEMM per mixer. Every section of a merged projection and the row
pitch of every matrix is rounded up to 8 elements, so any head count or width meets the 16-byte rules of the TMA
GEMMs; padding rows are zero and padding columns are never read.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch


def round8(n: int) -> int:
    return (n + 7) // 8 * 8


# ---- layer descriptions ------------------------------------------------------------------------------------
@dataclass(frozen=True)
class Rope:
    dims: int                      # leading dimensions of a head that are rotated
    base: float
    interleaved: bool = True       # pairs (2i, 2i+1); False: (i, i + dims/2)


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
class DenseMlp:
    ff: int
    act: str = "relu2"             # square of relu


@dataclass(frozen=True)
class Layer:
    mixer: AttentionMixer | Mamba2Mixer | LightningMixer
    mlp: DenseMlp | None = None


@dataclass
class StackConfig:
    hidden_size: int
    vocab_size: int
    norm_eps: float
    layers: list[Layer]
    norm_one_plus: bool = True     # layer and final norm weights are stored around zero: 1 + w
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
            elif isinstance(m, Mamba2Mixer):
                if m.heads % m.groups or m.inner % m.norm_groups:
                    raise ValueError(f"layer {i}: groups must divide the heads and norm_groups the inner size")
            elif len(m.decay) != m.heads:
                raise ValueError(f"layer {i}: {len(m.decay)} decays for {m.heads} heads")

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def has_state(self) -> bool:
        """Some layer carries recurrent state from token to token."""
        return any(not isinstance(l.mixer, AttentionMixer) for l in self.layers)

    @property
    def chunks(self) -> list[int]:
        """The distinct attention chunk sizes, in order of first use (0 = unlimited)."""
        out: list[int] = []
        for l in self.layers:
            if isinstance(l.mixer, AttentionMixer) and l.mixer.chunk not in out:
                out.append(l.mixer.chunk)
        return out

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
        if m.head_gate:
            s["g"] = m.heads
        return Sections(**s)
    if isinstance(m, Mamba2Mixer):
        return Sections(z=m.inner, xbc=m.conv_channels, dt=m.heads)
    return Sections(q=m.heads * m.dim, k=m.heads * m.dim, v=m.heads * m.vdim, g=m.heads * m.vdim)


def mixer_out(m) -> int:
    return m.heads * m.vdim


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
            elif isinstance(m, Mamba2Mixer):
                # convolution weights tap-major: one tap's channels are contiguous
                w |= {"conv": torch.zeros(m.conv, round8(m.conv_channels), dtype=torch.float32, device=device),
                      "conv_b": vec(round8(m.conv_channels)), "dt_bias": vec(m.heads), "A_log": vec(m.heads),
                      "D": vec(m.heads), "norm": vec(m.inner)}
            else:
                w |= {"decay": torch.tensor(m.decay, dtype=torch.float32).to(device),
                      "norm": vec(mixer_out(m))}
            if l.mlp is not None:
                w |= {"w_up": mat(l.mlp.ff, d), "w_down": mat(d, l.mlp.ff), "norm2": vec(d)}
            self.layers.append(w)

    def tensors(self):
        yield from (self.embed, self.lm_head, self.final_norm)
        for w in self.layers:
            yield from w.values()

    def section(self, i: int, name: str) -> torch.Tensor:
        """Rows of layer i's merged input projection that belong to `name`."""
        o, n = mixer_sections(self.cfg.layers[i].mixer).at[name]
        return self.layers[i]["w_in"][o:o + n]
