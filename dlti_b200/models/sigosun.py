"""Sigosun: a decoder whose layers mix tokens by chunked softmax attention (per-head output gates, optionally the keys
and values of an earlier layer), Mamba-2 or lightning attention, with squared-relu feed-forwards and norms on the
sublayer outputs only. This file is the design's config.json reader and its tensor names; the layers themselves are
models/stack.py and serve/stack_runner.py."""
from __future__ import annotations

import json
from pathlib import Path

import torch

from .stack import (AttentionMixer, DenseMlp, Layer, LightningMixer, Mamba2Mixer, Rope, StackConfig, StackWeights)

ARCHITECTURE = "Sigosun"


def _mixer(kind: str, m: dict):
    if kind == "attention":
        rot = m.get("rot")
        return AttentionMixer(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                              rope=Rope(rot["dims"], float(rot["base"])) if rot else None,
                              chunk=int((m.get("mask") or {}).get("size") or 0), kv_from=m.get("kv_from"))
    if kind == "mamba2":
        return Mamba2Mixer(heads=m["heads"], vdim=m["vdim"], state=m["state"], groups=m["groups"], conv=m["conv"],
                           norm_groups=m["norm_groups"])
    if kind == "lightning":
        return LightningMixer(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], decay=tuple(float(x) for x in m["decay"]))
    raise ValueError(f"unknown mixer type {kind!r}")


def _mlp(m: dict | None):
    if m is None:
        return None
    if m["kind"] != "dense":
        raise ValueError(f"unknown feed-forward kind {m['kind']!r}")
    return DenseMlp(m["ff"])


class SigosunConfig(StackConfig):
    @classmethod
    def from_dict(cls, d: dict, name: str = "sigosun") -> "SigosunConfig":
        return cls(hidden_size=d["width"], vocab_size=d["vocab"], norm_eps=float(d["norm"]["eps"]),
                   layers=[Layer(_mixer(l["type"], l["mixer"]), _mlp(l.get("mlp"))) for l in d["layers"]], name=name)

    def to_dict(self) -> dict:
        out = []
        for l in self.layers:
            m = l.mixer
            if isinstance(m, AttentionMixer):
                kind = "attention"
                e = dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, mask={"size": m.chunk})
                if m.rope is not None:
                    e["rot"] = {"base": m.rope.base, "dims": m.rope.dims}
                if m.kv_from is not None:
                    e["kv_from"] = m.kv_from
            elif isinstance(m, Mamba2Mixer):
                kind = "mamba2"
                e = dict(heads=m.heads, vdim=m.vdim, state=m.state, groups=m.groups, conv=m.conv, norm_groups=m.norm_groups)
            else:
                kind = "lightning"
                e = dict(heads=m.heads, dim=m.dim, vdim=m.vdim, decay=list(m.decay))
            out.append({"type": kind, "mixer": e, "mlp": None if l.mlp is None else {"kind": "dense", "ff": l.mlp.ff}})
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size,
                "norm": {"eps": self.norm_eps}, "layers": out}

    @classmethod
    def load(cls, directory: str | Path) -> "SigosunConfig":
        with open(Path(directory) / "config.json") as f:
            return cls.from_dict(json.load(f), name=Path(directory).name)

    def save(self, directory: str | Path) -> None:
        Path(directory).mkdir(parents=True, exist_ok=True)
        with open(Path(directory) / "config.json", "w") as f:
            json.dump(self.to_dict(), f, indent=1)


def named_tensors(w: StackWeights):
    """(checkpoint name, destination view) of every tensor of the design; the view has the checkpoint's shape."""
    cfg = w.cfg
    V, d = cfg.vocab_size, cfg.hidden_size
    yield "embed", w.embed
    yield "head", w.lm_head[:V]
    yield "final.norm", w.final_norm
    for i, (l, lw) in enumerate(zip(cfg.layers, w.layers)):
        m, p = l.mixer, f"l{i}."
        yield p + "norm1", lw["norm1"]
        yield p + "mix.o", lw["w_out"][:d]
        if isinstance(m, AttentionMixer):
            names = ["q", "g"] + (["k", "v"] if m.kv_from is None else [])
            for s in names:
                yield p + "mix." + s, w.section(i, s)
            yield p + "mix.q.norm", lw["q_norm"]
            if m.kv_from is None:
                yield p + "mix.k.norm", lw["k_norm"]
        elif isinstance(m, Mamba2Mixer):
            # one stored matrix [z | x | B | C | dt]; in memory its sections start at multiples of 8 rows
            yield p + "mix.in", [w.section(i, "z"), w.section(i, "xbc"), w.section(i, "dt")]
            yield p + "mix.conv", lw["conv"][:, :m.conv_channels].t()
            yield p + "mix.conv.b", lw["conv_b"][:m.conv_channels]
            for s in ("dt_bias", "A_log", "D", "norm"):
                yield p + "mix." + s, lw[s]
        else:
            for s in "qkvg":
                yield p + "mix." + s, w.section(i, s)
            yield p + "mix.norm", lw["norm"]
        if l.mlp is not None:
            yield p + "norm2", lw["norm2"]
            yield p + "mlp.up", lw["w_up"][:l.mlp.ff]
            yield p + "mlp.down", lw["w_down"][:d]


def load_weights(cfg: SigosunConfig, directory: str | Path, device, dtype: torch.dtype) -> StackWeights:
    from .hf_io import CheckpointReader
    w = StackWeights(cfg, device, dtype)
    return w.fill(named_tensors(w), CheckpointReader(directory).get)


def random_state(cfg: SigosunConfig, seed: int = 0, device="cpu") -> dict[str, torch.Tensor]:
    """Random-init checkpoint tensors (bfloat16) of this architecture: fan-in scaled matrices, convolution and decay
    parameters in the ranges such layers are trained from."""
    g = torch.Generator(device=device).manual_seed(seed)
    out: dict[str, torch.Tensor] = {}
    for name, dst in named_tensors(StackWeights(cfg, "meta", torch.bfloat16)):
        shape = (sum(p.shape[0] for p in dst), dst[0].shape[1]) if isinstance(dst, list) else tuple(dst.shape)
        leaf = name.split(".", 1)[1] if "." in name else name
        t = torch.empty(shape, dtype=torch.float32, device=device)
        if leaf == "mix.conv":
            t.uniform_(-shape[1] ** -0.5, shape[1] ** -0.5, generator=g)
        elif leaf == "mix.A_log":
            t.uniform_(1.0, 16.0, generator=g).log_()
        elif leaf == "mix.dt_bias":
            t.uniform_(-6.9, -2.3, generator=g).exp_()
            t.expm1_().log_()
        elif leaf == "mix.D" or leaf.endswith("q.norm") or leaf.endswith("k.norm") or leaf == "mix.norm":
            t.normal_(1.0, 0.1, generator=g)
        elif len(shape) == 1:
            t.normal_(0.0, 0.1, generator=g)
        else:
            t.normal_(0.0, 1.0 if name == "embed" else shape[1] ** -0.5, generator=g)
        out[name] = t.to(torch.bfloat16)
    return out


def from_state(cfg: SigosunConfig, state: dict[str, torch.Tensor], device, dtype: torch.dtype) -> StackWeights:
    w = StackWeights(cfg, device, dtype)
    return w.fill(named_tensors(w), state.__getitem__)


def save_checkpoint(cfg: SigosunConfig, state: dict[str, torch.Tensor], directory: str | Path) -> None:
    from safetensors.torch import save_file
    cfg.save(directory)
    save_file({k: v.contiguous() for k, v in state.items()}, str(Path(directory) / "model.safetensors"))


_ATTN_1B = AttentionMixer(heads=16, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, rope=Rope(128, 500000.0), chunk=2048)
_MAMBA_1B = Mamba2Mixer(heads=64, vdim=64, state=128, groups=1, conv=4, norm_groups=1)
_LIGHT_1B = LightningMixer(heads=16, dim=128, vdim=128, decay=tuple(1 - 2.0 ** (-5 - 0.25 * h) for h in range(16)))


def _shared(m: AttentionMixer, src: int) -> AttentionMixer:
    from dataclasses import replace
    return replace(m, kv_from=src)


PRESETS = {
    # sizes of a small test model: no two sizes alike, groups and norm groups above 1, a shared key/value layer
    "sigosun-tiny": SigosunConfig(
        hidden_size=136, vocab_size=300, norm_eps=1e-5, name="sigosun-tiny", layers=[
            Layer(Mamba2Mixer(heads=4, vdim=24, state=40, groups=2, conv=3, norm_groups=4), DenseMlp(88)),
            Layer(AttentionMixer(heads=6, kv_heads=3, dim=32, vdim=40, scale=0.2, rope=Rope(20, 1e4), chunk=48), DenseMlp(104)),
            Layer(LightningMixer(heads=3, dim=40, vdim=24, decay=(0.5, 0.9, 0.995)), None),
            Layer(AttentionMixer(heads=9, kv_heads=3, dim=32, vdim=40, scale=0.15, rope=Rope(20, 1e4), chunk=80, kv_from=1), None),
        ]),
    # layer sizes of a ~1B model: attention, attention on shared keys/values, Mamba-2, lightning, four times
    "sigosun-1b": SigosunConfig(
        hidden_size=2048, vocab_size=32000, norm_eps=1e-6, name="sigosun-1b",
        layers=[x for i in range(4) for x in (
            Layer(_ATTN_1B, DenseMlp(8192)), Layer(_shared(_ATTN_1B, 4 * i), DenseMlp(8192)),
            Layer(_MAMBA_1B, None), Layer(_LIGHT_1B, None))]),
}
