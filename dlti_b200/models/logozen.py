"""Logozen: a decoder whose layers mix tokens by latent attention (one cached latent per token, a rotated key part shared by
the heads, a sink and an output gate per head) or by mLSTM, with PolyNorm feed-forwards; every sublayer reads a layer norm
and a short causal convolution of a learned combination of several residual streams and writes back to all of them. This
file is the design's config.json reader and its tensor names; the layers themselves are models/stack.py and
serve/stack_runner.py."""
from __future__ import annotations

import json
from pathlib import Path

import torch

from .stack import DenseMlp, LatentAttentionMixer, Layer, MLstmMixer, Rope, StackConfig, StackWeights

ARCHITECTURE = "Logozen"


def _mixer(kind: str, m: dict):
    if kind == "latent_attention":
        rot = m.get("rot")
        return LatentAttentionMixer(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"],
                                    scale=float(m["scale"]), rope=Rope(rot["dims"], float(rot["base"])) if rot else None)
    if kind == "mlstm":
        return MLstmMixer(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], gate_cap=float(m["gate_cap"]))
    raise ValueError(f"unknown mixer type {kind!r}")


def _mlp(m: dict | None):
    if m is None:
        return None
    if m["kind"] != "dense":
        raise ValueError(f"unknown feed-forward kind {m['kind']!r}")
    return DenseMlp(m["ff"], act="polynorm")


class LogozenConfig(StackConfig):
    @classmethod
    def from_dict(cls, d: dict, name: str = "logozen") -> "LogozenConfig":
        return cls(hidden_size=d["width"], vocab_size=d["vocab"], norm_eps=float(d["norm"]["eps"]), norm_one_plus=False,
                   streams=d["streams"], canon=d["canon"]["taps"], embed_scale=float(d["embedding"]["scale"]),
                   layers=[Layer(_mixer(l["type"], l["mixer"]), _mlp(l.get("mlp"))) for l in d["layers"]], name=name)

    def to_dict(self) -> dict:
        out = []
        for l in self.layers:
            m = l.mixer
            if isinstance(m, LatentAttentionMixer):
                kind = "latent_attention"
                e = dict(heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim, kv_rank=m.kv_rank, scale=m.scale)
                if m.rope is not None:
                    e["rot"] = {"base": m.rope.base, "dims": m.rope.dims}
            else:
                kind = "mlstm"
                e = dict(heads=m.heads, dim=m.dim, vdim=m.vdim, gate_cap=m.gate_cap)
            out.append({"type": kind, "mixer": e, "mlp": None if l.mlp is None else {"kind": "dense", "ff": l.mlp.ff}})
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "streams": self.streams,
                "canon": {"taps": self.canon}, "embedding": {"scale": self.embed_scale}, "norm": {"eps": self.norm_eps}, "layers": out}

    @classmethod
    def load(cls, directory: str | Path) -> "LogozenConfig":
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
        for q in (1, 2) if l.mlp is not None else (1,):
            yield p + f"norm{q}", lw[f"norm{q}"]
            for s in ("in", "out", "mix"):
                yield p + f"hc{q}.{s}", lw[f"hc{q}.{s}"]
            yield p + f"canon{q}", lw[f"canon{q}"][:, :d].t()
        yield p + "mix.o", lw["w_out"][:d]
        yield p + "mix.q", w.section(i, "q")
        yield p + "mix.g", w.section(i, "g")
        if isinstance(m, LatentAttentionMixer):
            yield p + "mix.dkv", w.section(i, "dkv")
            yield p + "mix.dkv.norm", lw["kv_norm"]
            yield p + "mix.uk", lw["w_uk"][:m.heads * m.dim]
            yield p + "mix.uv", lw["w_uv"][:m.heads * m.vdim]
            yield p + "mix.sink", lw["sink"]
        else:
            gates = w.section(i, "gates")
            for j, s in enumerate("if"):
                yield p + f"mix.{s}", gates[j * m.heads:(j + 1) * m.heads]
                yield p + f"mix.{s}.b", lw["gate_b"][j * m.heads:(j + 1) * m.heads]
            yield p + "mix.k", w.section(i, "k")
            yield p + "mix.v", w.section(i, "v")
            yield p + "mix.norm", lw["norm"]
        if l.mlp is not None:
            yield p + "mlp.up", lw["w_up"][:l.mlp.ff]
            yield p + "mlp.down", lw["w_down"][:d]
            yield p + "mlp.act", lw["act"]


def load_weights(cfg: LogozenConfig, directory: str | Path, device, dtype: torch.dtype) -> StackWeights:
    from .hf_io import CheckpointReader
    w = StackWeights(cfg, device, dtype)
    return w.fill(named_tensors(w), CheckpointReader(directory).get)


def from_state(cfg: LogozenConfig, state: dict[str, torch.Tensor], device, dtype: torch.dtype) -> StackWeights:
    w = StackWeights(cfg, device, dtype)
    return w.fill(named_tensors(w), state.__getitem__)


def random_state(cfg: LogozenConfig, seed: int = 0, device="cpu") -> dict[str, torch.Tensor]:
    """Random-init checkpoint tensors (bfloat16) of this architecture: fan-in scaled matrices, streams that start out nearly
    separate, forget gates that are mostly open."""
    g = torch.Generator(device=device).manual_seed(seed)
    out: dict[str, torch.Tensor] = {}
    S = cfg.streams
    for name, dst in named_tensors(StackWeights(cfg, "meta", torch.bfloat16)):
        shape, leaf = tuple(dst.shape), name.split(".", 1)[-1]
        t = torch.empty(shape, dtype=torch.float32, device=device)
        if leaf.startswith("canon"):
            t.uniform_(-shape[1] ** -0.5, shape[1] ** -0.5, generator=g).mul_(0.5)
        elif leaf.startswith("hc"):
            t.normal_(0.0, 0.1, generator=g)
            if leaf.endswith("mix"):
                t += torch.eye(S, device=device)
            else:
                t += 1.0 / S if leaf.endswith("in") else 1.0
        elif leaf == "mix.f.b":
            t.normal_(4.0, 1.5, generator=g)
        elif leaf in ("mix.i.b", "mix.sink"):
            t.normal_(0.0, 1.0, generator=g)
        elif leaf == "mlp.act":
            t.normal_(0.3, 0.1, generator=g)
        elif leaf.endswith("norm") or leaf in ("norm1", "norm2"):
            t.normal_(1.0, 0.1, generator=g)
        else:
            t.normal_(0.0, 1.0 if name == "embed" else shape[1] ** -0.5, generator=g)
        out[name] = t.to(torch.bfloat16)
    return out


def save_checkpoint(cfg: LogozenConfig, state: dict[str, torch.Tensor], directory: str | Path) -> None:
    from safetensors.torch import save_file
    cfg.save(directory)
    save_file({k: v.contiguous() for k, v in state.items()}, str(Path(directory) / "model.safetensors"))


def _layers(pattern: str, att: LatentAttentionMixer, mem: MLstmMixer, ff: int) -> list[Layer]:
    return [Layer(att if c == "a" else mem, DenseMlp(ff, act="polynorm")) for c in pattern]


PRESETS = {
    # sizes of a small test model, no two alike
    "logozen-tiny": LogozenConfig(
        hidden_size=152, vocab_size=300, norm_eps=1e-5, norm_one_plus=False, streams=2, canon=4, embed_scale=2.0, name="logozen-tiny",
        layers=_layers("ma", LatentAttentionMixer(heads=5, dim=24, rot_dim=16, vdim=40, kv_rank=80, scale=0.2, rope=Rope(16, 1e4)),
                       MLstmMixer(heads=3, dim=40, vdim=56, gate_cap=9.0), 104)),
    # layer sizes of a ~1B model
    "logozen-1b": LogozenConfig(
        hidden_size=2048, vocab_size=32000, norm_eps=1e-6, norm_one_plus=False, streams=4, canon=4, embed_scale=45.0, name="logozen-1b",
        layers=_layers("mama" * 4, LatentAttentionMixer(heads=16, dim=64, rot_dim=64, vdim=128, kv_rank=512, scale=128 ** -0.5,
                                                        rope=Rope(64, 1e6)),
                       MLstmMixer(heads=8, dim=128, vdim=256, gate_cap=15.0), 8192)),
}
