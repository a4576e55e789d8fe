"""Ridazen: a pre-norm decoder of softmax attention (short convolutions on queries, keys and values, per-head norms, positions
only through a learned bias by distance and a query temperature, an output gate per element) with mixtures of squared-relu
experts and a gated shared one; every layer ends with an input of the token's own, and a part of the stack runs several times.
This file is the design's config.json reader and its tensor names; the layers themselves are models/stack.py and
serve/stack_runner.py."""
from __future__ import annotations

import json
from pathlib import Path

import torch

from .stack import AttentionMixer, DistanceBias, Layer, Loop, MoeMlp, QueryTemp, StackConfig, StackWeights, mixer_sections

ARCHITECTURE = "Ridazen"
BIAS_ROWS = 32               # distance buckets of models that are not loaded: otherwise the checkpoint's tensors say how many


def _mixer(kind: str, m: dict, bias_rows: int):
    if kind != "attention":
        raise ValueError(f"unknown mixer type {kind!r}")
    t = m.get("q_temp")
    return AttentionMixer(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]), head_gate=False,
                          conv=int(m.get("conv") or 0), q_temp=QueryTemp(float(t["coef"]), t["every"]) if t else None,
                          bias_by=DistanceBias(m.get("bias_rows", bias_rows), m["bias_max"]) if m.get("bias_max") else None, out_gate=True)


def _mlp(m: dict | None):
    if m is None:
        return None
    if m["kind"] != "moe":
        raise ValueError(f"unknown feed-forward kind {m['kind']!r}")
    r, s = m["router"], m.get("shared")
    return MoeMlp(experts=r["experts"], top=r["top"], ff=m["expert"]["ff"], act="relu2", score="softmax", shared_ff=s["ff"] if s else 0,
                  shared_gate=bool(s))


class RidazenConfig(StackConfig):
    @classmethod
    def from_dict(cls, d: dict, name: str = "ridazen", bias_rows: list[int] | None = None) -> "RidazenConfig":
        """bias_rows: distance buckets layer by layer, where config.json leaves them to the checkpoint."""
        loop, side, layers = d.get("loop"), d.get("token_side"), d["layers"]
        rows = bias_rows or [BIAS_ROWS] * len(layers)
        return cls(hidden_size=d["width"], vocab_size=d["vocab"], norm_eps=float(d["norm"]["eps"]), norm_one_plus=False, pre_norm=True,
                   residual_mult=float(d.get("residual_mult", 1.0)), token_side=side["dim"] if side else 0,
                   loop=Loop(loop["start"], loop["stop"], loop["times"]) if loop else None, logit_scale=float(d.get("logit_scale", 1.0)),
                   logit_softcap=float(d.get("logit_softcap") or 0.0),
                   layers=[Layer(_mixer(l["type"], l["mixer"], n), _mlp(l.get("mlp"))) for l, n in zip(layers, rows)], name=name)

    def to_dict(self) -> dict:
        out = []
        for l in self.layers:
            m, e = l.mixer, l.mlp
            mix = dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, conv=m.conv)
            if m.q_temp is not None:
                mix["q_temp"] = {"coef": m.q_temp.coef, "every": m.q_temp.every}
            if m.bias_by is not None:
                mix |= {"bias_max": m.bias_by.far, "bias_rows": m.bias_by.rows}
            mlp = None
            if e is not None:
                mlp = {"kind": "moe", "expert": {"ff": e.ff}, "router": {"experts": e.experts, "top": e.top}}
                if e.shared_ff:
                    mlp["shared"] = {"ff": e.shared_ff}
            out.append({"type": "attention", "mixer": mix, "mlp": mlp})
        d = {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
             "residual_mult": self.residual_mult, "logit_scale": self.logit_scale, "logit_softcap": self.logit_softcap, "layers": out}
        if self.token_side:
            d["token_side"] = {"dim": self.token_side}
        if self.loop is not None:
            d["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return d

    @classmethod
    def load(cls, directory: str | Path) -> "RidazenConfig":
        from .hf_io import CheckpointReader
        with open(Path(directory) / "config.json") as f:
            d = json.load(f)
        rows = [BIAS_ROWS] * len(d["layers"])
        try:
            ckpt = CheckpointReader(directory)
        except FileNotFoundError:                          # a configuration without weights
            ckpt = None
        for i in range(len(rows)):
            if ckpt is not None and ckpt.has(f"l{i}.mix.rel"):
                rows[i] = ckpt.shape(f"l{i}.mix.rel")[0]
        return cls.from_dict(d, Path(directory).name, rows)

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
    if cfg.token_side:
        yield "side.embed", w.side_embed
    for i, (l, lw) in enumerate(zip(cfg.layers, w.layers)):
        m, e, p = l.mixer, l.mlp, f"l{i}."
        yield p + "norm1", lw["norm1"]
        sec = mixer_sections(m)
        for s in "qkvg":
            yield p + "mix." + s, w.section(i, s)
        if m.conv:
            for s in "qkv":
                o, n = sec.at[s]
                yield p + f"mix.{s}.conv", lw["conv"][:, o:o + n].t()
        yield p + "mix.q.norm", lw["q_norm"]
        yield p + "mix.k.norm", lw["k_norm"]
        if m.bias_by is not None:
            yield p + "mix.rel", lw["rel"]
        yield p + "mix.o", lw["w_out"][:d]
        if e is not None:
            yield p + "norm2", lw["norm2"]
            for j in range(e.experts):
                yield p + f"mlp.e{j}.up", lw["e_up"][j, :e.ff]
                yield p + f"mlp.e{j}.down", lw["e_down"][j, :d]
            yield p + "mlp.router", w.mlp_section(i, "router")
            yield p + "mlp.router.b", lw["correction"]
            if e.shared_ff:
                yield p + "mlp.shared.up", w.mlp_section(i, "up")
                yield p + "mlp.shared.down", lw["w_down"][:d]
                yield p + "mlp.shared.sg", w.mlp_section(i, "sg")
        if cfg.token_side:
            yield p + "side.gate", lw["side_gate"][:cfg.token_side]
            yield p + "side.proj", lw["side_proj"][:d]
            yield p + "side.norm", lw["norm3"]


def load_weights(cfg: RidazenConfig, directory: str | Path, device, dtype: torch.dtype) -> StackWeights:
    from .hf_io import CheckpointReader
    w = StackWeights(cfg, device, dtype)
    return w.fill(named_tensors(w), CheckpointReader(directory).get)


def from_state(cfg: RidazenConfig, state: dict[str, torch.Tensor], device, dtype: torch.dtype) -> StackWeights:
    w = StackWeights(cfg, device, dtype)
    return w.fill(named_tensors(w), state.__getitem__)


def random_state(cfg: RidazenConfig, seed: int = 0, device="cpu") -> dict[str, torch.Tensor]:
    """Random-init checkpoint tensors (bfloat16) of this architecture: fan-in scaled matrices, norm weights around one."""
    g = torch.Generator(device=device).manual_seed(seed)
    out: dict[str, torch.Tensor] = {}
    for name, dst in named_tensors(StackWeights(cfg, "meta", torch.bfloat16)):
        shape, leaf = tuple(dst.shape), name.split(".", 1)[-1]
        t = torch.empty(shape, dtype=torch.float32, device=device)
        if leaf.endswith(".conv"):
            t.uniform_(-shape[1] ** -0.5, shape[1] ** -0.5, generator=g)
        elif leaf == "mix.rel":
            t.normal_(0.0, 1.0, generator=g)
        elif leaf == "mlp.router.b":
            t.normal_(0.0, 0.1, generator=g)
        elif leaf.endswith("norm") or leaf.startswith("norm"):
            t.normal_(1.0, 0.1, generator=g)
        else:
            t.normal_(0.0, 1.0 if name in ("embed", "side.embed") else shape[1] ** -0.5, generator=g)
        out[name] = t.to(torch.bfloat16)
    return out


def save_checkpoint(cfg: RidazenConfig, state: dict[str, torch.Tensor], directory: str | Path) -> None:
    from safetensors.torch import save_file
    cfg.save(directory)
    save_file({k: v.contiguous() for k, v in state.items()}, str(Path(directory) / "model.safetensors"))


def _att(heads: int, kv_heads: int, dim: int, vdim: int, conv: int, rows: int, far: int) -> AttentionMixer:
    return AttentionMixer(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=dim ** -0.5, head_gate=False, conv=conv,
                          q_temp=QueryTemp(0.1, 1024), bias_by=DistanceBias(rows, far), out_gate=True)


def _moe(experts: int, top: int, ff: int, shared: int) -> MoeMlp:
    return MoeMlp(experts=experts, top=top, ff=ff, act="relu2", score="softmax", shared_ff=shared, shared_gate=shared > 0)


def _model(name: str, width: int, vocab: int, layers: list[Layer], side: int, loop: Loop, eps: float = 1e-6) -> RidazenConfig:
    return RidazenConfig(hidden_size=width, vocab_size=vocab, norm_eps=eps, norm_one_plus=False, pre_norm=True, residual_mult=0.7,
                         token_side=side, loop=loop, logit_scale=0.8, logit_softcap=25.0, layers=layers, name=name)


PRESETS = {
    # sizes of a small test model, no two alike
    "ridazen-tiny": _model("ridazen-tiny", 136, 300, [
        Layer(_att(6, 3, 32, 40, 4, 12, 70), _moe(9, 3, 56, 88)), Layer(_att(4, 2, 24, 48, 2, 20, 50), _moe(5, 2, 72, 0)),
        Layer(_att(3, 1, 40, 24, 3, 10, 33), None)], side=20, loop=Loop(1, 2, 3)),
    # layer sizes of a ~3B model with ~0.7B active parameters, its middle run twice
    "ridazen-3b": _model("ridazen-3b", 2048, 32000, [Layer(_att(16, 4, 128, 128, 4, 32, 128), _moe(64, 8, 768, 1536)) for _ in range(12)],
                         side=128, loop=Loop(4, 8, 2)),
}
