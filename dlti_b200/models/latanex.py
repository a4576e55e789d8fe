"""Latanex: a decoder whose layers mix tokens by windowed softmax attention (biased projections, norms over whole query and
key rows, capped scores, a sink per head, values mixed with those of the first attention layer) or by a gated delta rule,
with dense SwiGLU feed-forwards or mixtures of clipped experts, and a dynamic tanh norm before and after every sublayer.
This file is the design's config.json reader and its tensor names; the layers themselves are models/stack.py and
serve/stack_runner.py."""
from __future__ import annotations

import json
from pathlib import Path

import torch

from .stack import AttentionMixer, DeltaMixer, DenseMlp, Layer, MoeMlp, StackConfig, StackWeights, mixer_sections

ARCHITECTURE = "Latanex"


def _mixer(kind: str, m: dict):
    if kind == "attention":
        return AttentionMixer(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=float(m["scale"]),
                              qk_norm=False, head_gate=False, window=int((m.get("mask") or {}).get("size") or 0),
                              softcap=float(m.get("softcap") or 0.0), sink=True, bias=True, row_norm=True, v_mix=bool(m.get("v_mix")))
    if kind == "delta":
        return DeltaMixer(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], conv=m["conv"])
    raise ValueError(f"unknown mixer type {kind!r}")


def _mlp(m: dict | None):
    if m is None:
        return None
    if m["kind"] == "dense":
        return DenseMlp(m["ff"], act="swiglu")
    if m["kind"] == "moe":
        r, e, s = m["router"], m["expert"], m.get("shared")
        g = r.get("groups") or {"count": 1, "keep": 1}
        return MoeMlp(experts=r["experts"], top=r["top"], ff=e["ff"], limit=float(e["limit"]), groups=g["count"], keep=g["keep"],
                      scale=float(r["scale"]), shared_ff=s["ff"] if s else 0, shared_limit=float(s["limit"]) if s else 0.0)
    raise ValueError(f"unknown feed-forward kind {m['kind']!r}")


class LatanexConfig(StackConfig):
    @classmethod
    def from_dict(cls, d: dict, name: str = "latanex") -> "LatanexConfig":
        return cls(hidden_size=d["width"], vocab_size=d["vocab"], norm_eps=float(d["norm"]["eps"]), norm_one_plus=False, tanh_norms=True,
                   embed_scale=float(d["embedding"]["scale"]), logit_scale=float(d["logit_scale"]),
                   layers=[Layer(_mixer(l["type"], l["mixer"]), _mlp(l.get("mlp"))) for l in d["layers"]], name=name)

    def to_dict(self) -> dict:
        out = []
        for l in self.layers:
            m, e = l.mixer, l.mlp
            mix = dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim)
            if isinstance(m, AttentionMixer):
                kind = "attention"
                mix |= {"scale": m.scale, "softcap": m.softcap, "mask": {"size": m.window}, "v_mix": m.v_mix}
            else:
                kind = "delta"
                mix |= {"conv": m.conv}
            if isinstance(e, MoeMlp):
                mlp = {"kind": "moe", "expert": {"ff": e.ff, "limit": e.limit},
                       "router": {"experts": e.experts, "top": e.top, "scale": e.scale, "groups": {"count": e.groups, "keep": e.keep}}}
                if e.shared_ff:
                    mlp["shared"] = {"ff": e.shared_ff, "limit": e.shared_limit}
            else:
                mlp = None if e is None else {"kind": "dense", "ff": e.ff}
            out.append({"type": kind, "mixer": mix, "mlp": mlp})
        return {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "embedding": {"scale": self.embed_scale},
                "logit_scale": self.logit_scale, "norm": {"eps": self.norm_eps}, "layers": out}

    @classmethod
    def load(cls, directory: str | Path) -> "LatanexConfig":
        with open(Path(directory) / "config.json") as f:
            return cls.from_dict(json.load(f), name=Path(directory).name)

    def save(self, directory: str | Path) -> None:
        Path(directory).mkdir(parents=True, exist_ok=True)
        with open(Path(directory) / "config.json", "w") as f:
            json.dump(self.to_dict(), f, indent=1)


def named_tensors(w: StackWeights):
    """(checkpoint name, destination view) of every tensor of the design; the view has the checkpoint's shape (single numbers:
    one element)."""
    cfg = w.cfg
    V, d = cfg.vocab_size, cfg.hidden_size
    yield "embed", w.embed
    yield "head", w.lm_head[:V]
    yield "final.norm", w.final_norm
    yield "final.norm.b", w.final_norm_b
    yield "final.norm.alpha", w.final_norm_alpha
    for i, (l, lw) in enumerate(zip(cfg.layers, w.layers)):
        m, e, p = l.mixer, l.mlp, f"l{i}."
        for q in (1, 2) if e is not None else (1,):
            for n in (f"norm{q}", f"norm{q}b"):
                for s in ("", ".b", ".alpha"):
                    yield p + n + s, lw[n + s]
        yield p + "mix.o", lw["w_out"][:d]
        for s in "qkv":
            yield p + "mix." + s, w.section(i, s)
        if isinstance(m, AttentionMixer):
            for s in "qkv":
                yield p + f"mix.{s}.b", w.section(i, s, "b_in")
            yield p + "mix.q.norm", lw["q_norm"]
            yield p + "mix.k.norm", lw["k_norm"]
            yield p + "mix.sink", lw["sink"]
            if cfg.v_mix_from(i) is not None:
                yield p + "mix.vmix", lw["v_mix"]
        else:
            sec, gates = mixer_sections(m), w.section(i, "gates")
            for s in "qkv":
                o, n = sec.at[s]
                yield p + f"mix.{s}.conv", lw["conv"][:, o:o + n].t()
            yield p + "mix.g", w.section(i, "g")
            yield p + "mix.a", gates[:m.heads]
            yield p + "mix.b", gates[m.heads:]
            for s in ("A_log", "dt_bias", "norm"):
                yield p + "mix." + s, lw[s]
        if isinstance(e, MoeMlp):
            for j in range(e.experts):
                yield p + f"mlp.e{j}.gate", lw["e_up"][j, 0:2 * e.ff:2]
                yield p + f"mlp.e{j}.up", lw["e_up"][j, 1:2 * e.ff:2]
                yield p + f"mlp.e{j}.down", lw["e_down"][j, :d]
            yield p + "mlp.router", w.mlp_section(i, "router")
            yield p + "mlp.correction", lw["correction"]
        pre = "mlp.shared." if isinstance(e, MoeMlp) else "mlp."
        if e is not None and "w_down" in lw:
            yield p + pre + "gate", w.mlp_section(i, "gate")
            yield p + pre + "up", w.mlp_section(i, "up")
            yield p + pre + "down", lw["w_down"][:d]


def load_weights(cfg: LatanexConfig, directory: str | Path, device, dtype: torch.dtype) -> StackWeights:
    from .hf_io import CheckpointReader
    w = StackWeights(cfg, device, dtype)
    return w.fill(named_tensors(w), CheckpointReader(directory).get)


def from_state(cfg: LatanexConfig, state: dict[str, torch.Tensor], device, dtype: torch.dtype) -> StackWeights:
    w = StackWeights(cfg, device, dtype)
    return w.fill(named_tensors(w), state.__getitem__)


def random_state(cfg: LatanexConfig, seed: int = 0, device="cpu") -> dict[str, torch.Tensor]:
    """Random-init checkpoint tensors (bfloat16) of this architecture: fan-in scaled matrices, decays in the range such layers are
    trained from, norms that start out in the straight part of the tanh."""
    g = torch.Generator(device=device).manual_seed(seed)
    out: dict[str, torch.Tensor] = {}
    for name, dst in named_tensors(StackWeights(cfg, "meta", torch.bfloat16)):
        shape, leaf = tuple(dst.shape), name.split(".", 1)[-1]
        t = torch.empty(shape, dtype=torch.float32, device=device)
        if leaf.endswith(".alpha"):
            t.uniform_(0.3, 0.8, generator=g)
            t = t.reshape(())
        elif leaf.endswith(".conv"):
            t.uniform_(-shape[1] ** -0.5, shape[1] ** -0.5, generator=g)
        elif leaf == "mix.A_log":
            t.uniform_(1.0, 16.0, generator=g).log_()
        elif leaf == "mix.dt_bias":
            t.uniform_(-6.9, -2.3, generator=g).exp_()
            t.expm1_().log_()
        elif leaf == "mix.vmix":
            t.uniform_(0.2, 0.8, generator=g)
            t = t.reshape(())
        elif leaf == "mix.sink":
            t.normal_(0.0, 1.0, generator=g)
        elif leaf.endswith(".b") and len(shape) == 1 or leaf == "mlp.correction":
            t.normal_(0.0, 0.1, generator=g)
        elif leaf.endswith("norm") or leaf.startswith("norm"):
            t.normal_(1.0, 0.1, generator=g)
        else:
            t.normal_(0.0, 1.0 if name == "embed" else shape[1] ** -0.5, generator=g)
        out[name] = t.to(torch.bfloat16)
    return out


def save_checkpoint(cfg: LatanexConfig, state: dict[str, torch.Tensor], directory: str | Path) -> None:
    from safetensors.torch import save_file
    cfg.save(directory)
    save_file({k: v.contiguous() for k, v in state.items()}, str(Path(directory) / "model.safetensors"))


def _att(heads: int, kv_heads: int, dim: int, vdim: int, window: int, cap: float = 50.0) -> AttentionMixer:
    return AttentionMixer(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=dim ** -0.5, qk_norm=False, head_gate=False,
                          window=window, softcap=cap, sink=True, bias=True, row_norm=True, v_mix=True)


def _model(name: str, width: int, vocab: int, layers: list[Layer], eps: float = 1e-6, embed: float = 4.0, logits: float = 0.5) -> LatanexConfig:
    return LatanexConfig(hidden_size=width, vocab_size=vocab, norm_eps=eps, norm_one_plus=False, tanh_norms=True, embed_scale=embed,
                         logit_scale=logits, layers=layers, name=name)


PRESETS = {
    # sizes of a small test model, no two alike
    "latanex-tiny": _model("latanex-tiny", 144, 300, [
        Layer(DeltaMixer(heads=4, kv_heads=2, dim=24, vdim=40, conv=3), DenseMlp(104, act="swiglu")),
        Layer(_att(6, 3, 32, 48, 56), MoeMlp(experts=8, top=3, ff=72, limit=2.0, groups=4, keep=2, scale=1.5, shared_ff=88, shared_limit=3.0)),
        Layer(_att(6, 3, 32, 48, 56), None)]),
    # layer sizes of a ~3B model with ~0.7B active parameters: a windowed attention layer after every three delta layers
    "latanex-3b": _model("latanex-3b", 2048, 32000, [
        Layer(_att(16, 4, 128, 128, 2048) if i % 4 == 3 else DeltaMixer(heads=16, kv_heads=16, dim=128, vdim=128, conv=4),
              DenseMlp(8192, act="swiglu") if i == 0 else
              MoeMlp(experts=64, top=6, ff=512, limit=7.0, groups=8, keep=4, scale=2.5, shared_ff=1024, shared_limit=7.0))
        for i in range(12)]),
}
