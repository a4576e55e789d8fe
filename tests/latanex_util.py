"""Small Latanex models for tests/test_latanex.py; the drivers are tests/stack_util.py."""
import torch

from dlti_b200.models import latanex as LX
from tests import ref_latanex as R
from tests.stack_util import Zoo


def _att(heads, kv_heads, dim, vdim, scale, window=0, cap=0.0, v_mix=True):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap, "mask": {"size": window}, "v_mix": v_mix}


def _delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def _moe(experts, top, ff, limit, groups=1, keep=1, scale=1.0, shared=None):
    e = {"kind": "moe", "expert": {"ff": ff, "limit": limit},
         "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": groups, "keep": keep}}}
    return e if shared is None else {**e, "shared": {"ff": shared[0], "limit": shared[1]}}


def _layer(mixer, mlp=None):
    return {"type": "delta" if "conv" in mixer else "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": mlp} if isinstance(mlp, int) else mlp}


def _cfg(vocab, width, scale, logit_scale, eps, *layers):
    return {"architecture": "Latanex", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "logit_scale": logit_scale,
            "norm": {"eps": eps}, "layers": list(layers)}


CONFIGS = {
    # nothing a multiple of 8: every kernel's general form; a layer that does not mix values between two that do
    "odd": _cfg(203, 100, 1.7, 0.3, 1e-5, _layer(_delta(4, 2, 18, 10, 3), _moe(10, 3, 21, 0.6, 5, 2, 1.7, (37, 0.9))),
                _layer(_att(6, 3, 14, 10, 0.4, 23, 4.0), 61), _layer(_att(4, 1, 9, 13, 0.5, 40, 0.0, False), _moe(7, 2, 30, 1.1, shared=(11, 0.5))),
                _layer(_att(3, 3, 20, 10, 0.3, 65, 9.0)), _layer(_delta(3, 3, 7, 35, 5), _moe(6, 4, 19, 0.8, 3, 3, 0.6))),
    # the packed prompt kernel, chunked scans, vectorised row kernels, dense activations in the GEMM's shape; a layer without a feed-forward
    "wide": _cfg(320, 256, 3.0, 2.0, 1e-6, _layer(_att(8, 2, 64, 128, 0.09, 130, 20.0), 128), _layer(_delta(6, 3, 72, 40, 4), _moe(12, 4, 72, 1.5, 4, 2, 2.5, (136, 2.0))),
                 _layer(_att(4, 2, 40, 128, 0.12, 33, 12.0)), _layer(_delta(2, 1, 128, 96, 2), _moe(32, 6, 40, 1.2, 8, 3, 1.5, (64, 1.0)))),
    # ones: one head, one tap, one expert, a window that sees the token itself only
    "ones": _cfg(96, 72, 1.0, 1.0, 1e-5, _layer(_att(1, 1, 8, 8, 0.5, 1, 3.0), _moe(1, 1, 8, 1.0)), _layer(_delta(1, 1, 8, 8, 1), 8),
                 _layer(_att(1, 1, 8, 8, 0.5, 17, 2.0), _moe(2, 1, 16, 1.0, 2, 1, 1.0, (8, 2.0)))),
    # heads above 128 and above 256, unlimited attention, uncapped scores, keys of the recurrence above 128 and above 256
    "tall": _cfg(160, 96, 2.0, 0.7, 1e-5, _layer(_att(4, 2, 136, 144, 0.06), 72), _layer(_delta(2, 1, 256, 64, 4), _moe(5, 2, 48, 2.0, scale=3.0)),
                 _layer(_att(2, 1, 264, 40, 0.05, 90, 6.0, False), _moe(9, 5, 24, 0.7, 3, 2, 1.0, (40, 0.7))), _layer(_delta(2, 2, 300, 24, 3))),
}


def choice_margin(z, correction, r):
    """How far router logits [n, experts] are from another choice: the smallest gap between what is taken and what is left, over
    groups and over experts."""
    c = R.sigmoid(z) + correction
    count, keep = r["groups"]["count"], r["groups"]["keep"]
    n = c.shape[1] // count
    gap = torch.full((c.shape[0],), 9.0, dtype=c.dtype)
    if keep < count:
        g = c.view(-1, count, n).sort(-1, descending=True).values[..., :2].sum(-1).sort(-1, descending=True)
        gap = torch.minimum(gap, g.values[:, keep - 1] - g.values[:, keep])
        shut = torch.ones(c.shape[0], count, dtype=torch.bool).scatter_(1, g.indices[:, :keep], False)
        c = c.masked_fill(shut.repeat_interleave(n, 1), -9.0)
    c = c.sort(-1, descending=True).values
    if r["top"] < c.shape[1]:
        gap = torch.minimum(gap, c[:, r["top"] - 1] - c[:, r["top"]])
    return gap


def _sharpen_for(d):
    def sharpen(st):
        g = torch.Generator().manual_seed(11)
        for k in st:
            if k.endswith("q.norm"):                          # sharp attention: a single key decides
                st[k] = (st[k].float() * 3).bfloat16()
            elif k.endswith("sink"):                          # sinks that weigh as much as the keys
                st[k] = (st[k].float() + 2).bfloat16()
            elif k.endswith("dt_bias"):                       # long and short memories
                st[k] = torch.linspace(-6, 1, st[k].numel()).bfloat16()
        # Routers read a few coordinates that are the token's own: large there, the residual saturates the norm whatever the layers
        # add. Tokens whose choice would be close in some layer get another pattern.
        moe = [(i, l["mlp"]["router"]) for i, l in enumerate(d["layers"]) if l["mlp"] and l["mlp"]["kind"] == "moe"]
        D, V = 16, d["vocab"]
        hidden = lambda i, s: s * st[f"l{i}.norm2"][:D].double() + st[f"l{i}.norm2.b"][:D].double()
        for i, r in moe:
            w = torch.zeros(r["experts"], d["width"])
            w[:, :D] = torch.randn(r["experts"], D, generator=g) * 0.4
            st[f"l{i}.mlp.router"] = w.bfloat16()
            st[f"l{i}.mlp.correction"] = (torch.randn(r["experts"], generator=g) * 0.3 - 0.4).bfloat16()        # also negative choice scores
        best, signs = torch.full((V,), -1.0, dtype=torch.double), torch.zeros(V, D)
        for _ in range(400):
            s = torch.randint(0, 2, (V, D), generator=g).double() * 2 - 1
            gap = torch.full((V,), 9.0, dtype=torch.double)
            for i, r in moe:
                z = hidden(i, s) @ st[f"l{i}.mlp.router"][:, :D].double().t()
                gap = torch.minimum(gap, choice_margin(z, st[f"l{i}.mlp.correction"].double(), r))
            better = gap > best
            best = torch.where(better, gap, best)
            signs[better] = s[better].float()
        assert best.min() > 0.01, float(best.min())
        st["embed"][:, :D] = (signs * 40 / d["embedding"]["scale"]).bfloat16()
    return sharpen


class LatanexZoo(Zoo):
    def __init__(self):
        super().__init__(LX, LX.LatanexConfig, R, CONFIGS, None)

    def model(self, name, seed=0):
        d = self.configs[name]
        cfg = self.config_cls.from_dict(d, name=name)
        st = self.design.random_state(cfg, seed)
        _sharpen_for(d)(st)
        return d, cfg, st, {k: v.double() for k, v in st.items()}


ZOO = LatanexZoo()
