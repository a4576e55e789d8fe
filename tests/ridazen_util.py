"""Small Ridazen models for tests/test_ridazen.py; the drivers are tests/stack_util.py."""
import torch

from dlti_b200.models import ridazen as RZ
from tests import ref_ridazen as R
from tests.stack_util import Zoo


def _att(heads, kv_heads, dim, vdim, scale, conv=0, temp=None, bias=None):
    """temp: (coef, every); bias: (rows, far)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {**m, "bias_max": bias[1], "bias_rows": bias[0]} if bias else m


def _moe(experts, top, ff, shared=None):
    e = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return {**e, "shared": {"ff": shared}} if shared else e


def _cfg(vocab, width, eps, mult, scale, cap, side, loop, *layers):
    d = {"architecture": "Ridazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "logit_scale": scale,
         "logit_softcap": cap, "layers": [{"type": "attention", "mixer": m, "mlp": e} for m, e in layers]}
    if side:
        d["token_side"] = {"dim": side}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


CONFIGS = {
    # nothing a multiple of 8: every kernel's general form; the middle of the stack three times
    "odd": _cfg(203, 100, 1e-5, 0.6, 1.3, 9.0, 13, (1, 3, 3), (_att(6, 3, 14, 10, 0.3, 3, (0.4, 17), (12, 70)), _moe(10, 3, 21, 37)),
                (_att(4, 1, 9, 13, 0.25, 5, (0.2, 40), (8, 31)), _moe(7, 2, 30)), (_att(3, 3, 20, 10, 0.2, 2, None, (20, 150)), None),
                (_att(2, 1, 11, 17, 0.3, 0, (0.5, 1)), _moe(6, 4, 19, 11))),
    # the packed prompt kernel, vectorised row kernels, activations in the GEMM's shape; heads of 64 and 128 and smaller ones in a packed row
    "wide": _cfg(320, 256, 1e-6, 0.8, 0.7, 20.0, 24, (0, 2, 2), (_att(8, 2, 64, 64, 0.09, 4, (0.3, 50), (32, 128)), _moe(12, 4, 72, 136)),
                 (_att(4, 2, 128, 128, 0.06, 3, (0.1, 96), (16, 300)), _moe(32, 6, 40, 64)), (_att(6, 3, 40, 72, 0.12, 2, (0.2, 33), (24, 60)), None)),
    # ones: one head, one tap, one expert, two distance buckets, one number per token, one pass
    "ones": _cfg(96, 72, 0.1, 1.0, 1.0, 5.0, 1, (0, 2, 1), (_att(1, 1, 8, 8, 0.5, 1, (1.0, 1), (2, 2)), _moe(1, 1, 8)),
                 (_att(1, 1, 8, 8, 0.4, 2, (0.3, 9), (2, 40)), _moe(2, 1, 16, 8)), (_att(1, 1, 8, 8, 0.5, 0, None, (4, 3)), None)),
    # heads above 128 and above 256, no loop, no token input, no cap
    "tall": _cfg(160, 96, 1e-5, 0.9, 0.5, 0.0, 0, None, (_att(4, 2, 136, 144, 0.05, 4, (0.2, 30), (16, 90)), _moe(5, 2, 48, 72)),
                 (_att(2, 1, 264, 40, 0.03, 2, (0.3, 64), (10, 200)), _moe(9, 5, 24, 40)), (_att(2, 2, 256, 256, 0.03, 3, None, (32, 64)), _moe(4, 1, 8))),
}


def choice_margin(z, top):
    """How far router logits [n, experts] are from another choice: the gap between what is taken and what is left."""
    c = z.sort(-1, descending=True).values
    return c[:, top - 1] - c[:, top] if top < c.shape[1] else torch.full((c.shape[0],), 9.0, dtype=c.dtype)


def _sharpen(d, st):
    g = torch.Generator().manual_seed(11)
    for k in st:
        if k.endswith("q.norm"):                              # sharp attention: a single key decides
            st[k] = (st[k].float() * 2).bfloat16()
        elif k.endswith(".rel"):                              # neighbouring buckets differ
            t = torch.randn(st[k].shape, generator=g) + 1.5 * (-1.0) ** torch.arange(st[k].shape[0])[:, None]
            st[k] = t.bfloat16()
    # Routers read a few coordinates that nothing is added to: up to a common factor they are the token's own. Tokens whose choice
    # would be close in some layer for some factor get another pattern.
    D, V = 16, d["vocab"]
    for k in st:
        if k.endswith(("mix.o", ".down", "side.proj")):
            st[k][:D] = 0
    moe = [(i, l["mlp"]["router"]) for i, l in enumerate(d["layers"]) if l["mlp"]]
    for i, r in moe:
        w = torch.zeros(r["experts"], d["width"])
        w[:, :D] = torch.randn(r["experts"], D, generator=g) * 0.8
        st[f"l{i}.mlp.router"] = w.bfloat16()
        st[f"l{i}.mlp.router.b"] = (torch.randn(r["experts"], generator=g) * 0.2).bfloat16()
    best, signs = torch.full((V,), -1.0, dtype=torch.double), torch.zeros(V, D)
    for _ in range(1500):
        s = torch.randint(0, 2, (V, D), generator=g).double() * 2 - 1
        gap = torch.full((V,), 9.0, dtype=torch.double)
        for i, r in moe:
            z = (s * st[f"l{i}.norm2"][:D].double()) @ st[f"l{i}.mlp.router"][:, :D].double().t()
            for f in (0.5, 0.8, 1.1, 1.4, 1.7, 2.0):
                gap = torch.minimum(gap, choice_margin(f * z + st[f"l{i}.mlp.router.b"].double(), r["top"]))
        better = gap > best
        best = torch.where(better, gap, best)
        signs[better] = s[better].float()
    assert best.min() > 0.03, float(best.min())
    st["embed"][:, :D] = (signs * 2).bfloat16()


class RidazenZoo(Zoo):
    def __init__(self):
        super().__init__(RZ, RZ.RidazenConfig, R, CONFIGS, None)

    def model(self, name, seed=0):
        d = self.configs[name]
        cfg = self.config_cls.from_dict(d, name=name)
        st = self.design.random_state(cfg, seed)
        _sharpen(d, st)
        return d, cfg, st, {k: v.double() for k, v in st.items()}


ZOO = RidazenZoo()
