"""Small Logozen models for tests/test_logozen.py; the drivers are tests/stack_util.py."""
import torch

from dlti_b200.models import logozen as LZ
from tests import ref_logozen as R
from tests.stack_util import Zoo


def _att(heads, dim, rot_dim, vdim, rank, scale, rot=None, base=1e4):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
            "rot": {"base": base, "dims": rot_dim if rot is None else rot}}


def _mem(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def _layer(mixer, ff=None):
    return {"type": "latent_attention" if "kv_rank" in mixer else "mlstm", "mixer": mixer, "mlp": None if ff is None else {"ff": ff, "kind": "dense"}}


def _cfg(vocab, width, streams, taps, scale, eps, *layers):
    return {"architecture": "Logozen", "vocab": vocab, "width": width, "streams": streams, "canon": {"taps": taps}, "embedding": {"scale": scale},
            "norm": {"eps": eps}, "layers": list(layers)}


CONFIGS = {
    # nothing a multiple of 8: every kernel's general form; part of the shared key part unrotated
    "odd": _cfg(203, 100, 5, 5, 1.7, 1e-5, _layer(_att(3, 14, 10, 18, 44, 0.3, rot=6), 90), _layer(_mem(3, 18, 10, 6.0), 61),
                _layer(_att(2, 9, 4, 7, 21, 0.4)), _layer(_mem(2, 7, 35, 15.0))),
    # the packed prompt kernel, chunked scans, vectorised row kernels; layers without a feed-forward
    "wide": _cfg(320, 256, 4, 4, 2.5, 1e-6, _layer(_mem(2, 72, 40, 9.0)), _layer(_att(6, 64, 64, 128, 256, 0.09, base=5e5), 264),
                 _layer(_att(3, 40, 24, 72, 136, 0.12, base=5e5)), _layer(_mem(3, 136, 48, 12.0), 200)),
    # ones: one stream, one tap, one head
    "ones": _cfg(96, 72, 1, 1, 1.0, 1e-5, _layer(_att(1, 8, 8, 8, 8, 0.5), 41), _layer(_mem(1, 8, 8, 4.0), 8)),
    # heads above 128 (expanded into pages of one row), more heads than one block of the absorbed kernel takes, a large latent
    "tall": _cfg(160, 96, 2, 2, 3.0, 1e-5, _layer(_att(20, 96, 48, 136, 320, 0.09), 72), _layer(_att(35, 16, 16, 24, 40, 0.2), 40), _layer(_mem(1, 256, 64, 10.0)),
                 _layer(_att(2, 200, 64, 24, 96, 0.07))),
}


def _sharpen(st):
    g = torch.Generator().manual_seed(11)
    for k in st:
        if k.endswith("mix.q") and k[:-1] + "dkv" in st:      # sharp attention: a single key decides
            st[k] = (st[k].float() * 2).bfloat16()
        elif k.endswith("sink"):                              # sinks that weigh as much as the keys
            st[k] = (st[k].float() + 4).bfloat16()
        elif k.endswith("mix.f.b"):                           # long and short memories
            st[k] = torch.linspace(-2, 8, st[k].numel()).bfloat16()
        elif k.endswith("mix.i.b"):                           # quiet heads stay below the running maximum's start, loud ones above
            st[k] = torch.linspace(-3, 4, st[k].numel()).bfloat16()
        elif ".hc" in k:
            st[k] = (st[k].float() + 0.2 * torch.randn(st[k].shape, generator=g)).bfloat16()


ZOO = Zoo(LZ, LZ.LogozenConfig, R, CONFIGS, _sharpen)
