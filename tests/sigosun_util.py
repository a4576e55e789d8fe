"""Small Sigosun models for tests/test_sigosun.py; the drivers are tests/stack_util.py."""
import random

from dlti_b200.models import sigosun as SG
from dlti_b200.ops import stack as K
from tests import ref_sigosun as R
from tests.stack_util import Zoo, mixed_schedule, random_portions, row_errors, rows_for


def _att(heads, kv, dim, vdim, rot, chunk, scale, base=1e4, **kw):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "rot": {"base": base, "dims": rot},
            "scale": scale, **kw}


def _layer(kind, mixer, ff=None):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"ff": ff, "kind": "dense"}}


CONFIGS = {
    # nothing a multiple of 8: every kernel's general form
    "odd": {"architecture": "Sigosun", "vocab": 203, "width": 100, "norm": {"eps": 1e-5}, "layers": [
        _layer("attention", _att(6, 2, 22, 18, 10, 37, 0.35), 90),
        _layer("mamba2", {"heads": 4, "vdim": 12, "state": 20, "groups": 2, "conv": 3, "norm_groups": 3}, 61),
        _layer("attention", _att(4, 2, 22, 18, 10, 50, 0.3, kv_from=0)),
        _layer("lightning", {"heads": 3, "dim": 18, "vdim": 10, "decay": [0.4, 0.93, 0.998]}, 44)]},
    # the packed prefill kernel, chunked scans, vectorised row kernels; a recurrent layer first, shared keys over two layers
    "wide": {"architecture": "Sigosun", "vocab": 320, "width": 256, "norm": {"eps": 1e-6}, "layers": [
        _layer("lightning", {"heads": 2, "dim": 72, "vdim": 40, "decay": [0.7, 0.99]}),
        _layer("attention", _att(6, 3, 128, 128, 128, 112, 0.1, base=5e5), 264),
        _layer("attention", _att(3, 3, 128, 128, 128, 150, 0.12, base=5e5, kv_from=1), 200),
        _layer("mamba2", {"heads": 6, "vdim": 32, "state": 72, "groups": 3, "conv": 4, "norm_groups": 2}),
        _layer("attention", _att(9, 3, 128, 128, 128, 80, 0.11, base=5e5, kv_from=1))]},
    # ones: one head, one group, two taps; keys and values of different sizes in the padded packed layout
    "ones": {"architecture": "Sigosun", "vocab": 96, "width": 72, "norm": {"eps": 1e-5}, "layers": [
        _layer("mamba2", {"heads": 1, "vdim": 40, "state": 16, "groups": 1, "conv": 2, "norm_groups": 5}, 56),
        _layer("attention", _att(1, 1, 64, 72, 40, 70, 0.3), 41),
        _layer("lightning", {"heads": 1, "dim": 8, "vdim": 8, "decay": [0.97]}, 8),
        _layer("mamba2", {"heads": 3, "vdim": 8, "state": 24, "groups": 3, "conv": 1, "norm_groups": 1})]},
    # heads above 128 (no packed layout) and many query heads on one key head
    "tall": {"architecture": "Sigosun", "vocab": 160, "width": 96, "norm": {"eps": 1e-5}, "layers": [
        _layer("attention", _att(20, 1, 136, 24, 64, 45, 0.12), 72),
        _layer("attention", _att(2, 2, 200, 256, 200, 96, 0.1), 40)]},
}


def _sharpen(st):
    for k in st:
        if k.endswith("q.norm"):                 # sharp attention: a single key decides
            st[k] = (st[k].float() * 3).bfloat16()


ZOO = Zoo(SG, SG.SigosunConfig, R, CONFIGS, _sharpen)
model, tokens, oracle, engine, check, mutated, Replay = (ZOO.model, ZOO.tokens, ZOO.oracle, ZOO.engine, ZOO.check, ZOO.mutated, ZOO.replay)

__all__ = ["CONFIGS", "K", "R", "Replay", "SG", "ZOO", "check", "engine", "mixed_schedule", "model", "mutated", "oracle", "random", "random_portions",
           "row_errors", "rows_for", "tokens"]
