"""Small Sigosun models and drivers for tests/test_sigosun*.py."""
import copy
import functools
import random

import torch

from dlti_b200.models import sigosun as SG
from dlti_b200.ops import stack as K
from dlti_b200.serve.engine import LLMEngine
from dlti_b200.serve.model_runner import TPContext
from dlti_b200.serve.params import Request, SamplingParams
from dlti_b200.serve.tokenizer import ByteTokenizer
from tests import ref_sigosun as R


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


@functools.lru_cache(None)
def model(name, seed=0):
    """(config dict, config object, checkpoint tensors, the same in double precision)."""
    d = CONFIGS[name]
    cfg = SG.SigosunConfig.from_dict(d, name=name)
    st = SG.random_state(cfg, seed)
    for k in st:
        if k.endswith("q.norm"):                 # sharp attention: a single key decides
            st[k] = (st[k].float() * 3).bfloat16()
    return d, cfg, st, {k: v.double() for k, v in st.items()}


def tokens(name, n, seed):
    g = torch.Generator().manual_seed(1000 * seed + n)
    return torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=g).tolist()


@functools.lru_cache(None)
def oracle(name, n, seed):
    d, _, _, w = model(name)
    return R.forward(d, w, tokens(name, n, seed))


def engine(name, device, dtype, num_blocks=64, max_len=512, **kw):
    _, cfg, st, _ = model(name)
    kw = {"max_num_seqs": 4, "use_cuda_graphs": True, **kw}
    return LLMEngine(cfg, SG.from_state(cfg, st, device, dtype), TPContext(), ByteTokenizer(cfg.vocab_size), num_blocks=num_blocks,
                     max_model_len=max_len, **kw)


class Replay:
    """Feeds requests (n, seed) through replay_step and collects the logits of every position."""

    def __init__(self, name, eng):
        self.name, self.eng, self.live, self.got = name, eng, {}, {}

    def step(self, entries, end=True):
        """entries: {(n, seed): number of next tokens}"""
        ents, order = [], []
        for key, c in entries.items():
            r = self.live.get(key)
            if r is None:
                r = self.live[key] = Request(str(key), [], SamplingParams(temperature=0.0))
                self.got[key] = []
            a = r.num_computed
            ents.append((r, tokens(self.name, *key)[a:a + c], list(range(c))))
            order.append((key, c))
        out, k = self.eng.replay_step(ents), 0
        for key, c in order:
            self.got[key].append(out[k:k + c])
            k += c
            if end and self.live[key].num_computed == key[0]:
                self.eng.replay_end(self.live.pop(key))

    def logits(self, key):
        return torch.cat(self.got[key])


def row_errors(got, want):
    return (got.double() - want).square().mean(1).sqrt() / want.std()


def check(name, rp, tol):
    """Every position within tol; with 16-bit activations a few may be worse, since a norm on a sublayer's small output
    magnifies its rounding."""
    for key in rp.got:
        e = row_errors(rp.logits(key), oracle(name, *key))
        if tol > 0.01:
            assert int((e > tol).sum()) <= 1 + 0.02 * len(e) and e.mean() < tol / 3, (name, key, e.sort().values[-5:])
            tol_max = 4 * tol
        else:
            tol_max = tol
        assert e.max() < tol_max, (name, key, "position", int(e.argmax()), float(e.max()))


def random_portions(n, rng, sizes):
    out = []
    while sum(out) < n:
        out.append(min(n - sum(out), rng.choice(sizes)))
    return out


def mixed_schedule(keys, rng, sizes, tail=6, live=4):
    """Steps {key: count}: up to `live` requests at a time, portions of some beside single tokens of others."""
    todo = {k: random_portions(max(1, k[0] - tail), rng, sizes) + [1] * min(tail, k[0] - 1) for k in keys}
    waiting, running, steps = list(keys), [], []
    while waiting or running:
        while waiting and len(running) < live:
            running.append(waiting.pop(0))
        st = {k: todo[k].pop(0) for k in running if rng.random() < 0.8}
        if st:
            steps.append(st)
        running = [k for k in running if todo[k]]
    return steps


def rows_for(lens, nd, bs, device, seed=0):
    """ops.stack.Rows of sequences lens = [(start, n)] (the first nd decode) over shuffled pages; also the page count."""
    g = torch.Generator().manual_seed(seed)
    need = [-(-(s + n) // bs) for s, n in lens]
    perm = torch.randperm(sum(need) + 3, generator=g)
    tabs = torch.zeros(len(lens), max(need) + 1, dtype=torch.int32)
    o = 0
    for i, k in enumerate(need):
        tabs[i, :k] = perm[o:o + k]
        o += k
    pos = torch.cat([torch.arange(s, s + n) for s, n in lens])
    seq = torch.cat([torch.full((n,), i) for i, (_, n) in enumerate(lens)])
    cu = [0]
    for _, n in lens[nd:]:
        cu.append(cu[-1] + n)
    slots = torch.tensor([int(tabs[i, p // bs]) * bs + p % bs for i, p in zip(seq.tolist(), pos.tolist())])
    ctx = torch.tensor([s + n for s, n in lens], dtype=torch.int32)
    d = lambda t: t.to(device)
    r = K.Rows(d(pos.int()), d(seq.int()), d(slots), d(ctx), d(torch.tensor(cu, dtype=torch.int32)) if len(cu) > 1 else None, d(tabs),
               d(torch.randperm(len(lens), generator=g).int()), nd, max([n for _, n in lens[nd:]], default=0), int(ctx.max()))
    return r, sum(need) + 3


def mutated(name, **edits):
    """A copy of the config dict with mixer entries of one layer replaced: planted mistakes for the oracle."""
    d = copy.deepcopy(CONFIGS[name])
    layer = edits.pop("layer")
    d["layers"][layer]["mixer"].update(edits)
    return d


__all__ = ["CONFIGS", "K", "R", "Replay", "SG", "check", "engine", "mixed_schedule", "model", "mutated", "oracle", "random", "random_portions",
           "row_errors", "rows_for", "tokens"]
