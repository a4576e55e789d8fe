"""Small layer-stack models of one design (config dicts, the design's module, its oracle) and drivers that run them through the
engine, for tests/test_sigosun.py and tests/test_logozen.py."""
import copy
import functools

import torch

from dlti_b200.ops import stack as K
from dlti_b200.serve.engine import LLMEngine, _pieces, chunk_pieces
from dlti_b200.serve.model_runner import TPContext
from dlti_b200.serve.params import Request, SamplingParams
from dlti_b200.serve.tokenizer import ByteTokenizer


class Zoo:
    """design: module with random_state and from_state; ref: module with forward(config dict, weights, tokens). sharpen changes
    random weights in place so that single keys decide."""

    def __init__(self, design, config_cls, ref, configs, sharpen):
        self.design, self.config_cls, self.ref, self.configs, self.sharpen = design, config_cls, ref, configs, sharpen
        self.model = functools.lru_cache(None)(self.model)
        self.oracle = functools.lru_cache(None)(self.oracle)

    def model(self, name, seed=0):
        """(config dict, config object, checkpoint tensors, the same in double precision)."""
        d = self.configs[name]
        cfg = self.config_cls.from_dict(d, name=name)
        st = self.design.random_state(cfg, seed)
        self.sharpen(st)
        return d, cfg, st, {k: v.double() for k, v in st.items()}

    def tokens(self, name, n, seed):
        g = torch.Generator().manual_seed(1000 * seed + n)
        return torch.randint(0, self.configs[name]["vocab"], (n,), generator=g).tolist()

    def oracle(self, name, n, seed):
        d, _, _, w = self.model(name)
        return self.ref.forward(d, w, self.tokens(name, n, seed))

    def engine(self, name, device, dtype, num_blocks=64, max_len=512, **kw):
        _, cfg, st, _ = self.model(name)
        kw = {"max_num_seqs": 4, "use_cuda_graphs": True, **kw}
        return LLMEngine(cfg, self.design.from_state(cfg, st, device, dtype), TPContext(), ByteTokenizer(cfg.vocab_size),
                         num_blocks=num_blocks, max_model_len=max_len, **kw)

    def replay(self, name, eng):
        return Replay(self, name, eng)

    def check(self, name, rp, tol):
        """Every position within tol; with 16-bit activations a few may be worse, since a norm on a sublayer's small output
        magnifies its rounding."""
        for key in rp.got:
            e = row_errors(rp.logits(key), self.oracle(name, *key))
            if tol > 0.01:
                assert int((e > tol).sum()) <= 1 + 0.02 * len(e) and e.mean() < tol / 3, (name, key, e.sort().values[-5:])
                tol_max = 4 * tol
            else:
                tol_max = tol
            assert e.max() < tol_max, (name, key, "position", int(e.argmax()), float(e.max()))

    def mutated(self, name, **edits):
        """A copy of the config dict with mixer entries of one layer replaced: planted mistakes for the oracle."""
        d = copy.deepcopy(self.configs[name])
        layer = edits.pop("layer")
        d["layers"][layer]["mixer"].update(edits)
        return d

    def greedy(self, name, prompt, n):
        d, _, _, w = self.model(name)
        seq = list(prompt)
        for _ in range(n):
            seq.append(int(self.ref.forward(d, w, seq)[-1].argmax()))
        return seq[len(prompt):]

    def check_generation(self, name, device, lens=(5, 33, 1, 60, 18, 2), n=9, **kw):
        """Greedy generation of more requests than slots through the scheduler, beside the oracle's own."""
        prompts = [self.tokens(name, k, 20 + k) for k in lens]
        eng = self.engine(name, device, torch.float32, max_num_seqs=3, **kw)
        outs = eng.generate(prompts, SamplingParams(max_tokens=n, temperature=0.0, ignore_eos=True))
        for p, o in zip(prompts, outs):
            assert o["token_ids"] == self.greedy(name, p, n)
        assert eng.blocks.num_free == eng.blocks.num_blocks and (eng.slots is None or len(eng.slots.free) == 3)
        return eng


class Replay:
    """Feeds requests (n, seed) through replay_step and collects the logits of every position."""

    def __init__(self, zoo, name, eng):
        self.zoo, self.name, self.eng, self.live, self.got = zoo, name, eng, {}, {}

    def step(self, entries, end=True):
        """entries: {(n, seed): number of next tokens}"""
        ents, order = [], []
        for key, c in entries.items():
            r = self.live.get(key)
            if r is None:
                r = self.live[key] = Request(str(key), [], SamplingParams(temperature=0.0))
                self.got[key] = []
            a = r.num_computed
            ents.append((r, self.zoo.tokens(self.name, *key)[a:a + c], list(range(c))))
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


def pieces_for(rows, nd, device, bs=16):
    """ops.stack.Pieces of all prompt rows of `rows` for unlimited attention, however short they are."""
    from dlti_b200.serve import engine as E
    cu, ctx = rows.cu.tolist(), rows.ctx.tolist()[nd:]
    starts = [c - (cu[i + 1] - cu[i]) for i, c in enumerate(ctx)]
    keep, E.PACK_FROM = E.PACK_FROM, 1
    try:
        arr, n, longest, ext, prefix = chunk_pieces(cu, starts, rows.tables.tolist()[nd:], bs, 0, 1 << 30)
    finally:
        E.PACK_FROM = keep
    return _pieces(torch.from_numpy(arr).to(device), cu[-1], n, longest, ext, prefix)
