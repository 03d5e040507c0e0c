"""What the tests of decoders with listed layers share: engines, portions, schedules of several requests, rows through one operator, the
scheduler."""
import dataclasses
import json

import pytest
import torch

from volta_engine_b200.runtime.batch import BatchRows
from volta_engine_b200.runtime.engine import Engine
from volta_engine_b200.runtime.generator import Generator
from volta_engine_b200.runtime.kv_cache import PagedKVCache
from volta_engine_b200.runtime.options import Options

DEVICES = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
DTYPES = ["fp32", "bf16"]
TOL = {"fp32": 1e-4, "bf16": 0.04}        # root mean square of the difference over that of the logits


@pytest.fixture(autouse=True)
def one_thread():
    """The models are so small that a pool of threads only gets in its own way."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def engine(model, pages=24, slots=4, max_seq=1024, **kw):
    model.reset_states()
    kv = PagedKVCache(model.kv_layers, 1, model.cfg.head_dim, pages, slots, max_seq, model.device, dtype=model.dtype, v_head_dim=model.kv_v_dim)
    return Engine(model, kv, use_graphs=kw.pop("use_graphs", model.device.type == "cuda"), **kw)


def off(got, want):
    """Per row: root mean square of the difference over the root mean square of the wanted logits."""
    g, w = got.double().cpu(), want.double()
    return ((g - w).pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt().mean()).max().item()


def run(eng, slot, toks, cuts, p0=0):
    """Tokens of one sequence in portions of the given sizes -> logits of all of them."""
    out, at = [], 0
    for c in cuts:
        part = toks[at:at + c]
        out.append(eng.forward_segments([(slot, part, p0 + at, list(range(len(part))))]).float().clone())
        at += c
    assert at == len(toks)
    return torch.cat(out)


CUTS = {"one by one": [1] * 150, "twos": [2] * 75, "prompt then decode": [110] + [1] * 40, "around pages": [63, 1, 1, 63, 2, 20],
        "short and long": [3, 17, 2, 64, 15, 16, 33], "halves": [75, 75]}


def schedule(lengths, seed):
    """Random steps over several requests: portions of some beside single tokens of others; at most four live at once."""
    g = torch.Generator().manual_seed(seed)
    left, live, steps = list(range(len(lengths))), [], []
    done = [0] * len(lengths)
    while left or live:
        while left and len(live) < 4:
            live.append(left.pop(0))
        step, ended = [], []
        for r in list(live):
            if len(live) > 1 and torch.rand((), generator=g) < 0.2:
                continue                         # left out of this step
            rest = lengths[r] - done[r]
            n = [1, 1, 2, 3, 16, 29, 64, 90][int(torch.randint(0, 8, (), generator=g))] if rest > 12 else 1
            n = min(n, rest)
            step.append((r, done[r], n))
            done[r] += n
            if done[r] == lengths[r]:
                ended.append(r)
        live = [r for r in live if r not in ended]
        if step:
            steps.append((step, ended))
    return steps


# ------------------------------------------------------------------------------------------ one operator
class Rows:
    """A paged cache (its rows wider than this layer's, filled with an earlier request's rows) and batches through an operator."""

    def __init__(self, dtype, device, kw, vw, extra=0, pages=24):
        self.dtype, self.device = dtype, device
        self.kv = PagedKVCache(2, 1, kw + extra, pages, 3, 1024, torch.device(device), dtype=dtype, v_head_dim=vw + extra)
        self.kv.k.fill_(3.0)
        self.kv.v.fill_(-3.0)

    def batch(self, parts):
        """parts: [(slot, first position, rows)] one batch, shortest first."""
        pos, slots = [], []
        for s, p0, x in parts:
            self.kv.reserve(s, p0 + x.shape[0])
            pos += range(p0, p0 + x.shape[0])
            slots += [s] * x.shape[0]
        b = BatchRows.make(pos, pos, slots, self.device)
        return self.run(b, torch.cat([p[2] for p in parts]))

    def walk(self, slot, x, cuts):
        at, got = 0, []
        for c in cuts:
            got.append(self.batch([(slot, at, x[at:at + c])]))
            at += c
        return torch.cat(got)


def vars_of(spec):
    return {f.name: getattr(spec, f.name) for f in dataclasses.fields(spec)}


# ------------------------------------------------------------------------------------------ scheduler
class Tok:
    eos_ids: list = []

    def decode_bytes(self, ids, skip_special=False):
        return bytes(i & 0x7F for i in ids)


def generator(model, slots=3, pages=24, chunk=48, cache=None, **opt):
    eng = engine(model, pages=pages, slots=slots, max_seq=512, prefill_chunk=chunk)
    o = Options.resolve(dict({"max_slots": slots, "prefix_interval": 64, "loop_detect": False}, **opt), env={})
    return Generator(eng, Tok(), o, prefix_cache=cache, eos_ids=[])


def run_all(gen, reqs):
    """Submit everything, step until all are done -> token lists in order."""
    out = [[] for _ in reqs]
    left = [len(reqs)]
    for i, r in enumerate(reqs):
        r.on_text = lambda t, ids, lp, i=i: out[i].extend(ids)
        r.on_finish = lambda reason, usage: left.__setitem__(0, left[0] - 1)
        gen.submit(r)
    for _ in range(2000):
        if not left[0]:
            break
        gen.step()
    assert not left[0]
    return out


def write_tokenizer(d, vocab):
    """A byte-level vocabulary of 256 pieces and no merges, enough for the launcher."""
    alphabet = [chr(b) if 33 <= b < 127 or 161 <= b < 173 or 174 <= b < 256 else None for b in range(256)]
    n = 0
    for b in range(256):
        if alphabet[b] is None:
            alphabet[b] = chr(256 + n)
            n += 1
    (d / "tokenizer.json").write_text(json.dumps({"model": {"type": "BPE", "vocab": {c: i for i, c in enumerate(alphabet)}, "merges": []},
                                                  "added_tokens": [], "pre_tokenizer": {"type": "ByteLevel"}}))
