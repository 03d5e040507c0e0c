"""The Vugipel decoder under the scheduler: greedy generation against the plain statement, prompts and decode rows in one forward,
sampling, speculation with rollback of the recurrent state, prefix snapshots, the launcher."""
import pytest
import torch

import vugipel_plain as plain
from listed_util import generator, run_all, write_tokenizer
from vugipel_util import CONFIGS, DEVICES, Weights, engine, make, off, one_thread, reference, tokens, write_model  # noqa: F401
from volta_engine_b200.runtime.generator import Request
from volta_engine_b200.runtime.prefix_cache import PrefixCache
from volta_engine_b200.runtime.sampling import SamplingParams

NAME = "eights"
VOCAB = CONFIGS[NAME]["vocab"]


def greedy(prompt, n):
    """Plain greedy continuation (the whole sequence again for every token)."""
    w = Weights(NAME, 3).t
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(plain.forward(CONFIGS[NAME], w, seq)[0][-1].argmax()))
    return seq[len(prompt):]


def prompts():
    return [tokens(n, VOCAB, 40 + n) for n in (70, 3, 130, 17, 64, 1)]


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation_matches_the_plain_statement(device):
    _, _, model = make(NAME, device, "fp32")
    for q in (prompts()[0][:30], prompts()[1]):
        r = generator(model).generate(Request(list(q), max_tokens=8))
        assert r["tokens"] == greedy(q, 8) and r["reason"] == "length"


@pytest.mark.parametrize("device", DEVICES)
def test_concurrent_requests_equal_each_alone(device):
    """Six requests over three slots: prompt portions run beside decode rows, slots and pages come round again."""
    _, _, model = make(NAME, device, "fp32")
    ps = prompts() if device == "cuda" else [p[:40] for p in prompts()]
    alone = [run_all(generator(model), [Request(list(p), max_tokens=10)])[0] for p in ps]
    gen = generator(model, pages=1 + 3 * 3)
    calls = []
    step = gen.engine.step_mixed
    gen.engine.step_mixed = lambda segs, **k: (calls.append([len(s[1]) for s in segs]), step(segs, **k))[1]
    assert run_all(gen, [Request(list(p), max_tokens=10) for p in ps]) == alone
    assert any(max(c) > 1 and min(c) == 1 and len(c) > 1 for c in calls)      # a portion and a decode row in one forward
    assert gen.engine.kv.free_pages() == gen.engine.kv.num_pages - 1


@pytest.mark.parametrize("device", DEVICES)
def test_sampled_requests_do_not_run_a_prompt_row_twice(device):
    """The same seed gives the same text alone and beside others, and top-k 1 equals greedy."""
    _, _, model = make(NAME, device, "fp32")
    ps = [p[:25] for p in prompts()[:3]]
    par = lambda i: SamplingParams(temperature=0.9, top_p=0.95, seed=100 + i)
    alone = [run_all(generator(model), [Request(list(p), max_tokens=8, params=par(i))])[0] for i, p in enumerate(ps)]
    assert run_all(generator(model), [Request(list(p), max_tokens=8, params=par(i)) for i, p in enumerate(ps)]) == alone
    g = run_all(generator(model), [Request(list(ps[0]), max_tokens=8)])[0]
    assert run_all(generator(model), [Request(list(ps[0]), max_tokens=8, params=SamplingParams(temperature=0.7, top_k=1, seed=5))])[0] == g


@pytest.mark.parametrize("device", DEVICES)
def test_speculative_blocks_roll_the_state_back(device):
    _, _, model = make(NAME, device, "fp32")
    p = (tokens(8, VOCAB, 3) * 8)[:60]
    want = run_all(generator(model), [Request(list(p), max_tokens=24)])[0]
    gen = generator(model, speculator="suffix", spec_ctrl=False, spec_depth=4)
    assert run_all(gen, [Request(list(p), max_tokens=24)])[0] == want
    assert gen.metrics.spec["rounds"] > 0


@pytest.mark.parametrize("device", DEVICES)
def test_rejected_rows_leave_no_trace(device):
    _, _, model = make(NAME, device, "fp32")
    t = tokens(60, VOCAB, 12)
    ref = engine(model)
    ref.forward_segments([(1, t[:40], 0, [])])
    ref.forward_segments([(1, t[40:42], 40, [])])
    want = [s.rec[1].clone() for s in model.layer_states()]
    assert len(want) == len(model.layers)
    eng = engine(model)
    for _ in range(5 if device == "cuda" else 2):                 # eager, captured, replayed
        eng.forward_segments([(1, t[:40], 0, [])])
        eng.step(t[40:45], list(range(40, 45)), [1] * 5, journal=True)
        eng.rollback(1, 2)
        got = [s.rec[1].clone() for s in model.layer_states()]
        assert all((a - b).abs().max() <= 1e-5 * b.abs().max() for a, b in zip(got, want))
        eng.kv.release(1)


@pytest.mark.parametrize("device", DEVICES)
def test_short_prompt_behind_a_verify_block(device):
    """Its rows are not recorded as a block: positions and slot are its own."""
    _, _, model = make(NAME, device, "fp32")
    t = tokens(60, VOCAB, 12)
    eng = engine(model)
    eng.forward_segments([(1, t[:40], 0, [])])
    eng.step(t[40:45], list(range(40, 45)), [1] * 5, journal=True)
    eng.prefill_rows(2, t[:10], 0, True)
    assert off(eng.row_logits[-1:], reference(NAME, t[:10])[9:]) < 1e-4
    eng.step(t[45:50], list(range(45, 50)), [1] * 5, journal=True)
    eng.prefill(3, t[:7])
    assert off(eng.forward_segments([(3, t[7:9], 7, [1])]), reference(NAME, t[:9])[8:]) < 1e-4


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("where", ["memory", "disk"])
def test_prefix_snapshots_carry_cache_and_state(where, device, tmp_path):
    _, _, model = make(NAME, device, "fp32")
    t = tokens(150, VOCAB, 33)
    want = run_all(generator(model), [Request(list(t), max_tokens=6)])[0]
    cache = PrefixCache(64 << 20, str(tmp_path) if where == "disk" else None)
    assert run_all(generator(model, cache=cache), [Request(list(t[:140]), max_tokens=4)])
    gen = generator(model, cache=cache)
    got, usage = [], {}
    r = Request(list(t), max_tokens=6)
    r.on_text, r.on_finish = (lambda x, ids, lp: got.extend(ids)), (lambda reason, u: usage.update(u))
    gen.submit(r)
    while not usage:
        gen.step()
    assert got == want and usage["cached_tokens"] >= 128


def test_server_on_a_model_directory(tmp_path):
    from volta_engine_b200.server import cli
    write_model(tmp_path, NAME)
    write_tokenizer(tmp_path, VOCAB)
    cfg, _ = cli.resolve_config(["--model-dir", str(tmp_path), "--port", "0", "--set", "max_slots=2", "--set", "max_seq=512", "--set", "kv_pool=1024", "--set", "dtype=fp32"], env={})
    srv, gen, eng = cli.build_server(cfg, "cpu")
    assert type(eng.model).__name__ == "VugipelModel" and eng.kv.k.dtype == torch.float32 and gen.mixed
    p = gen.tok.encode("a prompt")
    assert gen.generate(Request(list(p), max_tokens=6, ignore_eos=True))["tokens"] == greedy(p, 6)
    srv.http.stop()
