"""The Fofosun decoder under the scheduler: greedy generation against the plain statement, prompts and decode rows in one forward,
sampling, speculation with rollback of the recurrent state, prefix snapshots, the launcher."""
import pytest
import torch

import fofosun_plain as plain
from fofosun_util import CONFIGS, DEVICES, Weights, engine, make, one_thread, tokens, write_model  # noqa: F401
from listed_util import generator, run_all, write_tokenizer
from volta_engine_b200.runtime.generator import Request
from volta_engine_b200.runtime.prefix_cache import PrefixCache
from volta_engine_b200.runtime.sampling import SamplingParams

NAME = "eights"


def greedy(prompt, n):
    """Plain greedy continuation (the whole sequence again for every token)."""
    cfg, w = CONFIGS[NAME], Weights(CONFIGS[NAME], 3).t
    seq = list(prompt)
    for _ in range(n):
        seq.append(int(plain.forward(cfg, w, seq)[0][-1].argmax()))
    return seq[len(prompt):]


def prompts():
    return [tokens(n, CONFIGS[NAME]["vocab"], 40 + n) for n in (70, 3, 130, 17, 64, 1)]


@pytest.mark.parametrize("device", DEVICES)
def test_greedy_generation_matches_the_plain_statement(device):
    _, _, model = make(NAME, device, "fp32")
    p = prompts()
    for q in (p[0][:30], p[1]):
        gen = generator(model)
        r = gen.generate(Request(list(q), max_tokens=8))
        assert r["tokens"] == greedy(q, 8) and r["reason"] == "length"


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", ["fp32"])
def test_concurrent_requests_equal_each_alone(dtype, device):
    """Six requests over three slots: prompt portions run beside decode rows, slots and pages come round again."""
    _, _, model = make(NAME, device, dtype)
    alone = [run_all(generator(model), [Request(list(p), max_tokens=12)])[0] for p in prompts()]
    gen = generator(model, pages=1 + 3 * 3)
    calls = []
    step = gen.engine.step_mixed
    gen.engine.step_mixed = lambda segs, **k: (calls.append([len(s[1]) for s in segs]), step(segs, **k))[1]
    both = run_all(gen, [Request(list(p), max_tokens=12) for p in prompts()])
    assert both == alone
    assert any(max(c) > 1 and min(c) == 1 and len(c) > 1 for c in calls)      # a portion and a decode row in one forward
    assert gen.engine.kv.free_pages() == gen.engine.kv.num_pages - 1


@pytest.mark.parametrize("device", DEVICES)
def test_sampled_requests_do_not_run_a_prompt_row_twice(device):
    """A sampled first token must come from the state the prompt left: the same seed gives the same text alone and beside others,
    and top-k 1 equals greedy."""
    _, _, model = make(NAME, device, "fp32")
    ps = prompts()[:3]
    par = lambda i: SamplingParams(temperature=0.9, top_p=0.95, seed=100 + i)
    alone = [run_all(generator(model), [Request(list(p), max_tokens=10, params=par(i))])[0] for i, p in enumerate(ps)]
    assert run_all(generator(model), [Request(list(p), max_tokens=10, params=par(i)) for i, p in enumerate(ps)]) == alone
    g = run_all(generator(model), [Request(list(ps[0]), max_tokens=10)])[0]
    assert run_all(generator(model), [Request(list(ps[0]), max_tokens=10, params=SamplingParams(temperature=0.7, top_k=1, seed=5))])[0] == g


@pytest.mark.parametrize("device", DEVICES)
def test_speculative_blocks_roll_the_state_back(device):
    _, _, model = make(NAME, device, "fp32")
    p = (tokens(20, CONFIGS[NAME]["vocab"], 3) * 5)[:90]
    want = run_all(generator(model), [Request(list(p), max_tokens=24)])[0]
    gen = generator(model, speculator="suffix", spec_ctrl=False, spec_depth=4)
    assert run_all(gen, [Request(list(p), max_tokens=24)])[0] == want
    assert gen.metrics.spec["rounds"] > 0


@pytest.mark.parametrize("device", DEVICES)
def test_rejected_rows_leave_no_trace(device):
    _, _, model = make(NAME, device, "fp32")
    t = tokens(60, CONFIGS[NAME]["vocab"], 12)
    eng = engine(model)
    eng.forward_segments([(1, t[:40], 0, [])])
    want = None
    for _ in range(5):                            # eager, captured, replayed
        eng.step(t[40:45], list(range(40, 45)), [1] * 5, journal=True)
        eng.rollback(1, 2)
        got = [s.rec[1].clone() for s in model.layer_states() if s is not None]
        if want is None:
            ref = engine(model)
            ref.forward_segments([(1, t[:40], 0, [])])
            ref.forward_segments([(1, t[40:42], 40, [])])
            want = [s.rec[1].clone() for s in model.layer_states() if s is not None]
            eng = engine(model)
        else:
            assert all((a - b).abs().max() <= 1e-5 * b.abs().max() for a, b in zip(got, want))
        eng.kv.release(1)
        eng.forward_segments([(1, t[:40], 0, [])])


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("where", ["memory", "disk"])
def test_prefix_snapshots_carry_the_state(where, device, tmp_path):
    _, _, model = make(NAME, device, "fp32")
    t = tokens(150, CONFIGS[NAME]["vocab"], 33)
    want = run_all(generator(model), [Request(list(t), max_tokens=8)])[0]
    cache = PrefixCache(64 << 20, str(tmp_path) if where == "disk" else None)
    first = generator(model, cache=cache)
    assert run_all(first, [Request(list(t[:140]), max_tokens=4)])
    gen = generator(model, cache=cache)
    got = []
    r = Request(list(t), max_tokens=8)
    usage = {}
    r.on_text, r.on_finish = (lambda x, ids, lp: got.extend(ids)), (lambda reason, u: usage.update(u))
    gen.submit(r)
    while not usage:
        gen.step()
    assert got == want and usage["cached_tokens"] >= 128


def test_cancelled_requests_in_a_mixed_step():
    _, _, model = make(NAME, "cpu", "fp32")
    gen = generator(model)
    done = {}
    ids = []
    for i, p in enumerate(prompts()[:3]):
        r = Request(list(p), max_tokens=20, on_finish=lambda reason, u, i=i: done.__setitem__(i, reason))
        ids.append(gen.submit(r))
    gen.step()
    gen.cancel(ids[2])
    for _ in range(200):
        gen.step()
        if len(done) == 3:
            break
    assert done == {0: "length", 1: "length", 2: "cancelled"}


def test_server_on_a_model_directory(tmp_path):
    from volta_engine_b200.server import cli
    write_model(tmp_path, NAME)
    write_tokenizer(tmp_path, CONFIGS[NAME]["vocab"])
    cfg, _ = cli.resolve_config(["--model-dir", str(tmp_path), "--port", "0", "--set", "max_slots=2", "--set", "max_seq=512", "--set", "kv_pool=1024", "--set", "dtype=fp32"], env={})
    srv, gen, eng = cli.build_server(cfg, "cpu")
    assert type(eng.model).__name__ == "FofosunModel" and eng.kv.k.dtype == torch.float32 and gen.mixed
    p = gen.tok.encode("a prompt")
    assert gen.generate(Request(list(p), max_tokens=6, ignore_eos=True))["tokens"] == greedy(p, 6)
    srv.http.stop()
