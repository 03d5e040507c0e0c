"""The Fofosun decoder against its plain statement: whole prompts, portions, token-by-token decoding, mixed batches, slots and
pages that are used again, long decoding; in fp32 and bf16, on the CPU statements and on the GPU kernels."""
import io
import json

import pytest
import torch

from fofosun_util import CONFIGS, DEVICES, DTYPES, TOL, engine, make, off, one_thread, reference, tokens, write_model  # noqa: F401
from listed_util import CUTS, run, schedule

NAMES = list(CONFIGS)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompt(name, dtype, device):
    cfg, _, model = make(name, device, dtype)
    toks = tokens(150, cfg["vocab"])
    got = run(engine(model), 2, toks, [150])
    assert got.shape == (150, cfg["vocab"]) and off(got, reference(name, toks)) < TOL[dtype]


@pytest.mark.parametrize("device", DEVICES)
def test_residual_after_every_layer(device):
    import fofosun_plain as plain
    cfg, w, model = make("eights", device, "fp32")
    toks = tokens(40, cfg["vocab"], 5)
    _, want = plain.forward(cfg, w, toks)
    for cuts in ([40], [1] * 40):
        model.layer_tap = tap = []
        try:
            run(engine(model, use_graphs=False), 0, toks, cuts)
        finally:
            model.layer_tap = None
        n = len(cfg["layers"])
        got = torch.cat([torch.stack(tap[i:i + n]) for i in range(0, len(tap), n)], 1).double().cpu()
        assert (got - want).abs().max() < 2e-4 * want.abs().max()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["eights", "odd", "wide"])
def test_portions_and_decoding(name, dtype, device):
    cfg, _, model = make(name, device, dtype)
    toks = tokens(150, cfg["vocab"])
    want = reference(name, toks)
    eng = engine(model)
    for i, (what, cuts) in enumerate(CUTS.items()):
        if device == "cpu" and dtype == "bf16" and i % 2:
            continue
        slot = i % 4
        assert off(run(eng, slot, toks, cuts), want) < TOL[dtype], what
        eng.kv.release(slot)                     # the next way of cutting gets used pages and a used state slot
    assert eng.kv.free_pages() == eng.kv.num_pages - 1


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["eights", "odd", "recurrent"])
def test_mixed_batches_equal_each_alone(name, dtype, device):
    cfg, _, model = make(name, device, dtype)
    lengths = [150, 1, 23, 97, 64, 65, 130, 2]
    seqs = [tokens(150, cfg["vocab"])[:n] if n != 97 else tokens(97, cfg["vocab"], 9) for n in lengths]
    full = reference(name, seqs[0])
    want = [full[:n] if n != 97 else reference(name, seqs[3]) for n in lengths]
    pages = 1 + 3 * 3 + 2                        # what four live requests need at most: pages come round again
    eng = engine(model, pages=pages if model.kv_layers else 12)
    slots, free = {}, [3, 2, 1, 0]
    worst = 0.0
    for step, ended in schedule(lengths, 11):
        segs = []
        for r, at, n in step:
            if r not in slots:
                slots[r] = free.pop()
            segs.append((slots[r], seqs[r][at:at + n], at, list(range(n))))
        got = eng.forward_segments(segs)
        exp = torch.cat([want[r][at:at + n] for r, at, n in step])
        worst = max(worst, off(got, exp))
        for r in ended:
            eng.kv.release(slots[r])
            free.append(slots.pop(r))
    assert worst < TOL[dtype]


@pytest.mark.parametrize("device", DEVICES)
def test_only_the_wanted_rows_come_back_in_order(device):
    cfg, _, model = make("eights", device, "fp32")
    a, b = tokens(40, cfg["vocab"], 1), tokens(9, cfg["vocab"], 2)
    ra, rb = reference("eights", a), reference("eights", b)
    eng = engine(model)
    got = eng.forward_segments([(0, a[:30], 0, [29, 3]), (1, b[:5], 0, []), (2, b[:7], 0, [0, 6])])
    assert off(got, torch.stack([ra[29], ra[3], rb[0], rb[6]])) < 1e-4
    assert eng.forward_segments([(0, a[30:31], 30, []), (1, b[5:6], 5, [])]) is None
    got = eng.forward_segments([(1, b[6:7], 6, [0]), (0, a[31:32], 31, []), (2, b[7:8], 7, [0])])
    assert off(got, torch.stack([rb[6], rb[7]])) < 1e-4


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_keeps_the_state(dtype, device):
    cfg, _, model = make("eights", device, dtype)
    n = 400 if device == "cuda" else 230
    toks = tokens(n, cfg["vocab"], 4)
    eng = engine(model)
    got = run(eng, 1, toks, [20] + [1] * (n - 20))
    assert off(got, reference("eights", toks)) < TOL[dtype]


@pytest.mark.gpu
def test_steps_without_wanted_logits_do_not_overtake_each_other():
    """Rows of a step are uploaded from pinned memory; a step whose result nobody reads must not be overwritten by the next."""
    cfg, _, model = make("wide", "cuda", "fp32")
    toks = tokens(120, cfg["vocab"], 6)
    want = reference("wide", toks)
    eng = engine(model)
    for _ in range(2):
        for i, t in enumerate(toks[:-1]):
            eng.forward_segments([(0, [t], i, [])])
        assert off(eng.forward_segments([(0, toks[-1:], 119, [0])]), want[-1:]) < 1e-4
        eng.kv.release(0)


@pytest.mark.gpu
@pytest.mark.parametrize("rows", [1, 3, 8, 9, 16])
def test_decode_row_counts_and_graph_replay(rows):
    """Fused and separate forms of a decode step, eager and replayed."""
    cfg, _, model = make("wide", "cuda", "bf16")
    seqs = [tokens(24, cfg["vocab"], 20 + r) for r in range(rows)]
    want = [reference("wide", s) for s in seqs]
    for graphs in (False, True):
        eng = engine(model, pages=2 * rows + 2, slots=rows, use_graphs=graphs)
        for r, s in enumerate(seqs):
            eng.forward_segments([(r, s[:18], 0, [])])
        for i in range(18, 24):
            got = eng.forward_segments([(r, [s[i]], i, [0]) for r, s in enumerate(seqs)])
            assert off(got, torch.stack([w[i] for w in want])) < TOL["bf16"], (graphs, i)


# ------------------------------------------------------------------------------------------ the framework's own entry points
@pytest.mark.parametrize("device", DEVICES)
def test_model_directory_through_the_launcher_and_trace_run(tmp_path, device, capsys):
    from volta_engine_b200.tools import trace_run
    write_model(tmp_path / "m", "eights")
    toks = tokens(100, CONFIGS["eights"]["vocab"], 8)
    want = reference("eights", toks)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:70], "want": [69, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[70:71], "want": []}, {"id": "y", "tokens": toks[:2], "want": [1]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[71:100], "want": [28]}], "end": ["x", "y"]},
             {"step": 3, "entries": [{"id": "z", "tokens": toks[:1], "want": [0]}], "end": ["z"]}]
    rows = {0: [69, 0], 1: [1], 2: [99], 3: [0]}
    for dtype, tol in (("float32", 1e-4), ("bfloat16", TOL["bf16"])):
        rc = trace_run.main(["--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "192"],
                            stdin=io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), device=device)
        assert rc == 0
        assert [ln for ln in capsys.readouterr().out.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
        for i, ps in rows.items():
            raw = torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32)
            assert off(raw.reshape(len(ps), -1), want[ps]) < tol


def test_pool_of_exactly_the_asked_tokens_and_slots(tmp_path):
    from volta_engine_b200.tools import trace_run
    write_model(tmp_path, "eights")
    eng = trace_run.build(str(tmp_path), "float32", 130, 2, "cpu")
    assert eng.kv.free_pages() == 3 and eng.kv.max_slots == 2
    run_ = trace_run.TraceRunner(eng)
    t = tokens(128, CONFIGS["eights"]["vocab"])
    for _ in range(3):                           # 64 + 128 tokens live at a time, again and again
        run_.step([{"id": "a", "tokens": t[:64]}, {"id": "b", "tokens": t[:128]}], ["a", "b"])
    run_.step([{"id": "a", "tokens": t[:1]}, {"id": "b", "tokens": t[:1]}], [])
    with pytest.raises(RuntimeError):
        run_.step([{"id": "c", "tokens": t[:1]}], [])


def test_other_designs_are_refused(tmp_path):
    from volta_engine_b200.models.factory import load_model
    from volta_engine_b200.models.fofosun import FofosunConfig
    bad = dict(CONFIGS["eights"], layers=[dict(CONFIGS["eights"]["layers"][0], type="mamba")])
    with pytest.raises(NotImplementedError):
        FofosunConfig.from_dict(bad)
    bad = dict(CONFIGS["eights"], layers=[dict(CONFIGS["eights"]["layers"][0], mlp={"kind": "moe", "ff": 8})])
    with pytest.raises(NotImplementedError):
        FofosunConfig.from_dict(bad)
    write_model(tmp_path, "eights")
    with pytest.raises(NotImplementedError):
        load_model(tmp_path, "cpu", quantize="nvfp4")


def test_trace_run_says_which_models_it_does_not_run(tmp_path):
    from volta_engine_b200.models.dense import DenseConfig
    from volta_engine_b200.models.factory import kernel_sources, save_dense_checkpoint
    from volta_engine_b200.tools import trace_run
    save_dense_checkpoint(tmp_path / "d", DenseConfig.tiny())
    args = ["--model", str(tmp_path / "d"), "--out", str(tmp_path), "--max-tokens", "128"]
    assert trace_run.main(args + ["--dtype", "bfloat16"], stdin=io.StringIO(""), device="cpu") == 2
    assert trace_run.main(args + ["--dtype", "float32"], stdin=io.StringIO(""), device="cpu") == 3
    assert kernel_sources(tmp_path / "d") is None


def test_a_model_names_the_sources_of_its_kernels(tmp_path):
    """Every entry point the model's Python side calls is defined in the sources that a fresh checkout compiles for it."""
    import re
    from pathlib import Path
    import volta_engine_b200
    from volta_engine_b200.models.factory import kernel_sources
    write_model(tmp_path, "eights")
    part, names = kernel_sources(tmp_path)
    root = Path(volta_engine_b200.__file__).parent
    defined = set()
    for n in names:
        defined |= set(re.findall(r"^int ve_(\w+)\(", (root / "csrc" / "cuda" / n).read_text(), re.M))
    called = set()
    for f in ("ops/latent.py", "ops/linear_attn.py", "ops/rowops.py"):
        called |= set(re.findall(r'call\("(\w+)"', (root / f).read_text()))
    called |= {"gemm_bf16", "gemm_bf16_wide", "gemm_f32", "argmax", "argmax2", "topk"}
    assert part == "fofosun" and called <= defined
