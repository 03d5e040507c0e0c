"""The Siditar decoder against its plain statement: whole prompts, portions, token-by-token decoding, mixed batches, slots and
pages that are used again, long decoding; in fp32 and bf16, on the CPU statements and on the GPU kernels."""
import io
import json

import pytest
import torch

import siditar_plain as plain
from listed_util import CUTS, run, schedule
from siditar_util import CONFIGS, DEVICES, DTYPES, TOL, engine, make, off, one_thread, reference, tokens, write_model  # noqa: F401

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
def test_residual_after_every_layer_run(device):
    cfg, w, model = make("eights", device, "fp32")
    toks = tokens(40, cfg["vocab"], 5)
    _, want = plain.forward(cfg, w, toks)
    assert want.shape[0] == len(model.layers) == 5
    for cuts in ([40], [1] * 40):
        model.layer_tap = tap = []
        try:
            run(engine(model, use_graphs=False), 0, toks, cuts)
        finally:
            model.layer_tap = None
        n = want.shape[0]
        got = torch.cat([torch.stack(tap[i:i + n]) for i in range(0, len(tap), n)], 1).double().cpu()
        assert (got - want).abs().max() < 2e-4 * want.abs().max()


@pytest.mark.gpu
def test_residual_of_fused_decode_steps():
    cfg, w, model = make("wide", "cuda", "bf16")
    toks = tokens(20, cfg["vocab"], 5)
    _, want = plain.forward(cfg, w, toks)
    model.layer_tap = tap = []
    try:
        run(engine(model, use_graphs=False), 0, toks, [1] * 20)
    finally:
        model.layer_tap = None
    n = want.shape[0]
    got = torch.cat([torch.stack(tap[i:i + n]) for i in range(0, len(tap), n)], 1).double().cpu()
    assert (got - want).pow(2).mean().sqrt() < 0.03 * want.pow(2).mean().sqrt()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_portions_and_decoding(name, dtype, device):
    cfg, _, model = make(name, device, dtype)
    toks = tokens(150, cfg["vocab"])
    want = reference(name, toks)
    eng = engine(model)
    for i, (what, cuts) in enumerate(CUTS.items()):
        if device == "cpu" and (dtype == "bf16") == bool(i % 2):
            continue
        slot = i % 4
        assert off(run(eng, slot, toks, cuts), want) < TOL[dtype], what
        eng.kv.release(slot)                     # the next way of cutting gets used pages and a used state slot
    assert eng.kv.free_pages() == eng.kv.num_pages - 1


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["eights", "odd", "wide"])
def test_mixed_batches_equal_each_alone(name, dtype, device):
    if device == "cpu" and name == "wide":
        pytest.skip("long on the CPU statements")
    cfg, _, model = make(name, device, dtype)
    lengths = [150, 1, 23, 97, 64, 65, 130, 2]
    seqs = [tokens(150, cfg["vocab"])[:n] if n != 97 else tokens(97, cfg["vocab"], 9) for n in lengths]
    full = reference(name, seqs[0])
    want = [full[:n] if n != 97 else reference(name, seqs[3]) for n in lengths]
    eng = engine(model, pages=1 + 3 * 3 + 2)     # what four live requests need at most: pages come round again
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
def test_long_decoding(dtype, device):
    cfg, _, model = make("eights", device, dtype)
    n = 400 if device == "cuda" else 200
    toks = tokens(400, cfg["vocab"], 4)[:n]
    got = run(engine(model), 1, toks, [20] + [1] * (n - 20))
    assert off(got, reference("eights", toks)) < TOL[dtype]


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


@pytest.mark.gpu
def test_prompt_of_many_pages_beside_decode_rows():
    """Prompt portions over many pages (all stages of the page rings come round) and decode rows with many key splits."""
    cfg, _, model = make("wide", "cuda", "bf16")
    toks = tokens(900, cfg["vocab"], 7)
    want = reference("wide", toks)
    for cuts in ([900], [700, 1, 130, 69], [896, 1, 1, 1, 1]):
        eng = engine(model)
        assert off(run(eng, 3, toks, cuts), want) < TOL["bf16"], cuts


# ------------------------------------------------------------------------------------------ what a layer of its own shows
def changed(name, dtype="fp32", **fields):
    """The configuration ``name`` with other top-level fields, and its model on the CPU."""
    from siditar_util import Weights
    from volta_engine_b200.models.siditar import SiditarConfig, SiditarModel
    cfg = dict(CONFIGS[name], **fields)
    w = Weights(name, 3)
    return cfg, w.t, SiditarModel(SiditarConfig.from_dict(cfg), "cpu", None, dtype).load(w)


@pytest.mark.parametrize("loop", [None, (0, 3, 1), (2, 2, 4), (0, 1, 3), (2, 3, 2)])
def test_layers_that_run_again(loop):
    """Every pass has a cache layer and a state of its own: portions and decoding agree with the plain stack."""
    cfg, w, model = changed("eights", loop=dict(zip(("start", "stop", "times"), loop)) if loop else None)
    toks = tokens(24, cfg["vocab"], 2)
    want, _ = plain.forward(cfg, w, toks)
    assert model.kv_layers == len(model.layers) == len(plain.layer_runs(3, cfg["loop"]))
    assert off(run(engine(model), 0, toks, [11, 2, 9, 1, 1]), want) < 1e-4


def test_weights_are_loaded_once_whatever_the_passes():
    _, _, once = changed("eights", loop=None)
    _, _, twice = changed("eights", loop={"start": 0, "stop": 3, "times": 2})
    assert once.weight_bytes() == twice.weight_bytes()
    assert twice.decode_bytes_per_token() > 1.5 * once.decode_bytes_per_token()
    assert twice.layers[0].mixer.in_proj is twice.layers[3].mixer.in_proj
    assert twice.state_bytes_per_slot() == 2 * once.state_bytes_per_slot()


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


def test_what_is_refused(tmp_path):
    from volta_engine_b200.models.factory import load_model
    from volta_engine_b200.models.siditar import SiditarConfig
    L = CONFIGS["eights"]["layers"][0]
    for bad in (dict(CONFIGS["eights"], layers=[dict(L, type="mamba")]), dict(CONFIGS["eights"], layers=[dict(L, mlp={"kind": "moe", "ff": 8})]),
                dict(CONFIGS["eights"], streams=9)):
        with pytest.raises(NotImplementedError):
            SiditarConfig.from_dict(bad)
    for loop in ({"start": 2, "stop": 1, "times": 1}, {"start": 0, "stop": 4, "times": 1}, {"start": 0, "stop": 1, "times": 0}):
        with pytest.raises(ValueError):
            SiditarConfig.from_dict(dict(CONFIGS["eights"], loop=loop))
    write_model(tmp_path, "eights")
    with pytest.raises(NotImplementedError):
        load_model(tmp_path, "cpu", quantize="nvfp4")


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
    for f in ("ops/gqa.py", "ops/linear_attn.py", "ops/rowops.py"):
        called |= set(re.findall(r'call\("(\w+)"', (root / f).read_text()))
    called |= {"gemm_bf16", "gemm_bf16_wide", "gemm_f32", "argmax", "argmax2", "topk"}
    assert part == "siditar" and called <= defined
