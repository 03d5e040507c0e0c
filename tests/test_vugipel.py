"""The Vugipel decoder against its plain statement: whole prompts, portions, token-by-token decoding, mixed batches, slots and pages
that are used again, long decoding; in fp32 and bf16, on the CPU statements and on the GPU kernels."""
import io
import json

import pytest
import torch

import vugipel_plain as plain
from vugipel_util import CONFIGS, DEVICES, DTYPES, NAMES, TOL, Weights, engine, gru, make, moe, off, one_thread, reference, side_by_side, tokens, write_model, wrong  # noqa: F401
from listed_util import CUTS, run, schedule


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompt(name, dtype, device):
    cfg, _, model = make(name, device, dtype)
    toks = tokens(150, cfg["vocab"])
    got = run(engine(model), 2, toks, [150])
    assert got.shape == (150, cfg["vocab"]) and wrong(got, reference(name, toks), dtype) < TOL[dtype]


@pytest.mark.parametrize("device", DEVICES)
def test_residual_after_every_layer(device):
    cfg, w, model = make("eights", device, "fp32")
    toks = tokens(40, cfg["vocab"], 5)
    _, want = plain.forward(cfg, w, toks)
    n = want.shape[0]
    assert n == len(model.layers) == 5
    for cuts in ([40], [1] * 40, [17, 1, 2, 20]):
        model.layer_tap = tap = []
        try:
            run(engine(model, use_graphs=False), 0, toks, cuts)
        finally:
            model.layer_tap = None
        got = torch.cat([torch.stack(tap[i:i + n]) for i in range(0, len(tap), n)], 1).double().cpu()
        assert (got - want).abs().max() < 1e-5 * want.abs().max()


@pytest.mark.gpu
@pytest.mark.parametrize("cuts", [[1] * 20, [20], [7, 13]])
def test_residual_of_fused_decode_steps_and_prompts(cuts):
    """The residual behind a layer, results that linears and experts add to it themselves included."""
    cfg, w, model = make("wide", "cuda", "bf16")
    toks = tokens(20, cfg["vocab"], 5)
    _, want = plain.forward(cfg, w, toks)
    model.layer_tap = tap = []
    try:
        run(engine(model, use_graphs=False), 0, toks, cuts)
    finally:
        model.layer_tap = None
    n = want.shape[0]
    got = torch.cat([torch.stack(tap[i:i + n]) for i in range(0, len(tap), n)], 1).double().cpu()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
    assert err.quantile(0.85) < 0.02


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
        assert wrong(run(eng, slot, toks, cuts), want, dtype) < TOL[dtype], what
        eng.kv.release(slot)                     # the next way of cutting gets used pages
    assert eng.kv.free_pages() == eng.kv.num_pages - 1


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["eights", "odd", "wide"])
def test_mixed_batches_equal_each_alone(name, dtype, device):
    cfg, _, model = make(name, device, dtype)
    lengths = [150, 1, 23, 97, 64, 65, 130, 2]
    seqs = [tokens(150, cfg["vocab"])[:n] if n != 97 else tokens(97, cfg["vocab"], 9) for n in lengths]
    full = reference(name, seqs[0])
    want = [full[:n] if n != 97 else reference(name, seqs[3]) for n in lengths]
    eng = engine(model, pages=1 + 3 * 3 + 2)     # what four live requests need at most: pages come round again
    slots, free = {}, [3, 2, 1, 0]
    got, exp = [], []
    for step, ended in schedule(lengths, 11):
        segs = []
        for r, at, n in step:
            if r not in slots:
                slots[r] = free.pop()
            segs.append((slots[r], seqs[r][at:at + n], at, list(range(n))))
        got.append(eng.forward_segments(segs).float().cpu().clone())
        exp.append(torch.cat([want[r][at:at + n] for r, at, n in step]))
        for r in ended:
            eng.kv.release(slots[r])
            free.append(slots.pop(r))
    assert wrong(torch.cat(got), torch.cat(exp), dtype) < TOL[dtype]


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


@pytest.mark.gpu
def test_wanted_rows_of_a_few_rows_that_carry_their_norms():
    """A short portion (fused form) of which one row's logits, or none, are asked for: the last result still enters the residual."""
    cfg, _, model = make("wide", "cuda", "bf16")
    t = tokens(12, cfg["vocab"], 6)
    want = reference("wide", t)
    eng = engine(model)
    got = eng.forward_segments([(0, t[:6], 0, [5, 1])])
    assert wrong(got, want[[5, 1]], "bf16") < 2 * TOL["bf16"]
    assert eng.forward_segments([(0, t[6:8], 6, [])]) is None
    got = eng.forward_segments([(0, t[8:12], 8, [3])])
    assert wrong(got, want[[11]], "bf16") < 2 * TOL["bf16"]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype, device):
    """Every window passes over decoded tokens, the first tokens stay in sight, the states go on."""
    cfg, _, model = make("eights", device, dtype)
    n = 400 if device == "cuda" else 200
    toks = tokens(400, cfg["vocab"], 4)[:n]
    got = run(engine(model), 1, toks, [20] + [1] * (n - 20))
    assert wrong(got, reference("eights", toks), dtype) < TOL[dtype]


@pytest.mark.gpu
@pytest.mark.parametrize("rows", [1, 3, 8, 9, 16])
def test_decode_row_counts_and_graph_replay(rows):
    """Fused and separate forms of a decode step, eager and replayed."""
    cfg, _, model = make("wide", "cuda", "bf16")
    seqs = [tokens(24, cfg["vocab"], 20 + r) for r in range(rows)]
    want = [reference("wide", s) for s in seqs]
    for graphs in (False, True):
        eng = engine(model, pages=2 * rows + 2, slots=rows, use_graphs=graphs)
        got, exp = [], []
        for r, s in enumerate(seqs):
            eng.forward_segments([(r, s[:14], 0, [])])
        for i in range(14, 24):
            got.append(eng.forward_segments([(r, [s[i]], i, [0]) for r, s in enumerate(seqs)]).float().cpu().clone())
            exp.append(torch.stack([w[i] for w in want]))
        assert wrong(torch.cat(got), torch.cat(exp), "bf16") < TOL["bf16"], graphs


@pytest.mark.gpu
def test_prompt_of_many_pages_beside_decode_rows():
    """Prompt portions over many pages: all stages of the page rings come round, every tile starts somewhere else in its window."""
    cfg, _, model = make("wide", "cuda", "bf16")
    toks = tokens(900, cfg["vocab"], 7)
    want = reference("wide", toks)
    for cuts in ([900], [700, 1, 130, 69], [896, 1, 1, 1, 1], [333, 17, 550]):
        eng = engine(model)
        assert wrong(run(eng, 3, toks, cuts), want, "bf16") < TOL["bf16"], cuts


# ------------------------------------------------------------------------------------------ one thing at a time
def changed(**fields):
    """The configuration "odd" with other top-level fields, its weights, and its model on the CPU."""
    from volta_engine_b200.models.vugipel import VugipelConfig, VugipelModel, RandomSource
    cfg = dict(CONFIGS["odd"], **fields)
    src = RandomSource(VugipelConfig.from_dict(cfg), 4)
    return cfg, {n: src.tensor(n) for n in src.shapes}, VugipelModel(VugipelConfig.from_dict(cfg), "cpu", None, "fp32").load(src)


LEFT, RIGHT = (2, 1, 8, 12, 0.4, 11, 3, 8, 100.0, 5.0), (2, 6, 4, [0.9, 0.99])


def left(**changes):
    names = ("heads", "kv_heads", "dim", "vdim", "scale", "window", "first", "dims", "base", "cap")
    return tuple(changes.get(n, v) for n, v in zip(names, LEFT))


ONE = {
    "small eps": {"norm": {"eps": 1e-7}},
    "large eps": {"norm": {"eps": 0.5}},
    "no feed-forward anywhere": {"layers": [gru(9), side_by_side(LEFT, RIGHT)]},
    "one layer": {"layers": [gru(11, moe(4, 1, 5))]},
    "recurrences alone": {"layers": [gru(16, moe(4, 2, 8)), gru(24)]},
    "attention first": {"layers": [side_by_side(LEFT, RIGHT, mlp=moe(3, 1, 6)), gru(7)]},
    "all experts": {"layers": [side_by_side(LEFT, RIGHT, mlp=moe(6, 6, 7))]},
    "one expert": {"layers": [gru(5, moe(1, 1, 7))]},
    "same layer twice": {"layers": [side_by_side(LEFT, RIGHT, mlp=moe(3, 1, 6))] * 2},
    "a narrow cap": {"layers": [side_by_side(left(cap=0.3), RIGHT)]},
    "a wide cap": {"layers": [side_by_side(left(cap=500.0), RIGHT)]},
    "no first tokens": {"layers": [side_by_side(left(first=0), RIGHT)]},
    "first tokens beyond the window": {"layers": [side_by_side(left(first=20), RIGHT)]},
    "first tokens beyond the prompt": {"layers": [side_by_side(left(first=90), RIGHT)]},
    "one rotated pair": {"layers": [side_by_side(left(dims=2), RIGHT)]},
    "one pair of values": {"layers": [side_by_side(left(vdim=2), RIGHT)]},
    "scales of one": {"layers": [side_by_side(LEFT, RIGHT, (1.0, 1.0))]},
    "left alone": {"layers": [side_by_side(LEFT, RIGHT, (1.0, 0.0))]},
    "right alone": {"layers": [side_by_side(LEFT, RIGHT, (0.0, 1.0))]},
    "negative scales": {"layers": [side_by_side(LEFT, RIGHT, (-0.8, -1.5))]},
    "a head that forgets at once, one that never does": {"layers": [side_by_side(LEFT, (2, 6, 4, [0.0, 1.0]))]},
}


@pytest.mark.parametrize("what", list(ONE))
def test_one_thing_changed(what):
    cfg, w, model = changed(**ONE[what])
    toks = tokens(40, cfg["vocab"], 2)
    want, _ = plain.forward(cfg, w, toks)
    assert off(run(engine(model), 0, toks, [21, 2, 15, 1, 1]), want) < 1e-4


def test_a_mask_may_be_left_out():
    """A mask that is absent hides nothing; one without first tokens keeps none."""
    for mask in (None, {"size": 9}):
        L = side_by_side(LEFT, RIGHT)
        L["mixer"]["left"]["mask"] = mask
        cfg, w, model = changed(layers=[L])
        toks = tokens(90, cfg["vocab"], 2)
        assert off(run(engine(model), 0, toks, [70, 2, 16, 1, 1]), plain.forward(cfg, w, toks)[0]) < 1e-4


def test_bytes_of_a_step_and_of_the_model():
    _, _, model = make("eights", "cpu", "bf16")
    assert model.weight_bytes() > model.decode_bytes_per_token()         # not every expert is read for a token
    once = sum(t.numel() * 2 for n, t in Weights("eights", 3).t.items() if t.dim() == 2)
    assert abs(model.weight_bytes() - once) < 0.1 * once
    assert model.state_bytes_per_slot() == 4 * (88 + 3 * 16 * 24 + 136 + 2 * 40 * 48 + 56 * 16)


# ------------------------------------------------------------------------------------------ the framework's own entry points
@pytest.mark.parametrize("device", DEVICES)
def test_model_directory_through_the_launcher_and_trace_run(tmp_path, device, capsys):
    from volta_engine_b200.tools import trace_run
    write_model(tmp_path / "m", "eights")
    toks = tokens(100, CONFIGS["eights"]["vocab"], 8)
    want = reference("eights", toks)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:70], "want": [69, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[70:71], "want": []}, {"id": "y", "tokens": toks[:2], "want": [1]}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[71:100], "want": list(range(29))}], "end": ["x", "y"]},
             {"step": 3, "entries": [{"id": "z", "tokens": toks[:1], "want": [0]}], "end": ["z"]}]
    rows = {0: [69, 0], 1: [1], 2: list(range(71, 100)), 3: [0]}
    for dtype, short in (("float32", "fp32"), ("bfloat16", "bf16")):
        rc = trace_run.main(["--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "192"],
                            stdin=io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), device=device)
        assert rc == 0
        assert [ln for ln in capsys.readouterr().out.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
        got = []
        for i, ps in rows.items():
            raw = torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32)
            got.append(raw.reshape(len(ps), -1))
        assert wrong(torch.cat(got), want[sum(rows.values(), [])], short) < TOL[short]


def test_what_is_refused(tmp_path):
    from volta_engine_b200.models.factory import load_model
    from volta_engine_b200.models.vugipel import VugipelConfig, router_of
    C = CONFIGS["eights"]
    L = C["layers"][0]
    for bad in (dict(L, type="mamba"), dict(L, type="lightning"), dict(L, mlp={"kind": "dense", "ff": 8})):
        with pytest.raises(NotImplementedError):
            VugipelConfig.from_dict(dict(C, layers=[bad]))
    for experts, top in ((12, 0), (3, 4)):
        with pytest.raises(ValueError):
            router_of(moe(experts, top, 8)["router"])
    with pytest.raises(NotImplementedError):
        router_of(moe(2048, 4, 8)["router"])
    for field, value in (("mask", {"size": 0, "keep_first": 1}), ("rot", {"base": 10.0, "dims": 26}), ("vdim", 7)):
        bad = json.loads(json.dumps(C))
        bad["layers"][1]["mixer"]["left"][field] = value
        write = tmp_path / field
        write_model(write, "eights")
        (write / "config.json").write_text(json.dumps(bad))
        with pytest.raises(ValueError):
            load_model(write, "cpu")
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
    for f in ("ops/gqa.py", "ops/min_gru.py", "ops/linear_attn.py", "ops/rowops.py", "ops/routed.py"):
        called |= set(re.findall(r'call\("(\w+)"', (root / f).read_text()))
    called |= {"gemm_bf16", "gemm_bf16_wide", "gemm_f32", "argmax", "argmax2", "topk"}
    assert part == "vugipel" and called <= defined
