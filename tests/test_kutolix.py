"""The Kutolix decoder against its plain statement: whole prompts, portions, token-by-token decoding, mixed batches, slots and pages
that are used again, long decoding; in fp32 and bf16, on the CPU statements and on the GPU kernels."""
import io
import json

import pytest
import torch

import kutolix_plain as plain
from kutolix_util import CONFIGS, DEVICES, DTYPES, NAMES, TOL, Weights, attention, dense, engine, latent, make, moe, off, one_thread, reference, tokens, write_model, wrong  # noqa: F401
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
    """The residual behind a layer, a result that the next linear adds (or sums and adds) included."""
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
    """Every window passes over decoded tokens."""
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
    from volta_engine_b200.models.kutolix import KutolixConfig, KutolixModel, RandomSource
    cfg = dict(CONFIGS["odd"], **fields)
    src = RandomSource(KutolixConfig.from_dict(cfg), 4)
    return cfg, {n: src.tensor(n) for n in src.shapes}, KutolixModel(KutolixConfig.from_dict(cfg), "cpu", None, "fp32").load(src)


ONE = {
    "embedding scale 1": {"embedding": {"scale": 1.0}},
    "factor 1": {"residual_mult": 1.0},
    "small eps": {"norm": {"eps": 1e-7}},
    "large eps": {"norm": {"eps": 0.5}},
    "narrow cap": {"logit_softcap": 0.7},
    "no feed-forward anywhere": {"layers": [attention(2, 1, 8, 12, 0.4, 11, 8, 100.0), latent(2, 6, 4, 5, 9, 0.5, 13, 50.0, (2.0, 30, 4.0, 1.0))]},
    "one layer": {"layers": [attention(2, 2, 10, 4, 0.6, 9, 2, 20.0, moe(4, 1, 5, 0.3))]},
    "all experts": {"layers": [latent(1, 6, 4, 5, 9, 0.5, 13, 50.0, (2.0, 30, 4.0, 1.0), moe(6, 6, 7, 0.9, 2, 2))]},
    "one expert of one group": {"layers": [attention(2, 1, 8, 12, 0.4, 11, 4, 100.0, moe(6, 1, 7, 0.9, 2, 1))]},
    "same layer twice": {"layers": [attention(2, 1, 8, 12, 0.4, 11, 8, 100.0, dense(9))] * 2},
}


@pytest.mark.parametrize("what", list(ONE))
def test_one_thing_changed(what):
    cfg, w, model = changed(**ONE[what])
    toks = tokens(40, cfg["vocab"], 2)
    want, _ = plain.forward(cfg, w, toks)
    assert off(run(engine(model), 0, toks, [21, 2, 15, 1, 1]), want) < 1e-4


def test_windows_may_be_left_out():
    """A mask that is absent hides nothing; rotations without scaling."""
    L = [attention(2, 1, 8, 12, 0.4, 11, 8, 100.0), latent(2, 6, 4, 5, 9, 0.5, 13, 50.0, (2.0, 30, 4.0, 1.0))]
    for a in L:
        a["mixer"]["mask"] = None
        a["mixer"]["rot"].pop("scaling", None)
    cfg, w, model = changed(layers=L)
    toks = tokens(90, cfg["vocab"], 2)
    assert off(run(engine(model), 0, toks, [70, 2, 16, 1, 1]), plain.forward(cfg, w, toks)[0]) < 1e-4


def test_the_head_is_the_embedding():
    _, _, model = make("eights", "cpu", "bf16")
    assert model.lm_head.weight.data_ptr() == model.embed.data_ptr()
    assert model.weight_bytes() > model.decode_bytes_per_token()         # not every expert is read for a token
    dup = sum(t.numel() * 2 for n, t in Weights("eights", 3).t.items() if t.dim() == 2)
    assert abs(model.weight_bytes() - dup) < 0.1 * dup


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
    from volta_engine_b200.models.kutolix import KutolixConfig, router_of
    C = CONFIGS["eights"]
    L = C["layers"][0]
    for bad in (dict(L, type="mamba"), dict(L, mlp={"kind": "sparse", "ff": 8})):
        with pytest.raises(NotImplementedError):
            KutolixConfig.from_dict(dict(C, layers=[bad]))
    for experts, top, count, keep in ((12, 5, 3, 1), (12, 2, 5, 2), (12, 0, 1, 1), (12, 2, 2, 3)):
        with pytest.raises(ValueError):
            router_of(moe(experts, top, 8, 1.0, count, keep)["router"])
    with pytest.raises(NotImplementedError):
        router_of(moe(2048, 4, 8, 1.0)["router"])
    for field, value in (("mask", {"size": 0}), ("rot", {"base": 10.0, "dims": 26})):
        bad = json.loads(json.dumps(C))
        bad["layers"][1]["mixer"][field] = value
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
    for f in ("ops/gqa.py", "ops/latent.py", "ops/rowops.py", "ops/routed.py"):
        called |= set(re.findall(r'call\("(\w+)"', (root / f).read_text()))
    called |= {"gemm_bf16", "gemm_bf16_wide", "gemm_f32", "argmax", "argmax2", "topk"}
    assert part == "kutolix" and called <= defined
