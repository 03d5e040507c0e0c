"""``bench.py --config siditar``: prefill and decode rates of the Siditar design at a few widths with random bf16 weights, beside the
closest other models of this engine at equal size, and its kernels beside the like kernels of those models, each against its own
roofline.

The closest models: Fofosun (layers listed one by one, fp32 residual, linear recurrences) and the dense grouped-query decoder. Equal
size: the same width, layer count, heads of 128, vocabulary and, through the feed-forward width, weight bytes per layer (within 3 %);
bf16 weights, activations and cache. Siditar and the dense model have one kv head for four query heads. Device time with CUDA
events; weights of a decode step are larger than L2, kernels are timed alone with L2 flushed between iterations.
"""
from __future__ import annotations

import json

import torch

from . import bench_fofosun as BF

WIDTHS = (1024, 2048, 4096)
VOCAB = BF.VOCAB
BIAS_ROWS, BIAS_MAX = 32, 128


def siditar_config(width: int, layers: int, streams: int = 2) -> dict:
    h = width // 128
    left = {"heads": h, "kv_heads": max(1, h // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "bias_max": BIAS_MAX, "q_temp": {"coef": 0.1, "every": 8192}}
    right = {"heads": h, "dim": 128, "vdim": 128, "tau": 16.0}
    layer = {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": 1.0, "right_scale": 1.0},
             "mlp": {"kind": "dense", "ff": width * 23 // 8, "limit": 7.0}}
    return {"architecture": "Siditar", "width": width, "vocab": VOCAB, "norm": {"eps": 1e-5}, "streams": streams, "loop": {"start": 0, "stop": 0, "times": 1},
            "layers": [layer] * layers}


def dense_config(width: int, layers: int):
    from ..models.dense import DenseConfig
    h = width // 128
    return DenseConfig(n_layers=layers, hidden=width, n_q=h, n_kv=max(1, h // 4), head_dim=128, ffn=width * 9 // 2, vocab=VOCAB, qk_norm=True, quant="bf16",
                       lm_head_quant="bf16")


def build(which: str, width: int, layers: int, dev, pages: int, slots: int, max_seq: int):
    from ..runtime.kv_cache import PagedKVCache
    if which == "fofosun":
        return BF.build(which, width, layers, dev, pages, slots, max_seq)
    if which == "siditar":
        from ..models.siditar import SiditarConfig, SiditarModel
        model = SiditarModel(SiditarConfig.from_dict(siditar_config(width, layers)), dev).init_random(seed=1)
        return model, PagedKVCache(model.kv_layers, 1, model.cfg.head_dim, pages, slots, max_seq, dev, v_head_dim=model.kv_v_dim)
    from ..models.dense import DenseModel
    model = DenseModel(dense_config(width, layers), dev).init_random(seed=1)
    return model, PagedKVCache(layers, model.nkv, 128, pages, slots, max_seq, dev)


def run_kernels(width: int, dev) -> dict:
    """Like kernels at one width: a 2048-row prompt portion behind 6144 cached tokens, and one decode row at 8192."""
    from ..models.fofosun import FofosunConfig, FofosunModel
    from ..models.siditar import SiditarConfig, SiditarModel
    from ..ops import kernels as K
    from ..ops.gqa import gqa_scores, gqa_store
    from ..ops.linear_attn import linattn_rows
    from ..ops.rowops import gemv_rows
    from ..runtime.batch import BatchRows
    from ..runtime.kv_cache import PagedKVCache
    kb = BF.KernelBench(dev)
    H, T, ctx = width // 128, 2048, 8192
    G = max(1, H // 4)
    bf = torch.bfloat16
    mine = SiditarModel(SiditarConfig.from_dict(siditar_config(width, 2)), dev).init_random(seed=1)
    other = FofosunModel(FofosunConfig.from_dict(BF.fofosun_config(width, 2)), dev).init_random(seed=1)
    pages = ctx // 64 + 2
    kv = PagedKVCache(1, 1, mine.cfg.head_dim, pages, 2, ctx, dev, v_head_dim=mine.kv_v_dim)
    kvd = PagedKVCache(1, G, 128, pages, 2, ctx, dev)
    for c in (kv, kvd):
        c.reserve(0, ctx)
        c.k.normal_()
        c.v.normal_()
    p0 = ctx - T
    D = H * 128
    ws = K.AttnWorkspace(16, H, 128, 32, dev)
    for n in (T, 1):
        b = BatchRows.make([0] * n, list(range(ctx - n, ctx)), [0] * n, dev, G=H // G, prefill=n > 1, nsplit=max(1, 444 // G))
        kind = "prompt" if n > 1 else "decode"
        b.row_path or b.segments()
        L, O = mine.layers[0], other.layers
        mx = L.mixer
        # ---- recurrences
        rec_flops, sbytes = 4.0 * n * H * 128 * 128, 2 * H * 128 * 128 * 4
        mx.bind(kv)
        proj = torch.randn(n, mx.in_proj.out_features, device=dev)
        pr = proj[:, mx.left.spec.cols:]
        kb.add(f"recurrence {kind}", "siditar (gated linear attention)", lambda: linattn_rows(pr, b, mx.state, mx.right.spec), n * (D * 4 + 16) * 4 + sbytes, rec_flops)
        for li, name in ((0, "hgrn2"), (1, "lightning")):
            om = O[li].mixer
            om.bind(kv)
            po = torch.randn(n, om.in_proj.out_features, device=dev)
            kb.add(f"recurrence {kind}", f"fofosun ({name})", lambda: linattn_rows(po, b, om.state, om.spec), n * D * 4 * 4 + sbytes, rec_flops)
        # ---- attention behind its projections, cache rows written
        pairs = n * (p0 + n / 2) if n > 1 else ctx
        flops = 4.0 * pairs * H * 128
        kvb = ctx * G * 256 * 2
        out = torch.empty(n, D, dtype=bf if n > 1 else torch.float32, device=dev)
        spec = mx.left.spec
        q, _ = gqa_store(spec, proj, b.pos, b.slot, kv, kv.k[0], kv.v[0])
        kb.add(f"attention {kind}", "siditar", lambda: gqa_scores(spec, q, b, kv, kv.k[0], kv.v[0], out), kvb + n * D * 4, flops)
        qkv = torch.randn(n, (H + 2 * G) * 128, device=dev).to(bf)
        kp, vp = kvd.layer(0)
        ns = 1 if n > 1 else max(1, min(32, 444 // G))
        kb.add(f"attention {kind}", "dense", lambda: K.attention(qkv, b.pos, b.slot, kvd.page_table, kp, vp, H, G, 128, 128 ** -0.5, tiles=b.tiles, nsplit=ns, ws=ws),
               kvb + n * D * 4, flops)
        qn = torch.ones(128, dtype=bf, device=dev)

        def dense_store():
            K.rmsnorm_heads_(qkv, qn, n, H, 128, qkv.stride(0), 1e-6, 0.0, 0)
            K.rmsnorm_heads_(qkv, qn, n, G, 128, qkv.stride(0), 1e-6, 0.0, H * 128)
            K.rope_store(qkv, b.pos, b.slot, kvd.page_table, kp, vp, H, G, 128, 128, 1e6)
        kb.add(f"head norms and cache rows {kind}", "siditar", lambda: gqa_store(spec, proj, b.pos, b.slot, kv, kv.k[0], kv.v[0]), n * spec.cols * 6, 0)
        kb.add(f"head norms and cache rows {kind}", "dense (with rotation)", dense_store, n * spec.cols * 4, 0)
        # ---- norms, activations, linears
        S = mine.cfg.streams
        h, ho = torch.randn(n, S, width, device=dev), torch.randn(n, width, device=dev)
        if n > 1:
            x = torch.randn(n, width, device=dev).to(bf)
            kb.add("residual + norm prompt", f"siditar ({S} streams, layer norm)", lambda: L.norm1.rows(h, bf, x, L.write1), n * width * (8 * S + 4), 0)
            kb.add("residual + norm prompt", "fofosun (Dynamic Tanh)", lambda: O[0].norm1.rows(ho, bf, x, O[0].write1), n * width * 12, 0)
            ff = L.ff.down.in_features
            z, zo = torch.randn(n, 2 * ff, device=dev).to(bf), torch.randn(n, O[0].ff.down.in_features, device=dev).to(bf)
            kb.add("activation prompt", "siditar (clamped gated unit)", lambda: L.ff.act.rows(z, bf), n * ff * 6, 0)
            kb.add("activation prompt", "dense (SwiGLU)", lambda: K.gated_act(z, ff), n * ff * 6, 0)
            kb.add("activation prompt", "fofosun (PolyNorm)", lambda: O[0].ff.act.rows(zo, bf), zo.numel() * 4, 0)
            o, y = torch.randn(n, D, device=dev), torch.empty(n, 2 * D, dtype=bf, device=dev)
            gate = mx.right.gate(pr)
            kb.add("output norm prompt", "siditar (gate in fp32)", lambda: mx.right.norm.rows(o, bf, gate=gate, out=y[:, D:]), n * D * 10, 0)
            om = O[1].mixer
            po = torch.randn(n, om.in_proj.out_features, device=dev)
            kb.add("output norm prompt", "fofosun (lightning)", lambda: om.norm.rows(o, bf, gate=om.gate(po)), n * D * 10, 0)
            for who, lin, nm, f32 in (("siditar", mx.in_proj, "in projection", True), ("fofosun", om.in_proj, "in projection", True), ("siditar", mx.out, "out", False),
                                      ("fofosun", om.out, "out", False), ("siditar", L.ff.up, "gate and up", False), ("fofosun", O[0].ff.up, "up", False)):
                xi = torch.randn(n, lin.in_features, device=dev).to(bf)
                kb.add(f"linear prompt ({nm})", who, lambda: lin.forward(xi, out_f32=f32), lin.nbytes() + n * (lin.in_features * 2 + lin.out_features * (4 if f32 else 2)),
                       2.0 * n * lin.in_features * lin.out_features)
        else:
            z, zo = torch.randn(1, L.ff.down.in_features, device=dev).to(bf), torch.randn(1, O[0].ff.up.out_features, device=dev)
            att, o = torch.randn(1, D, device=dev), torch.randn(1, D, device=dev)
            om = O[1].mixer
            po = torch.randn(1, om.in_proj.out_features, device=dev)
            kb.add("linear decode: norm + in projection", "siditar", lambda: gemv_rows(mx.in_proj, 1, out_f32=True, **L.norm1.prologue(h)), mx.in_proj.nbytes(), 0)
            kb.add("linear decode: norm + in projection", "fofosun", lambda: gemv_rows(om.in_proj, 1, out_f32=True, **O[1].norm1.prologue(ho)), om.in_proj.nbytes(), 0)
            kb.add("linear decode: output norm + out + residual", "siditar", lambda: gemv_rows(mx.out, 1, residual=(h, L.write1),
                                                                                            **mx.right.norm.prologue(o, mx.right.gate(pr), head=att)), mx.out.nbytes(), 0)
            kb.add("linear decode: output norm + out + residual", "fofosun", lambda: gemv_rows(om.out, 1, residual=(ho, O[1].write1),
                                                                                            **om.norm.prologue(o, om.gate(po))), om.out.nbytes(), 0)
            kb.add("linear decode: norm + gate and up + activation", "siditar", lambda: gemv_rows(L.ff.up, 1, **L.norm2.prologue(h), **L.ff.act.epilogue()), L.ff.up.nbytes(), 0)
            kb.add("linear decode: norm + up", "fofosun", lambda: gemv_rows(O[0].ff.up, 1, out_f32=True, **O[0].norm2.prologue(ho)), O[0].ff.up.nbytes(), 0)
            kb.add("linear decode: down + residual", "siditar", lambda: gemv_rows(L.ff.down, 1, residual=(h, L.write2), x=z), L.ff.down.nbytes(), 0)
            kb.add("linear decode: activation + down + residual", "fofosun", lambda: gemv_rows(O[0].ff.down, 1, residual=(ho, O[0].write2), **O[0].ff.act.prologue(zo)),
                   O[0].ff.down.nbytes(), 0)
    return {"width": width, "prompt_rows": T, "context": ctx, "peaks": kb.pk, "kernels": kb.rows}


def run(args, ClockSampler) -> int:
    from ..ops import kernels as K
    torch.cuda.set_device(0)
    dev = torch.device("cuda", 0)
    layers = args.layers or 8
    plen = min(args.prompt_len, 8192)
    sampler = ClockSampler(0)
    sampler.start()
    models = []
    for w in WIDTHS:
        for which in ("siditar", "fofosun", "dense"):
            models.append(BF.run_model(which, w, layers, dev, plen, args.steps, max(3, args.warmup), min(args.prefill_chunk, 2048), build))
            torch.cuda.empty_cache()
    kernels = run_kernels(2048, dev)
    clocks = sampler.stop()
    head = next(m for m in models if m["model"] == "siditar" and m["width"] == 2048)
    print(json.dumps({"metric": "decode_tok_s_1stream", "value": head["decode_1"]["tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": args.steps,
                      "warmup": max(3, args.warmup), "ms_per_step": head["decode_1"]["ms_per_step"], "higher_is_better": True, "scaling": "strong",
                      "vs_baseline": None, "dtype": "bf16", "data": "synthetic (random token ids, random bf16 weights)",
                      "config": {"model": f"Siditar, width 2048, {layers} layers", "seq_len": plen, "global_batch": 1, "parallelism": "tp1",
                                 "l2": "decode: weights per step larger than L2; kernels: L2 flushed between iterations"},
                      "models": models, "kernels": kernels, "clocks": clocks, "device_status": K.check_status(dev)}))
    return 0
