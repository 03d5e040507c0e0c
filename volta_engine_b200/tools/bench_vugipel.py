"""``bench.py --config vugipel``: prefill and decode rates of the Vugipel design at a few widths with random bf16 weights, beside the closest
other model of this engine at equal size, and its kernels beside the like kernels of the other designs with listed layers, each against its
own roofline.

Closest: Kutolix with routed feed-forwards (attention and latent attention in turn, the same experts, window, layer count and vocabulary;
here minGRU layers and layers of attention beside retention in turn, whose widths make the weights per token agree). Recurrences are
compared with Fofosun's. bf16 activations and cache. Device time with CUDA events; weights of a decode step are larger than L2, kernels
are timed alone with L2 flushed between iterations.
"""
from __future__ import annotations

import json

import torch

from . import bench_fofosun as BF
from . import bench_kutolix as BK

WIDTHS, VOCAB, WINDOW, EXPERTS, TOP = BK.WIDTHS, BK.VOCAB, BK.WINDOW, BK.EXPERTS, BK.TOP
FIRST = 64


def vugipel_config(width: int, layers: int) -> dict:
    h = width // 128
    r = max(1, h // 4)
    both = {"left": {"heads": h, "kv_heads": max(1, h // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 30.0,
                     "mask": {"size": WINDOW, "keep_first": FIRST}, "rot": {"base": 1e6, "dims": 128}},
            "right": {"heads": r, "dim": 128, "vdim": 128, "decay": [1.0 - 2.0 ** (-5 - 5 * i / max(1, r - 1)) for i in range(r)]}, "left_scale": 1.0, "right_scale": 0.5}
    kinds = [("mingru", {"width": width * 3 // 4}), ("parallel", both)]
    mlp = {"kind": "moe", "router": {"experts": EXPERTS, "top": TOP}, "expert": {"ff": width * 3 // 8}}
    return {"architecture": "Vugipel", "width": width, "vocab": VOCAB, "norm": {"eps": 1e-5},
            "layers": [{"type": kinds[i % 2][0], "mixer": kinds[i % 2][1], "mlp": mlp} for i in range(layers)]}


def make(width: int, layers: int, dev):
    from ..models.vugipel import VugipelConfig, VugipelModel
    return VugipelModel(VugipelConfig.from_dict(vugipel_config(width, layers)), dev).init_random(seed=1)


def build(which: str, width: int, layers: int, dev, pages: int, slots: int, max_seq: int):
    from ..runtime.kv_cache import PagedKVCache
    if which != "vugipel":
        return BK.build(which, width, layers, dev, pages, slots, max_seq)
    model = make(width, layers, dev)
    return model, PagedKVCache(model.kv_layers, 1, model.cfg.head_dim, pages, slots, max_seq, dev, v_head_dim=model.kv_v_dim)


def run_kernels(width: int, dev) -> dict:
    """Like kernels at one width: a 2048-row prompt portion behind 6144 cached tokens, and one decode row at 8192."""
    from ..models.fofosun import FofosunConfig, FofosunModel
    from ..models.kutolix import KutolixConfig, KutolixModel
    from ..ops.gqa import gqa_scores, gqa_store
    from ..ops.linear_attn import LinAttnSpec, LinAttnState, linattn_rows
    from ..ops.min_gru import MinGruState, min_gru_rows
    from ..ops.routed import routed_few, routed_many
    from ..ops.rowops import gemv_rows
    from ..runtime.batch import BatchRows
    from ..runtime.kv_cache import PagedKVCache
    kb = BF.KernelBench(dev)
    H, T, ctx, bf = width // 128, 2048, 8192, torch.bfloat16
    G, D = max(1, H // 4), width
    mine = make(width, 2, dev)
    kut = KutolixModel(KutolixConfig.from_dict(BK.kutolix_config(width, 1, True)), dev).init_random(seed=1)
    fof = FofosunModel(FofosunConfig.from_dict(BF.fofosun_config(width, 2)), dev).init_random(seed=1)
    kv = PagedKVCache(1, 1, mine.cfg.head_dim, ctx // 64 + 2, 2, ctx, dev, v_head_dim=mine.kv_v_dim)
    kv.reserve(0, ctx)
    kv.k.normal_()
    kv.v.normal_()
    R, P, O = mine.layers[0], mine.layers[1], kut.layers[0]
    left, spec, ks = P.mixer.left, P.mixer.left.spec, O.mixer.spec
    retention = LinAttnSpec(H, 128, 128, decay=torch.linspace(0.9, 0.999, H, device=dev), plain=True, q_scale=128 ** -0.5)
    for n in (T, 1):
        b = BatchRows.make([0] * n, list(range(ctx - n, ctx)), [0] * n, dev)
        kind = "prompt" if n > 1 else "decode"
        b.row_path or b.segments()
        # ---- recurrences: projections in, results out, state in and out
        gru, rs = MinGruState(width, 2, dev), LinAttnState(retention, 2, dev)
        pg, pr = torch.randn(n, 3 * width, device=dev), torch.randn(n, 4 * D, device=dev)
        kb.add(f"recurrence {kind}", "vugipel (minGRU, output gate included)", lambda: min_gru_rows(pg, b, gru, bf), n * width * 14 + 8 * width, 0)
        sbytes, flops = 2 * H * 128 * 128 * 4, 4.0 * n * H * 128 * 128
        kb.add(f"recurrence {kind}", "vugipel (retention, heads as the others)", lambda: linattn_rows(pr, b, rs, retention), n * D * 16 + sbytes, flops)
        for li, name in ((0, "hgrn2"), (1, "lightning")):
            m = fof.layers[li].mixer
            m.bind(kv)
            kb.add(f"recurrence {kind}", f"fofosun ({name})", lambda: linattn_rows(pr, b, m.state, m.spec), n * D * 16 + sbytes, flops)
        # ---- attention behind its projections
        keys = ctx - max(0, ctx - n - WINDOW + 1)
        out = torch.empty(n, D, dtype=bf if n > 1 else torch.float32, device=dev)
        proj = torch.randn(n, spec.cols, device=dev)
        q, back = gqa_store(spec, proj, b.pos, b.slot, kv, kv.k[0], kv.v[0])
        pairs = BK._kept(n, ctx)
        kb.add(f"attention {kind}", "vugipel (soft cap, first tokens, values turned back)", lambda: gqa_scores(spec, q, b, kv, kv.k[0], kv.v[0], out, None, back),
               (keys + FIRST) * G * 512 + n * D * 4 + n * 512, 4.0 * (pairs + n * FIRST) * D)
        pk = torch.randn(n, ks.cols, device=dev).to(bf if n > 1 else torch.float32)
        qk, _ = gqa_store(ks, pk, b.pos, b.slot, kv, kv.k[0], kv.v[0])
        kb.add(f"attention {kind}", "kutolix (gate, sink)", lambda: gqa_scores(ks, qk, b, kv, kv.k[0], kv.v[0], out, ks.gate(pk)),
               keys * G * 512 + n * D * (4 + pk.element_size()), 4.0 * pairs * D)
        kb.add(f"rotation, head norms, cache rows {kind}", "vugipel (values too)", lambda: gqa_store(spec, proj, b.pos, b.slot, kv, kv.k[0], kv.v[0]), n * spec.cols * 6, 0)
        kb.add(f"rotation, head norms, cache rows {kind}", "kutolix", lambda: gqa_store(ks, pk, b.pos, b.slot, kv, kv.k[0], kv.v[0]),
               n * ks.gate_col * (pk.element_size() + 2), 0)
        # ---- norms, linears
        h, ho, x = torch.randn(n, width, device=dev), torch.randn(n, width, device=dev), torch.randn(n, width, device=dev).to(bf)
        lins = (("vugipel (minGRU)", R.mixer.in_proj, "in projection"), ("vugipel (attention and retention)", P.mixer.in_proj, "in projection"),
                ("kutolix", O.mixer.in_proj, "in projection"), ("vugipel (minGRU)", R.mixer.out, "out"), ("vugipel (attention and retention)", P.mixer.out, "out"),
                ("kutolix", O.mixer.out, "out"))
        if n > 1:
            kb.add("residual + norm prompt", "vugipel", lambda: R.norm2.rows(h, bf, x, None), n * width * 12, 0)
            kb.add("residual + norm prompt", "kutolix (norm of the result)", lambda: O.norm2.rows(ho, bf, x, O.write1), n * width * 12, 0)
            right = P.mixer.right
            orow, gate = torch.randn(n, D, device=dev), torch.randn(n, D, device=dev)
            yo = torch.empty(n, 2 * D, dtype=bf, device=dev)
            kb.add("output norm prompt", "vugipel (SiLU gate)", lambda: right.norm.rows(orow, bf, gate=gate, out=yo[:, D:]), n * D * 10, 0)
            kb.add("output norm prompt", "fofosun", lambda: fof.layers[0].mixer.norm.rows(orow, bf), n * D * 6, 0)
            for who, lin, nm in lins:
                xi = torch.randn(n, lin.in_features, device=dev).to(bf)
                f32 = nm != "out" and who != "kutolix"
                kb.add(f"linear prompt ({nm})", who, lambda: lin.forward(xi, out_f32=f32),
                       lin.nbytes() + n * (lin.in_features * 2 + lin.out_features * (4 if f32 else 2)), 2.0 * n * lin.in_features * lin.out_features)
        else:
            res, part = torch.randn(1, width, device=dev), torch.randn(1, width, device=dev)
            right = P.mixer.right
            dr = right.spec.heads * right.spec.dv
            att, orow, gate = torch.randn(1, D, device=dev), torch.randn(1, dr, device=dev), torch.randn(1, dr, device=dev)
            y, xa = torch.randn(1, R.mixer.width, device=dev).to(bf), torch.randn(1, D, device=dev).to(bf)
            kb.add("linear decode: residual + norm + in projection", "vugipel (minGRU)", lambda: gemv_rows(R.mixer.in_proj, 1, out_f32=True, **R.norm1.prologue(res)),
                   R.mixer.in_proj.nbytes(), 0)
            kb.add("linear decode: residual + norm + in projection", "vugipel (attention and retention)",
                   lambda: gemv_rows(P.mixer.in_proj, 1, out_f32=True, **P.norm1.prologue(res)), P.mixer.in_proj.nbytes(), 0)
            kb.add("linear decode: residual + norm + in projection", "kutolix", lambda: gemv_rows(O.mixer.in_proj, 1, out_f32=True, **O.norm1.prologue(res, part, O.write2)),
                   O.mixer.in_proj.nbytes(), 0)
            kb.add("linear decode: out", "vugipel (minGRU; residual)", lambda: gemv_rows(R.mixer.out, 1, residual=(ho, None), x=y), R.mixer.out.nbytes(), 0)
            kb.add("linear decode: out", "vugipel (output norm; residual)", lambda: gemv_rows(P.mixer.out, 1, residual=(ho, None), **right.norm.prologue(orow, gate, head=att)),
                   P.mixer.out.nbytes(), 0)
            kb.add("linear decode: out", "kutolix", lambda: gemv_rows(O.mixer.out, 1, out_f32=True, x=xa), O.mixer.out.nbytes(), 0)
            kept = torch.empty(1, width, dtype=bf, device=dev)
            kb.add("linear decode: residual + norm + router", "vugipel", lambda: gemv_rows(R.ff.router, 1, out_f32=True, x_out=kept, **R.norm2.prologue(res)),
                   R.ff.router.nbytes(), 0)
            kb.add("linear decode: residual + norm + router", "kutolix", lambda: gemv_rows(O.ff.router, 1, out_f32=True, **O.norm2.prologue(res, part, O.write1)),
                   O.ff.router.nbytes(), 0)
        # ---- experts behind the router's product
        z = torch.randn(n, EXPERTS, device=dev)
        per_expert, live = 3 * width * R.ff.experts.ff, EXPERTS if n > 1 else TOP
        for who, F in (("vugipel", R.ff), ("kutolix", O.ff)):
            if n > 1:
                kb.add("experts prompt", who, lambda: routed_many(F.choice, F.experts, z, x), live * per_expert * 2 + n * width * 2 * (1 + TOP), 2.0 * n * TOP * per_expert)
            else:
                kb.add("experts decode", who, (lambda: routed_few(F.choice, F.experts, z, x, residual=ho)) if who == "vugipel" else
                       (lambda: routed_few(F.choice, F.experts, z, h, torch.float32)), live * per_expert * 2, 0)
        if n > 1:
            for who, F, read, write in (("vugipel", R.ff, R.norm1, None), ("kutolix", O.ff, O.norm1, O.write2)):
                rr = routed_many(F.choice, F.experts, z, x)
                kb.add("sum of routed results + residual + norm prompt", who, lambda: read.rows(h, bf, rr, write), n * width * (TOP * 2 + 10), 0)
    return {"width": width, "prompt_rows": T, "context": ctx, "window": WINDOW, "first": FIRST, "peaks": kb.pk, "kernels": kb.rows}


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
        for which in ("vugipel", "kutolix_moe"):
            models.append(BF.run_model(which, w, layers, dev, plen, args.steps, max(3, args.warmup), min(args.prefill_chunk, 2048), build))
            torch.cuda.empty_cache()
    kernels = run_kernels(2048, dev)
    clocks = sampler.stop()
    head = next(m for m in models if m["model"] == "vugipel" and m["width"] == 2048)
    print(json.dumps({"metric": "decode_tok_s_1stream", "value": head["decode_1"]["tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": args.steps,
                      "warmup": max(3, args.warmup), "ms_per_step": head["decode_1"]["ms_per_step"], "higher_is_better": True, "scaling": "strong",
                      "vs_baseline": None, "dtype": "bf16", "data": "synthetic (random token ids, random bf16 weights)",
                      "config": {"model": f"Vugipel, width 2048, {layers} layers", "seq_len": plen, "global_batch": 1, "parallelism": "tp1",
                                 "l2": "decode: weights per step larger than L2; kernels: L2 flushed between iterations"},
                      "models": models, "kernels": kernels, "clocks": clocks, "device_status": K.check_status(dev)}))
    return 0
