"""``bench.py --config kutolix``: prefill and decode rates of the Kutolix design at a few widths with random bf16 weights, beside the
closest other models of this engine at equal size, and its kernels beside the like kernels of those models, each against its own
roofline.

Two stacks: attention and latent attention in turn with dense feed-forwards, beside the dense grouped-query decoder (same width, layer
count, heads of 128, window, vocabulary; its feed-forward width makes the weights per token agree); and the same mixers with 8 of 64
experts, beside the mixture-of-experts decoder (experts of the same shape, which that model holds as NVFP4). Latent attention is
compared with Fofosun's. bf16 activations and cache. Device time with CUDA events; weights of a decode step are larger than L2,
kernels are timed alone with L2 flushed between iterations.
"""
from __future__ import annotations

import json

import torch

from . import bench_fofosun as BF

WIDTHS = (1024, 2048, 4096)
VOCAB, WINDOW = BF.VOCAB, 4096
EXPERTS, TOP = 64, 8


def kutolix_config(width: int, layers: int, moe: bool = False) -> dict:
    h = width // 128
    att = {"heads": h, "kv_heads": max(1, h // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": WINDOW}, "rot": {"base": 1e6, "dims": 128}}
    lat = {"heads": h, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5, "mask": {"size": WINDOW},
           "rot": {"base": 1e4, "dims": 64, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    if moe:
        mlp = {"kind": "moe", "router": {"experts": EXPERTS, "top": TOP, "groups": {"count": 8, "keep": 4}}, "expert": {"ff": width * 3 // 8, "limit": 7.0}}
    else:
        mlp = {"kind": "dense", "ff": width * 3}
    kinds = [("attention", att), ("latent_attention", lat)]
    return {"architecture": "Kutolix", "width": width, "vocab": VOCAB, "norm": {"eps": 1e-5}, "embedding": {"scale": 8.0}, "residual_mult": 0.5,
            "logit_softcap": 30.0, "layers": [{"type": kinds[i % 2][0], "mixer": kinds[i % 2][1], "mlp": mlp} for i in range(layers)]}


def _attention_shape(width: int, layers: int) -> dict:
    h = width // 128
    return dict(n_layers=layers, hidden=width, n_q=h, n_kv=max(1, h // 4), head_dim=128, vocab=VOCAB, qk_norm=True, quant="bf16", lm_head_quant="bf16",
                sliding_window=WINDOW, tie_embeddings=True)


def dense_config(width: int, layers: int):
    from ..models.dense import DenseConfig
    return DenseConfig(ffn=(width * 19 // 6 + 267 + 64) // 128 * 128, **_attention_shape(width, layers))


def moe_config(width: int, layers: int):
    from ..models.moe import MoEConfig
    return MoEConfig(ffn=0, n_experts=EXPERTS, top_k=TOP, expert_ffn=width * 3 // 8, expert_quant="nvfp4_random", **_attention_shape(width, layers))


def build(which: str, width: int, layers: int, dev, pages: int, slots: int, max_seq: int):
    from ..runtime.kv_cache import PagedKVCache
    if which.startswith("kutolix"):
        from ..models.kutolix import KutolixConfig, KutolixModel
        model = KutolixModel(KutolixConfig.from_dict(kutolix_config(width, layers, which.endswith("moe"))), dev).init_random(seed=1)
        return model, PagedKVCache(model.kv_layers, 1, model.cfg.head_dim, pages, slots, max_seq, dev, v_head_dim=model.kv_v_dim)
    if which == "moe":
        from ..models.moe import MoEModel
        model = MoEModel(moe_config(width, layers), dev).init_random(seed=1)
    else:
        from ..models.dense import DenseModel
        model = DenseModel(dense_config(width, layers), dev).init_random(seed=1)
    return model, PagedKVCache(layers, model.nkv, 128, pages, slots, max_seq, dev)


def _kept(n: int, ctx: int) -> float:
    """(query, key) pairs of the last n positions of ctx under the window."""
    return float(sum(min(p + 1, WINDOW) for p in range(ctx - n, ctx)))


def run_kernels(width: int, dev) -> dict:
    """Like kernels at one width: a 2048-row prompt portion behind 6144 cached tokens, and one decode row at 8192."""
    from .._lib import call, ptr
    from ..models.fofosun import FofosunConfig, FofosunModel
    from ..models.kutolix import KutolixConfig, KutolixModel
    from ..models.moe import MoEModel
    from ..ops import kernels as K
    from ..ops.gqa import gqa_scores, gqa_store
    from ..ops.latent import latent_rows
    from ..ops.routed import route, routed_few, routed_many
    from ..ops.rowops import gemv_rows
    from ..runtime.batch import BatchRows
    from ..runtime.kv_cache import PagedKVCache
    kb = BF.KernelBench(dev)
    H, T, ctx = width // 128, 2048, 8192
    G, D = max(1, H // 4), width
    bf = torch.bfloat16
    mine = KutolixModel(KutolixConfig.from_dict(kutolix_config(width, 2)), dev).init_random(seed=1)
    routed = KutolixModel(KutolixConfig.from_dict(kutolix_config(width, 1, True)), dev).init_random(seed=1)
    moe = MoEModel(moe_config(width, 1), dev).init_random(seed=1)
    fof = FofosunModel(FofosunConfig.from_dict(BF.fofosun_config(width, 4)), dev).init_random(seed=1)
    pages = ctx // 64 + 2
    kv = PagedKVCache(2, 1, mine.cfg.head_dim, pages, 2, ctx, dev, v_head_dim=mine.kv_v_dim)
    kvd = PagedKVCache(1, G, 128, pages, 2, ctx, dev)
    kvf = PagedKVCache(1, 1, fof.cfg.head_dim, pages, 2, ctx, dev, v_head_dim=8)
    for c in (kv, kvd, kvf):
        c.reserve(0, ctx)
        c.k.normal_()
        c.v.normal_()
    ws = K.AttnWorkspace(16, H, 128, 32, dev)
    A, B, E, F = mine.layers[0], mine.layers[1], routed.layers[0].ff, fof.layers
    spec, mx, lx, fx = A.mixer.spec, A.mixer, B.mixer, F[3].mixer
    for n in (T, 1):
        b = BatchRows.make([0] * n, list(range(ctx - n, ctx)), [0] * n, dev, G=H // G, prefill=n > 1, nsplit=max(1, 444 // G))
        kind, ty = ("prompt", bf) if n > 1 else ("decode", torch.float32)
        size = torch.empty(0, dtype=ty).element_size()
        b.row_path or b.segments()
        keys = ctx - max(0, ctx - n - WINDOW + 1)
        # ---- attention behind its projections, gate included
        pairs = _kept(n, ctx)
        proj = torch.randn(n, mx.in_proj.out_features, device=dev).to(ty)
        out = torch.empty(n, D, dtype=bf, device=dev)
        q, _ = gqa_store(spec, proj, b.pos, b.slot, kv, kv.k[0], kv.v[0])
        kb.add(f"attention {kind}", "kutolix (gate, sink)", lambda: gqa_scores(spec, q, b, kv, kv.k[0], kv.v[0], out, spec.gate(proj)),
               keys * G * 512 + n * D * (4 + size), 4.0 * pairs * D)
        qkv = torch.randn(n, (H + 2 * G) * 128, device=dev).to(bf)
        kp, vp = kvd.layer(0)
        ns = 1 if n > 1 else max(1, min(32, 444 // G))
        kb.add(f"attention {kind}", "dense", lambda: K.attention(qkv, b.pos, b.slot, kvd.page_table, kp, vp, H, G, 128, 128 ** -0.5, window=WINDOW, tiles=b.tiles,
                                                                 nsplit=ns, ws=ws), keys * G * 512 + n * D * 4, 4.0 * pairs * D)
        qn = torch.ones(128, dtype=bf, device=dev)

        def dense_store():
            K.rmsnorm_heads_(qkv, qn, n, H, 128, qkv.stride(0), 1e-6, 0.0, 0)
            K.rmsnorm_heads_(qkv, qn, n, G, 128, qkv.stride(0), 1e-6, 0.0, H * 128)
            K.rope_store(qkv, b.pos, b.slot, kvd.page_table, kp, vp, H, G, 128, 128, 1e6)
        cols = spec.gate_col
        kb.add(f"rotation, head norms, cache rows {kind}", "kutolix", lambda: gqa_store(spec, proj, b.pos, b.slot, kv, kv.k[0], kv.v[0]), n * cols * (size + 2), 0)
        kb.add(f"rotation, head norms, cache rows {kind}", "dense", dense_store, n * cols * 4, 0)
        # ---- latent attention behind its projections, cache rows written
        for who, m, cache, li, window in (("kutolix", lx, kv, 1, WINDOW), ("fofosun (no window)", fx, kvf, 0, 0)):
            s = m.spec
            seen = keys if window else ctx
            pr = pairs if window else n * (ctx - n) + n * (n + 1) / 2
            a = torch.randn(n, H * 192 + 576, device=dev).to(ty if window else torch.float32)
            q2 = a[:, : H * 192] if window else torch.randn(n, H * 192, device=dev).to(ty)
            flops = 2.0 * pr * H * (192 + 128) + 2.0 * seen * 512 * H * 256 if n > 1 else 2.0 * pr * H * (576 + 512)
            nbytes = seen * 576 * 2 + (m.w_uk.numel() + m.w_uv.numel()) * 2 + n * H * 320 * 2
            kb.add(f"latent attention {kind}", who,
                   lambda: latent_rows(s, q2, a[:, H * 192:], m.kv_norm, m.w_uk, m.w_uv, m.ukv, b, cache, cache.k[li]), nbytes, flops)
        # ---- norms, activations, linears
        h, ho = torch.randn(n, width, device=dev), torch.randn(n, width, device=dev)
        ff = A.ff.down.in_features
        if n > 1:
            x = torch.randn(n, width, device=dev).to(bf)
            kb.add("residual + norm prompt", "kutolix (norm of the result)", lambda: A.norm2.rows(h, bf, x, A.write1), n * width * 12, 0)
            kb.add("residual + norm prompt", "fofosun (Dynamic Tanh)", lambda: F[0].norm1.rows(ho, bf, x, F[0].write1), n * width * 12, 0)
            z = torch.randn(n, 2 * ff, device=dev).to(bf)
            kb.add("activation prompt", "kutolix", lambda: A.ff.act.rows(z, bf), n * ff * 6, 0)
            kb.add("activation prompt", "dense", lambda: K.gated_act(z, ff), n * ff * 6, 0)
            for who, lin, nm in (("kutolix", mx.in_proj, "in projection"), ("fofosun", F[0].mixer.in_proj, "in projection"), ("kutolix", mx.out, "out"),
                                 ("fofosun", F[0].mixer.out, "out"), ("kutolix", A.ff.up, "gate and up"), ("fofosun", F[0].ff.up, "gate and up"),
                                 ("kutolix", A.ff.down, "down"), ("fofosun", F[0].ff.down, "down")):
                xi = torch.randn(n, lin.in_features, device=dev).to(bf)
                kb.add(f"linear prompt ({nm})", who, lambda: lin.forward(xi), lin.nbytes() + n * (lin.in_features + lin.out_features) * 2,
                       2.0 * n * lin.in_features * lin.out_features)
        else:
            res, part = torch.randn(1, width, device=dev), torch.randn(1, width, device=dev)
            att, fz = torch.randn(1, D, device=dev).to(bf), torch.randn(1, ff, device=dev).to(bf)
            fi = F[0].mixer
            po, oo, zo = torch.randn(1, fi.in_proj.out_features, device=dev), torch.randn(1, D, device=dev), torch.randn(1, F[0].ff.up.out_features, device=dev)
            kb.add("linear decode: residual + norm + in projection", "kutolix", lambda: gemv_rows(mx.in_proj, 1, out_f32=True, **A.norm1.prologue(res, part, A.write2)),
                   mx.in_proj.nbytes(), 0)
            kb.add("linear decode: residual + norm + in projection", "fofosun", lambda: gemv_rows(fi.in_proj, 1, out_f32=True, **F[0].norm1.prologue(ho)),
                   fi.in_proj.nbytes(), 0)
            kb.add("linear decode: out", "kutolix", lambda: gemv_rows(mx.out, 1, out_f32=True, x=att), mx.out.nbytes(), 0)
            kb.add("linear decode: out", "fofosun (output norm, residual)", lambda: gemv_rows(fi.out, 1, residual=(ho, F[0].write1), **fi.norm.prologue(oo, fi.gate(po))),
                   fi.out.nbytes(), 0)
            kb.add("linear decode: residual + norm + gate and up + activation", "kutolix",
                   lambda: gemv_rows(A.ff.up, 1, **A.norm2.prologue(res, part, A.write1), **A.ff.act.epilogue()), A.ff.up.nbytes(), 0)
            kb.add("linear decode: residual + norm + gate and up + activation", "fofosun (norm + up)",
                   lambda: gemv_rows(F[0].ff.up, 1, out_f32=True, **F[0].norm2.prologue(ho)), F[0].ff.up.nbytes(), 0)
            kb.add("linear decode: down", "kutolix", lambda: gemv_rows(A.ff.down, 1, out_f32=True, x=fz), A.ff.down.nbytes(), 0)
            kb.add("linear decode: down", "fofosun (activation, residual)", lambda: gemv_rows(F[0].ff.down, 1, residual=(ho, F[0].write2), **F[0].ff.act.prologue(zo)),
                   F[0].ff.down.nbytes(), 0)
        # ---- routed feed-forward: experts behind the router's product, without the sum of a prompt row's results
        xr = torch.randn(n, width, device=dev).to(bf)
        zr = torch.randn(n, EXPERTS, device=dev)
        ids, w = route(E.choice, zr)
        bank, ex = moe.layers[0].bank, E.experts
        live = EXPERTS if n > 1 else TOP
        per_expert = 3 * width * ex.ff
        flops = 2.0 * n * TOP * per_expert
        if n > 1:
            kb.add("experts prompt", "kutolix (bf16)", lambda: routed_many(E.choice, ex, zr, xr), live * per_expert * 2 + n * width * 2 * (1 + TOP), flops)
            kb.add("experts prompt", "moe (NVFP4)", lambda: (_select(moe, zr), moe._grouped(bank, xr, ids, n * TOP, TOP, 0)),
                   live * per_expert * 0.5625 + n * width * 2 * (1 + TOP), flops)
            rr = routed_many(E.choice, ex, zr, xr)
            kb.add("sum of routed results prompt", "kutolix (with residual + norm)", lambda: A.norm1.rows(h, bf, rr, A.write2), n * width * (TOP * 2 + 10), 0)
            y = torch.empty(n, width, dtype=bf, device=dev)
            kb.add("sum of routed results prompt", "moe", lambda: call("moe_combine", "plpppiiplplpliii", ptr(rr.d), rr.d.stride(0), ptr(rr.w), ptr(ids), ptr(rr.inv), 0,
                                                                       EXPERTS, 0, 0, 0, 0, ptr(y), y.stride(0), n, TOP, width), n * width * (TOP * 2 + 2), 0)
        else:
            kb.add("experts decode", "kutolix (bf16)", lambda: routed_few(E.choice, ex, zr, res, torch.float32), live * per_expert * 2, 0)

            def theirs():
                i, wt = _select(moe, zr)
                t = torch.empty(TOP, ex.ff, dtype=bf, device=dev)
                call("nvfp4_moe_gemv", "ppppiiplipliiiiif", ptr(bank.gu_p), ptr(bank.gu_s), ptr(bank.gu_g), ptr(i), 0, EXPERTS, ptr(xr), xr.stride(0), TOP, ptr(t), t.stride(0),
                     TOP, 2 * ex.ff, width, 1, 0, 0.0)
                d = torch.empty(TOP, width, dtype=bf, device=dev)
                call("nvfp4_moe_gemv", "ppppiiplipliiiiif", ptr(bank.dn_p), ptr(bank.dn_s), ptr(bank.dn_g), ptr(i), 0, EXPERTS, ptr(t), t.stride(0), 1, ptr(d), d.stride(0),
                     TOP, width, ex.ff, 0, 0, 0.0)
                y = torch.empty(1, width, dtype=bf, device=dev)
                call("moe_combine", "plpppiiplplpliii", ptr(d), d.stride(0), ptr(wt), ptr(i), 0, 0, EXPERTS, 0, 0, 0, 0, ptr(y), y.stride(0), 1, TOP, width)
            kb.add("experts decode", "moe (NVFP4)", theirs, live * per_expert * 0.5625, 0)
            kb.add("linear decode: residual + norm + router", "kutolix", lambda: gemv_rows(E.router, 1, out_f32=True, **A.norm2.prologue(res, part, A.write1)),
                   E.router.nbytes(), 0)
            mr = moe.layers[0].router
            kb.add("linear decode: residual + norm + router", "moe (router alone)", lambda: mr.forward(xr, out_f32=True), mr.nbytes(), 0)
    return {"width": width, "prompt_rows": T, "context": ctx, "window": WINDOW, "peaks": kb.pk, "kernels": kb.rows}


def _select(moe, z):
    from .._lib import call, ptr
    n = z.shape[0]
    i = torch.empty(n, TOP, dtype=torch.int32, device=z.device)
    w = torch.empty(n, TOP, dtype=torch.float32, device=z.device)
    call("router_select", "pliiiipfiippp", ptr(z), z.stride(0), n, EXPERTS, TOP, 0, 0, 1.0, 1, 1, ptr(i), ptr(w), 0)
    return i, w


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
        for which in ("kutolix", "dense", "kutolix_moe", "moe"):
            models.append(BF.run_model(which, w, layers, dev, plen, args.steps, max(3, args.warmup), min(args.prefill_chunk, 2048), build))
            torch.cuda.empty_cache()
    kernels = run_kernels(2048, dev)
    clocks = sampler.stop()
    head = next(m for m in models if m["model"] == "kutolix" and m["width"] == 2048)
    print(json.dumps({"metric": "decode_tok_s_1stream", "value": head["decode_1"]["tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": args.steps,
                      "warmup": max(3, args.warmup), "ms_per_step": head["decode_1"]["ms_per_step"], "higher_is_better": True, "scaling": "strong",
                      "vs_baseline": None, "dtype": "bf16", "data": "synthetic (random token ids, random bf16 weights)",
                      "config": {"model": f"Kutolix, width 2048, {layers} layers", "seq_len": plen, "global_batch": 1, "parallelism": "tp1",
                                 "l2": "decode: weights per step larger than L2; kernels: L2 flushed between iterations"},
                      "models": models, "kernels": kernels, "clocks": clocks, "device_status": K.check_status(dev)}))
    return 0
