"""``bench.py --config fofosun``: prefill and decode rates of the Fofosun design at a few widths with random bf16 weights, beside the
closest other assembly of this engine at equal size (``models/glm5.py`` with dense feed-forwards: Kimi-delta-attention mixers
and latent attention), and its kernels beside the like kernels of that assembly, each against its own roofline.

Equal size: the same width, layer count, head counts and widths, ranks, vocabulary and feed-forward parameters (the other
assembly's gated feed-forward has three matrices of width f, this one two of width 1.5 f); bf16 weights, activations and
cache on both sides; one latent-attention layer in four. Device time with CUDA events; weights of a decode step are larger
than L2, kernels are timed alone with L2 flushed (a 256 MB write) between iterations.
"""
from __future__ import annotations

import json
import os

import torch

WIDTHS = (1024, 2048, 4096)
VOCAB = 32768


def fofosun_config(width: int, layers: int) -> dict:
    heads, ff = width // 128, width * 6
    mlp = {"kind": "dense", "ff": ff}
    rec = {"heads": heads, "dim": 128, "vdim": 128}
    light = dict(rec, decay=[1.0 - 2.0 ** (-2 - 6 * h / max(1, heads - 1)) for h in range(heads)])
    att = {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "q_rank": width // 2, "rot": {"base": 10000.0, "dims": 64},
           "scale": 192 ** -0.5}
    kinds = [("hgrn2", rec), ("lightning", light), ("hgrn2", rec), ("latent_attention", att)]
    return {"architecture": "Fofosun", "width": width, "vocab": VOCAB, "norm": {"eps": 1e-5},
            "layers": [{"type": kinds[i % 4][0], "mixer": kinds[i % 4][1], "mlp": mlp} for i in range(layers)]}


def closest_config(width: int, layers: int):
    from ..models.glm5 import Glm5NextConfig
    h = width // 128
    return Glm5NextConfig(n_layers=layers, hidden=width, n_q=h, n_kv=1, head_dim=576, ffn=width * 4, vocab=VOCAB, n_experts=1, top_k=1, expert_ffn=128,
                          shared_ffn=0, first_dense_layers=layers, full_interval=4, linear_mixer="kda", gdn_k_heads=h, gdn_v_heads=h, kda_rank=128,
                          attn_gate=False, residual="plain", mtp_layers=0, q_lora_rank=width // 2, dsa=False, quant="bf16", lm_head_quant="bf16")


def build(which: str, width: int, layers: int, dev, pages: int, slots: int, max_seq: int):
    from ..runtime.kv_cache import PagedKVCache
    if which == "fofosun":
        from ..models.fofosun import FofosunConfig, FofosunModel
        model = FofosunModel(FofosunConfig.from_dict(fofosun_config(width, layers)), dev).init_random(seed=1)
        return model, PagedKVCache(model.kv_layers, 1, model.cfg.head_dim, pages, slots, max_seq, dev, v_head_dim=8)
    from ..models.glm5 import Glm5NextModel
    model = Glm5NextModel(closest_config(width, layers), dev).init_random(seed=1)
    return model, model.make_cache(pages, slots, max_seq)


def run_model(which: str, width: int, layers: int, dev, prompt_len: int, steps: int, warm: int, chunk: int, build=build) -> dict:
    """Prefill and decode rates of one model. ``build(which, width, layers, device, pages, slots, max_seq)`` -> (model, cache)."""
    from .. import _lib
    from ..runtime.engine import Engine
    streams = 16
    per = (prompt_len + 8 * (steps + warm) + 127) // 64
    model, kv = build(which, width, layers, dev, per + streams * 8 + 8, streams, prompt_len + 8 * (steps + warm) + 64)
    eng = Engine(model, kv, prefill_chunk=chunk)
    g = torch.Generator().manual_seed(0)
    prompt = torch.randint(0, VOCAB, (prompt_len,), generator=g).tolist()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)

    def timed(fn):
        torch.cuda.synchronize()
        e0.record()
        r = fn()
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1), r
    out = {"model": which, "width": width, "layers": layers, "weight_gb": round(model.decode_bytes_per_token() / 1e9, 3)}
    for _ in range(2):
        eng.prefill(0, prompt)
        kv.release(0)
    ms = []
    for _ in range(3):
        t, tok = timed(lambda: eng.prefill(0, prompt))
        ms.append(t)
        kv.release(0)
    out["prefill_tok_s"] = round(prompt_len / min(ms) * 1e3, 1)
    tok = eng.prefill(0, prompt)
    pos = prompt_len
    l0 = _lib.launch_count
    eng.decode_chain([tok], [pos], [0], 1)
    out["launches_per_step"] = _lib.launch_count - l0
    pos += 1
    for n, rows in (("decode_1", 1), ("decode_16", streams)):
        if rows > 1:
            for s in range(1, rows):
                eng.prefill(s, prompt[:256])
        ids, poss, slots = [5] * rows, [pos] + [256] * (rows - 1), list(range(rows))
        eng.decode_chain(ids, poss, slots, max(3, warm))
        for s, p in zip(slots, poss):
            kv.reserve(s, p + warm + steps + 8)
        t, _ = timed(lambda: [eng._run_rows(rows) for _ in range(steps)])
        pos += steps + max(3, warm)
        out[n] = {"ms_per_step": round(t / steps, 4), "tok_s": round(rows * steps / t * 1e3, 1),
                  "weight_gbs": round(model.decode_bytes_per_token() / (t / steps) / 1e6, 1)}
    return out


def peaks() -> dict:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            p = json.load(f)
        return {"gbs": p["hbm_gbs"], "tflops": p["bf16_tflops"], "of": "measured"}
    return {"gbs": 6650.0, "tflops": 1590.0, "of": "fallback"}


class KernelBench:
    def __init__(self, dev):
        self.dev, self.pk = dev, peaks()
        self.flush = torch.empty(64 << 20, dtype=torch.float32, device=dev)
        self.rows = []

    def time(self, fn, iters: int = 10) -> float:
        """Median microseconds of one call with a cold L2."""
        for _ in range(3):
            fn()
        ts = []
        for _ in range(iters):
            for _ in range(3):                      # (long enough that the host is ahead of the device when the call is made)
                self.flush.fill_(1.0)
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            ts.append((e0, e1))
        torch.cuda.synchronize()
        ts = sorted(a.elapsed_time(b) for a, b in ts)
        return ts[len(ts) // 2] * 1e3

    def add(self, what: str, who: str, fn, nbytes: float, flops: float):
        us = self.time(fn)
        bound = max(nbytes / self.pk["gbs"] / 1e3, flops / self.pk["tflops"] / 1e6)
        self.rows.append({"kernel": what, "of": who, "us": round(us, 2), "roofline_us": round(bound, 2), "fraction": round(bound / us, 4)})


def run_kernels(width: int, dev) -> dict:
    """Like kernels of the two designs at one width: a 2048-row prompt portion behind 6144 cached tokens, and one decode row."""
    from .._lib import call, ptr
    from ..models.fofosun import FofosunConfig, FofosunModel
    from ..models.glm5 import Glm5NextModel
    from ..ops import kernels as K
    from ..ops.linear_attn import linattn_rows
    from ..ops.rowops import gemv_rows
    from ..runtime.batch import BatchRows
    from ..runtime.kv_cache import PagedKVCache
    kb = KernelBench(dev)
    H, T, ctx = width // 128, 2048, 8192
    bf, f32 = torch.bfloat16, torch.float32
    mine = FofosunModel(FofosunConfig.from_dict(fofosun_config(width, 4)), dev).init_random(seed=1)
    other = Glm5NextModel(closest_config(width, 4), dev).init_random(seed=1)
    kv = PagedKVCache(1, 1, mine.cfg.head_dim, ctx // 64 + 2, 2, ctx, dev, v_head_dim=8)
    kvo = other.make_cache(ctx // 64 + 2, 2, ctx)
    for c in (kv, kvo):
        c.reserve(0, ctx)
        c.k.normal_()
    other.ensure_workspace(16, 32)
    p0 = ctx - T
    big = lambda: BatchRows.make([0] * T, list(range(p0, ctx)), [0] * T, dev, G=1, prefill=True)
    one = lambda: BatchRows.make([0], [ctx - 1], [0], dev, nsplit=32)
    D = H * 128
    for n, mk in ((T, big), (1, one)):
        b, kind = mk(), "prompt" if n > 1 else "decode"
        b.row_path or b.segments()
        # recurrence: projections in, outputs out, state in and out
        rec_flops = 4.0 * n * H * 128 * 128
        for li, name in ((0, "hgrn2"), (1, "lightning")):
            mx = mine.layers[li].mixer
            mx.bind(kv)
            proj = torch.randn(n, mx.in_proj.out_features, device=dev)
            kb.add(f"recurrence {kind}", name, lambda: linattn_rows(proj, b, mx.state, mx.spec), n * D * 4 * 4 + 2 * mx.state.rec[0].numel() * 4, rec_flops)
        d, C = other.dims, other.dims.conv_dim
        st = other._states(kvo)[0]
        pr = torch.randn(n, d.proj_out, device=dev).to(bf)
        u, gb = torch.rand(n, C, device=dev), torch.rand(n, 2 * H, device=dev)
        kd, o = torch.rand(n, D, device=dev), torch.empty(n, D, device=dev)
        kb.add(f"recurrence {kind}", "kda", lambda: call("kda_recurrent", "plppppppppiiiiiii", ptr(pr), pr.stride(0), ptr(b.pos), ptr(b.slot), ptr(st.conv), ptr(st.rec),
                                                         ptr(u), ptr(gb), ptr(o), ptr(kd), n, d.n_k, d.n_v, d.dk, d.dv, d.conv_k, st.conv.shape[0]),
               n * D * 4 * 5 + 2 * st.rec[0].numel() * 4, rec_flops)
        # latent attention behind its query projection, with the cache row written
        pairs = n * (p0 + n / 2) if n > 1 else ctx
        mx = mine.layers[3].mixer
        s = mx.spec
        q = torch.randn(n, H * 192, device=dev, dtype=f32 if n == 1 else bf)
        a = torch.randn(n, 576, device=dev)
        flops = 2.0 * pairs * H * (192 + 128) + 2.0 * ctx * 512 * H * 256 if n > 1 else 2.0 * pairs * H * (576 + 512)
        kb_bytes = ctx * 576 * 2 + (mx.w_uk.numel() + mx.w_uv.numel()) * 2 + n * H * 320 * 2
        from ..ops.latent import latent_rows
        kb.add(f"latent attention {kind}", "fofosun", lambda: latent_rows(s, q, a, mx.kv_norm, mx.w_uk, mx.w_uv, mx.ukv, b, kv, kv.k[0]), kb_bytes, flops)
        L = other.layers[3]
        qo, ck, kr = torch.randn(n, H * 192, device=dev).to(bf), torch.randn(n, 512, device=dev).to(bf), torch.randn(n, 64, device=dev).to(bf)

        def theirs():
            pool = kvo.k[0]
            call("mla_rope_store", "pliiplplpppipifi", ptr(qo), qo.stride(0), 192, H, ptr(ck), ck.stride(0), ptr(kr), kr.stride(0), ptr(b.pos), ptr(b.slot),
                 ptr(kvo.page_table), kvo.page_table.shape[1], ptr(pool), n, 1e4, 0)
            if n > 1:
                return other._attn_prefill_expanded(L, qo, b, kvo, pool)
            qa, ol = torch.empty(n, H, 576, dtype=bf, device=dev), torch.empty(n, H, 512, dtype=bf, device=dev)
            call("mla_absorb_q", "pliippii", ptr(qo), qo.stride(0), 192, 128, ptr(L.w_uk), ptr(qa), n, H)
            op, lp, _ = other.mla_ws
            call("mla_decode", "pppppppipliiifp", ptr(qa), ptr(ol), ptr(op), ptr(lp), ptr(b.pos), ptr(b.slot), ptr(kvo.page_table), kvo.page_table.shape[1], ptr(pool),
                 pool.shape[0], n, H, 32, 192 ** -0.5, ptr(K.status_word(dev)))
            att = torch.empty(n, H * 128, dtype=bf, device=dev)
            call("mla_expand_out", "pppliii", ptr(ol), ptr(L.w_uv), ptr(att), att.stride(0), n, H, 128)
        kb.add(f"latent attention {kind}", "glm5 assembly", theirs, kb_bytes, flops)
        # norms, activations, linears
        h, x = torch.randn(n, width, device=dev), torch.randn(n, width, device=dev).to(bf)
        ly = mine.layers[0]
        if n > 1:
            kb.add("add + norm prompt", "fofosun (fp32 residual)", lambda: ly.norm1.rows(h, bf, x, ly.write1), n * width * 12, 0)
            hb = h.to(bf)
            kb.add("add + norm prompt", "glm5 assembly", lambda: K.rmsnorm(x, L.attn_norm, 1e-5, 1.0, residual=hb), n * width * 8, 0)
            z = torch.randn(n, width * 6, device=dev).to(bf)
            gu = torch.randn(n, width * 8, device=dev).to(bf)
            kb.add("activation prompt", "polynorm", lambda: ly.ff.act.rows(z, bf), 2 * z.numel() * 2, 0)
            kb.add("activation prompt", "glm5 assembly", lambda: K.gated_act(gu, width * 4), gu.numel() * 3, 0)
            orow = torch.randn(n, D, device=dev)
            kb.add("output norm prompt", "hgrn2", lambda: mine.layers[0].mixer.norm.rows(orow, bf), n * D * 6, 0)
            zz = torch.randn(n, D, device=dev).to(bf)
            ob, nw = torch.empty(n, D, device=dev, dtype=bf), torch.ones(128, device=dev)
            kb.add("output norm prompt", "kda", lambda: call("kda_gated_norm", "pplppiiif", ptr(orow), ptr(zz), zz.stride(0), ptr(nw), ptr(ob), n, H, 128, 1e-5), n * D * 8, 0)
            for lin, nm in ((ly.ff.up, "up"), (ly.mixer.out, "out")):
                xi = torch.randn(n, lin.in_features, device=dev).to(bf)
                kb.add(f"linear prompt ({nm})", "shared kernel", lambda: lin.forward(xi), lin.nbytes() + n * (lin.in_features + lin.out_features) * 2,
                       2.0 * n * lin.in_features * lin.out_features)
        else:
            z = torch.randn(1, width * 6, device=dev)
            kb.add("linear decode: norm + up", "fofosun", lambda: gemv_rows(ly.ff.up, 1, out_f32=True, **ly.norm2.prologue(h)), ly.ff.up.nbytes(), 0)
            kb.add("linear decode: activation + down + add", "fofosun", lambda: gemv_rows(ly.ff.down, 1, residual=(h, ly.write2), **ly.ff.act.prologue(z)), ly.ff.down.nbytes(), 0)
            kb.add("linear decode: in projection", "fofosun", lambda: gemv_rows(ly.mixer.in_proj, 1, out_f32=True, **ly.norm1.prologue(h)), ly.mixer.in_proj.nbytes(), 0)
            gul = other.layers[0].gate_up
            kb.add("linear decode: gate and up", "glm5 assembly (bf16)", lambda: gul.forward(x), gul.nbytes(), 0)
            dn, xa = other.layers[0].down, torch.randn(1, width * 4, device=dev).to(bf)
            kb.add("linear decode: down", "glm5 assembly (bf16)", lambda: dn.forward(xa), dn.nbytes(), 0)
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
        for which in ("fofosun", "closest"):
            models.append(run_model(which, w, layers, dev, plen, args.steps, max(3, args.warmup), min(args.prefill_chunk, 2048)))
            torch.cuda.empty_cache()
    kernels = run_kernels(2048, dev)
    clocks = sampler.stop()
    head = next(m for m in models if m["model"] == "fofosun" and m["width"] == 2048)
    print(json.dumps({"metric": "decode_tok_s_1stream", "value": head["decode_1"]["tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": args.steps,
                      "warmup": max(3, args.warmup), "ms_per_step": head["decode_1"]["ms_per_step"], "higher_is_better": True, "scaling": "strong",
                      "vs_baseline": None, "dtype": "bf16", "data": "synthetic (random token ids, random bf16 weights)",
                      "config": {"model": f"Fofosun, width 2048, {layers} layers", "seq_len": plen, "global_batch": 1, "parallelism": "tp1",
                                 "l2": "decode: weights per step larger than L2; kernels: L2 flushed between iterations"},
                      "models": models, "kernels": kernels, "clocks": clocks, "device_status": K.check_status(dev)}))
    return 0
