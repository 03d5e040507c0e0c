"""Every mechanism of the Fofosun decoder alone against the plain statement: element-wise norms, grouped RMS norms, PolyNorm,
the fused decode linears, the two recurrences, latent attention. Inputs are made so that a lost state, a missing key or a
wrong rotation shows."""
import pytest
import torch

import fofosun_plain as plain
from fofosun_util import DEVICES, one_thread  # noqa: F401
from volta_engine_b200.ops.latent import LatentSpec, latent_rows
from volta_engine_b200.ops.linear import LinearBF16
from volta_engine_b200.ops.linear_attn import LinAttnSpec, LinAttnState, linattn_rows
from volta_engine_b200.ops.rowops import DynamicTanh, GroupRMS, PolyNorm, embed_rows, gemv_rows
from volta_engine_b200.runtime.batch import BatchRows
from volta_engine_b200.runtime.kv_cache import PagedKVCache

TYPES = [torch.float32, torch.bfloat16]


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def close(got, want, dtype, f32=2e-6, bf16=2 ** -8):
    w = want.double()
    tol = f32 if dtype == torch.float32 else bf16
    assert got.shape == w.shape and bool(((got.double().cpu() - w).abs() <= tol * (w.abs() + w.pow(2).mean().sqrt())).all())


# ------------------------------------------------------------------------------------------ row operators
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows,width", [(1, 64), (5, 75), (3, 2052), (200, 132), (33, 8)])
def test_dynamic_tanh_with_the_pending_sum(rows, width, dtype, device):
    h, w, b = rnd(rows, width, seed=1, scale=3), rnd(width, seed=2), rnd(width, seed=3)
    part, scale = rnd(rows, width, seed=4).to(dtype), rnd(width, seed=5)
    n = DynamicTanh(w.to(device), b.to(device), 0.83)
    hd = h.clone().to(device)
    close(n.rows(hd, dtype), plain.dyt_norm(h.double(), w.double(), b.double(), 0.83), dtype)
    assert torch.equal(hd.cpu(), h)
    got = n.rows(hd, dtype, part.to(device), scale.to(device))
    summed = h.double() + part.double() * scale.double()
    close(hd, summed, torch.float32)
    close(got, plain.dyt_norm(summed, w.double(), b.double(), 0.83), dtype)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("groups,size,gated", [(1, 72, False), (6, 20, False), (3, 130, True), (1, 1500, True), (16, 128, False)])
def test_grouped_rms_norm(groups, size, gated, dtype, device):
    cols = groups * size
    x, g = rnd(5, cols, seed=1, scale=0.01), rnd(5, cols, seed=2, scale=4)       # small rows: the place of eps matters
    w = rnd(size if not gated else cols, seed=3)
    norm = GroupRMS(w.to(device), 3e-4, size if groups > 1 else 0)
    want = plain.unit_rms(x.double().reshape(5, groups, size), 3e-4).reshape(5, cols) * w.double().repeat(cols // w.numel())
    if gated:
        want = want * plain.sigmoid(g.double())
    close(norm.rows(x.to(device), dtype, gate=g.to(device) if gated else None), want, dtype)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows,ff", [(1, 53), (7, 320), (2, 2056), (3, 9000)])
def test_polynorm(rows, ff, dtype, device):
    z = rnd(rows, ff, seed=6, scale=0.3).to(dtype)
    coef = torch.tensor([0.7, -0.4, 0.25, 0.1])
    want = plain.poly_norm(z.double(), coef.double(), 1e-3)
    close(PolyNorm(coef.to(device), 1e-3).rows(z.to(device), dtype), want, dtype, f32=5e-6)


@pytest.mark.parametrize("device", DEVICES)
def test_embedding_rows(device):
    for dtype in TYPES:
        t = rnd(30, 75, seed=1).to(dtype)
        ids = torch.tensor([29, 0, 7, 7], dtype=torch.int32)
        assert torch.equal(embed_rows(ids.to(device), t.to(device)).cpu(), t[ids.long()].float())


@pytest.mark.gpu
@pytest.mark.parametrize("N,K,M", [(96, 64, 1), (1000, 2048, 1), (130, 75, 3), (2056, 1000, 8), (6000, 264, 5), (20000, 520, 2), (75, 4104, 4), (264, 8192, 1)])
def test_decode_linear_with_prologues(N, K, M):
    """y = W f(x) with every prologue and epilogue, against 64-bit."""
    dev = "cuda"
    W = (rnd(N, K, seed=1) * K ** -0.5).to(torch.bfloat16)
    lin = LinearBF16(W.to(dev))
    x, w, b = rnd(M, K, seed=2), rnd(K, seed=3), rnd(K, seed=4)
    Wd = W.double()

    def want(v):
        return v.to(torch.bfloat16).double() @ Wd.t()

    def check(got, v, tol=6e-3):
        e = want(v)
        assert (got.double().cpu() - e).abs().max() < tol * e.pow(2).mean().sqrt() + 1e-6
    dyt = DynamicTanh(w.to(dev), b.to(dev), 0.9)
    check(gemv_rows(lin, M, out_f32=True, **dyt.prologue(x.to(dev))), plain.dyt_norm(x.double(), w.double(), b.double(), 0.9).float())
    h = rnd(M, N, seed=7).to(dev)
    h0, ls = h.clone(), 1 + rnd(N, seed=8).abs()
    G = next(g for g in (8, 5, 3, 25, 1) if K % g == 0)
    gate = rnd(M, K, seed=9)
    rms = GroupRMS(w[:G].contiguous().to(dev), 1e-4, G)
    v = (plain.unit_rms(x.double().reshape(M, K // G, G), 1e-4).reshape(M, K) * w[:G].double().repeat(K // G) * plain.sigmoid(gate.double())).float()
    gemv_rows(lin, M, residual=(h, ls.to(dev)), **rms.prologue(x.to(dev), gate.to(dev)))
    check((h - h0) / ls.to(dev), v, tol=3e-2)
    whole = GroupRMS(w.to(dev), 1e-4)
    check(gemv_rows(lin, M, out_f32=True, **whole.prologue(x.to(dev))), plain.rms_norm(x.double(), w.double(), 1e-4).float())
    poly = PolyNorm(torch.tensor([0.5, 0.3, -0.2, 0.1]).to(dev), 1e-4)
    check(gemv_rows(lin, M, **poly.prologue(x.to(dev))).float(), plain.poly_norm(x.double(), torch.tensor([0.5, 0.3, -0.2, 0.1]).double(), 1e-4).float(), tol=3e-2)
    if K % 8 == 0:
        for m in (M, 16):
            xb = rnd(m, K, seed=5).to(torch.bfloat16)
            e = xb.double() @ Wd.t()
            assert (gemv_rows(lin, m, x=xb.to(dev), out_f32=True).double().cpu() - e).abs().max() < 1e-4 * e.abs().max()


@pytest.mark.gpu
def test_linears_of_widths_that_are_not_multiples_of_the_tile():
    from volta_engine_b200.ops.kernels import gemm_f32
    for T, N, K in ((40, 130, 80), (70, 75, 75), (17, 328, 104), (130, 64, 33)):
        W, x = rnd(N, K, seed=1), rnd(T, K, seed=2)
        e = x.double() @ W.double().t()
        assert (gemm_f32(W.cuda(), x.cuda()).double().cpu() - e).abs().max() < 1e-5 * e.abs().max()
        Wb, xb = W.to(torch.bfloat16), x.to(torch.bfloat16)
        e = xb.double() @ Wb.double().t()
        got = LinearBF16(Wb.cuda()).forward(xb.cuda(), out_f32=True)
        assert (got.double().cpu() - e).abs().max() < 1e-5 * e.abs().max()


@pytest.mark.gpu
@pytest.mark.parametrize("T,N,K", [(130, 256, 64), (257, 300, 104), (520, 1000, 33), (129, 5, 712), (300, 513, 256)])
def test_wide_gemm_at_the_edges_of_its_tiles(T, N, K):
    from volta_engine_b200._lib import call, ptr
    from volta_engine_b200.ops.kernels import status_word
    Kp = -(-K // 8) * 8
    W, x = torch.zeros(N, Kp, dtype=torch.bfloat16), torch.zeros(T, Kp, dtype=torch.bfloat16)
    W[:, :K], x[:, :K] = rnd(N, K, seed=1).to(torch.bfloat16), rnd(T, K, seed=2).to(torch.bfloat16)
    res = rnd(T, N, seed=3).to(torch.bfloat16)
    e = x.double() @ W.double().t()
    bias = rnd(N, seed=4)
    Wd, xd, rd, bd = W.cuda(), x.cuda(), res.cuda(), bias.cuda()
    for f32, biased in ((True, False), (False, False), (True, True), (False, True)):
        out = torch.full((T + 1, N), 9.0, dtype=torch.float32 if f32 else torch.bfloat16, device="cuda")
        call("gemm_bf16_wide", "plplplppliiifpp", ptr(Wd), Kp, ptr(xd), Kp, 0 if f32 else ptr(out), N, ptr(out) if f32 else 0, 0 if f32 else ptr(rd), N, T, N, Kp,
             1.0, ptr(bd) if biased else 0, ptr(status_word(Wd.device)))
        want = e if f32 else e + res.double()
        if biased:
            want = want + bias.double()
        assert (out[:T].double().cpu() - want).abs().max() < (1e-5 if f32 else 6e-3) * want.abs().max()
        assert bool((out[T] == 9.0).all())


# ------------------------------------------------------------------------------------------ recurrences
def lin_case(mode, H, dk, dv, seed=0):
    if mode == "lightning":
        return LinAttnSpec(H, dk, dv, decay=torch.linspace(0.5, 1.0, H) if H > 1 else torch.tensor([0.97]))
    low = torch.rand(H * dk, generator=torch.Generator().manual_seed(seed))
    low[::3] = 0.999                              # channels that hardly forget
    low[1::3] = 0.0                               # channels that can forget everything at once
    return LinAttnSpec(H, dk, dv, lower=low, bias=rnd(H * dk, seed=seed + 1, scale=2))


def lin_plain(spec, proj):
    """Rows of the raw projection through the plain recurrence, one step at a time."""
    p, H, dk, dv = proj.double(), spec.heads, spec.dk, spec.dv
    T = p.shape[0]
    q = plain.silu(p[:, :H * dk]).reshape(T, H, dk)
    x, v = p[:, H * dk:2 * H * dk], p[:, 2 * H * dk:2 * H * dk + H * dv].reshape(T, H, dv)
    if spec.decay is not None:
        f = spec.decay.double().reshape(1, H, 1).expand(T, H, dk)
        k, v = plain.silu(x).reshape(T, H, dk), plain.silu(v)
    else:
        low = spec.lower.double()
        f = (low + (1 - low) * plain.sigmoid(x + spec.bias.double())).reshape(T, H, dk)
        k = 1 - f
    S, out = torch.zeros(H, dk, dv, dtype=torch.float64), []
    for t in range(T):
        S = f[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]).reshape(-1))
    return torch.stack(out), S


def on(spec, device):
    move = lambda t: None if t is None else t.to(device)
    return LinAttnSpec(spec.heads, spec.dk, spec.dv, move(spec.decay), move(spec.lower), move(spec.bias))


LIN = [("hgrn2", 2, 32, 32), ("hgrn2", 3, 24, 40), ("hgrn2", 1, 128, 128), ("hgrn2", 2, 13, 7), ("hgrn2", 2, 64, 96), ("hgrn2", 1, 200, 33),
       ("lightning", 4, 64, 64), ("lightning", 1, 16, 48), ("lightning", 3, 128, 80), ("lightning", 2, 9, 21), ("lightning", 2, 96, 128)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("form", ["fp32", "bf16 rows", "chunked"])
@pytest.mark.parametrize("mode,H,dk,dv", LIN)
def test_recurrence_in_portions(mode, H, dk, dv, form, device):
    """One long sequence in portions of all kinds beside a second one, in slots that hold another sequence's state before."""
    dtype = torch.bfloat16 if form == "bf16 rows" else torch.float32
    base = lin_case(mode, H, dk, dv)
    spec = on(base, device)
    st = LinAttnState(spec, 3, device)
    st.rec.fill_(7.0)                             # what an earlier request left behind
    cols = spec.cols + 5
    a, b = rnd(330, cols, seed=3, scale=1.5).to(dtype), rnd(90, cols, seed=4, scale=1.5).to(dtype)
    a[:, H * dk:2 * H * dk] *= 2
    a[37, H * dk:2 * H * dk] = -60.0              # everything forgettable is forgotten at this row
    wa, Sa = lin_plain(base, a)
    wb, _ = lin_plain(base, b)
    got_a, got_b, at, bt = [], [], 0, 0
    for na, nb in ((1, 0), (64, 1), (2, 0), (100, 40), (63, 3), (17, 16), (1, 1), (16, 0), (65, 29), (1, 0)):
        ids = list(range(at, at + na)) + list(range(bt, bt + nb))
        batch = BatchRows.make(ids, ids, [2] * na + [0] * nb, device)
        proj = torch.cat([a[at:at + na], b[bt:bt + nb]]).to(device)
        o = linattn_rows(proj, batch, st, spec, chunked=form == "chunked")
        got_a.append(o[:na].cpu())
        got_b.append(o[na:].cpu())
        at, bt = at + na, bt + nb
    for got, want in ((torch.cat(got_a), wa), (torch.cat(got_b), wb)):
        ref = want.pow(2).mean().sqrt()
        tol = 3e-3 if form == "chunked" else 3e-5            # the chunked form rounds the values to bf16
        assert (got.double() - want).abs().max() < tol * (want.abs().max() + ref)
    assert (st.rec[2].double().cpu() - Sa).abs().max() < tol * Sa.abs().max()
    assert bool((st.rec[1] == 7.0).all())         # the slot nobody used


# ------------------------------------------------------------------------------------------ latent attention
def latent_case(H, d, rot, dv, kr, seed=0, base=500.0, scale=None):
    spec = LatentSpec(H, d, rot, dv, kr, scale or (d + rot) ** -0.5, base, 1e-5)
    w = {"uk": (rnd(H * d, kr, seed=seed) * kr ** -0.5).to(torch.bfloat16), "uv": (rnd(H * dv, kr, seed=seed + 1) * kr ** -0.5).to(torch.bfloat16),
         "norm": 1 + rnd(kr, seed=seed + 2, scale=0.2)}
    return spec, w


def latent_plain(spec, w, q, kv):
    """q [T, H (d + rot)], kv [T, kr + rot] as projected -> [T, H dv]."""
    H, d, r, dv, kr = spec.heads, spec.dim, spec.rot, spec.vdim, spec.kv_rank
    T = q.shape[0]
    q, kv = q.double().reshape(T, H, d + r), kv.double()
    c = plain.rms_norm(kv[:, :kr], w["norm"].double(), spec.eps)
    k = (c @ w["uk"].double().t()).reshape(T, H, d)
    v = (c @ w["uv"].double().t()).reshape(T, H, dv)
    qr = torch.stack([plain.rotate_pairs(q[t, :, d:], t, spec.theta, r) for t in range(T)])
    kr_ = torch.stack([plain.rotate_pairs(kv[t, kr:], t, spec.theta, r) for t in range(T)])
    out, weights = torch.zeros(T, H, dv, dtype=torch.float64), []
    for t in range(T):
        s = (torch.einsum("hd,jhd->hj", q[t, :, :d], k[:t + 1]) + torch.einsum("hd,jd->hj", qr[t], kr_[:t + 1])) * spec.scale
        p = torch.softmax(s, -1)
        weights.append(p)
        out[t] = torch.einsum("hj,jhv->hv", p, v[:t + 1])
    return out.reshape(T, H * dv), weights


class LatentRun:
    """A paged cache and one sequence's rows through the operator, in portions."""

    def __init__(self, spec, w, dtype, device, slots=3, pages=20, pitch=0, layers=2):
        self.spec, self.dtype, self.device = spec.bind(device), dtype, device
        width = max(pitch, spec.width)
        self.kv = PagedKVCache(layers, 1, width, pages, slots, 640, torch.device(device), dtype=dtype, v_head_dim=8)
        self.kv.k.fill_(3.0)                       # rows of earlier requests
        t = dtype if dtype == torch.float32 else torch.bfloat16
        self.uk, self.uv, self.norm = w["uk"].to(device, t), w["uv"].to(device, t), w["norm"].to(device)
        self.ukv = LinearBF16(torch.cat([self.uk, self.uv], 0)) if t == torch.bfloat16 else None

    def rows(self, parts):
        """parts: [(slot, first position, q, kv)] one batch, shortest first -> the rows' outputs."""
        ids, pos, slots = [], [], []
        for s, p0, q, _ in parts:
            self.kv.reserve(s, p0 + q.shape[0])
            pos += range(p0, p0 + q.shape[0])
            slots += [s] * q.shape[0]
        b = BatchRows.make(pos, pos, slots, self.device, nsplit=5)
        q, kv = torch.cat([p[2] for p in parts]), torch.cat([p[3] for p in parts])
        qd = q.to(self.device, torch.float32 if b.row_path or self.dtype == torch.float32 else torch.bfloat16)
        return latent_rows(self.spec, qd.contiguous(), kv.to(self.device), self.norm, self.uk, self.uv, self.ukv, b, self.kv, self.kv.k[1]).float().cpu()


LAT = [(3, 40, 8, 24, 72), (2, 21, 6, 18, 50), (2, 128, 64, 128, 512), (17, 40, 24, 16, 64), (1, 64, 32, 72, 136), (2, 24, 16, 40, 544), (2, 192, 64, 256, 256),
       (1, 100, 24, 64, 320)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,d,rot,dv,kr", LAT)
def test_latent_attention_in_portions(H, d, rot, dv, kr, dtype, device):
    """Every row's query is lined up with one key of its past (page borders, the first token, itself, the row before), so the
    row's output is almost that key's value: a missing, shifted or wrongly rotated key changes it at once."""
    spec, w = latent_case(H, d, rot, dv, kr, seed=H)
    T = 210
    kv = rnd(T, kr + rot, seed=5).to(torch.bfloat16).float()
    pick = [max(0, min(t, [0, t, t - 1, 63, 64, 127, 128, t // 2, 1][t % 9])) for t in range(T)]
    c = plain.rms_norm(kv[:, :kr].double(), w["norm"].double(), spec.eps)
    k = (c @ w["uk"].double().t()).reshape(T, H, d)
    q = torch.zeros(T, H, d + rot, dtype=torch.float64)
    for t in range(T):
        j = pick[t]
        kr_ = plain.rotate_pairs(kv[j, kr:].double(), j - t, spec.theta, rot)      # the score sees the difference of positions
        q[t] = torch.cat([k[j], kr_.expand(H, rot)], -1)
        q[t] *= 24.0 / spec.scale / (q[t] * q[t]).sum(-1, keepdim=True)            # score 24 for the key picked
    q = q.reshape(T, -1).float().to(torch.bfloat16).float()
    want, weights = latent_plain(spec, w, q, kv)
    assert min(p[:, pick[t]].min().item() for t, p in enumerate(weights)) > 0.5
    tol = 2e-5 if dtype == torch.float32 else 0.03
    for n, cuts in enumerate(([T], [64, 64, 82], [1] * 10 + [60, 16, 2, 41, 1, 1, 15, 17] + [1] * 47, [130] + [2] * 40)):
        if device == "cpu" and n % 2:
            continue
        r = LatentRun(spec, w, dtype, device, pitch=spec.width + 64 * (n % 2))
        at, got = 0, []
        for cnt in cuts:
            got.append(r.rows([(1, at, q[at:at + cnt], kv[at:at + cnt])]))
            at += cnt
        got = torch.cat(got)[:at]
        assert (got.double() - want[:at]).abs().max() < tol * want.abs().max(), (n, cuts)


@pytest.mark.gpu
@pytest.mark.parametrize("H,d,rot,dv,kr", [c for c in LAT if c[1] % 8 == 0])
def test_latent_attention_on_the_mma_kernel(H, d, rot, dv, kr, monkeypatch):
    from volta_engine_b200.ops import latent as L
    monkeypatch.setattr(L, "TC_PREFILL", False)
    test_latent_attention_in_portions(H, d, rot, dv, kr, torch.bfloat16, "cuda")


@pytest.mark.gpu
def test_latent_prompt_of_many_key_tiles():
    """Both streams, moving references and several query tiles: scores grow along the sequence, then fall."""
    spec, w = latent_case(2, 64, 32, 96, 64, seed=3)
    T = 600
    kv = rnd(T, 96, seed=5).to(torch.bfloat16).float()
    q = (rnd(T, 2 * 96, seed=6) * torch.linspace(0.2, 3, T)[:, None]).to(torch.bfloat16).float()
    kv[:, 64:] *= torch.cat([torch.linspace(0.1, 2.5, T // 2), torch.linspace(2.5, 0.1, T - T // 2)])[:, None]
    kv = kv.to(torch.bfloat16).float()
    want, _ = latent_plain(spec, w, q, kv)
    for cuts in ([T], [1, 399, 200], [129, 127, 344]):
        r, at, got = LatentRun(spec, w, torch.bfloat16, "cuda"), 0, []
        for cnt in cuts:
            got.append(r.rows([(2, at, q[at:at + cnt], kv[at:at + cnt])]))
            at += cnt
        err = ((torch.cat(got).double() - want).abs().max() / want.abs().max()).item()
        assert err < 0.03, err


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
def test_latent_attention_of_a_mixed_batch(dtype, device):
    spec, w = latent_case(3, 40, 8, 24, 72, seed=9)
    r = LatentRun(spec, w, dtype, device)
    seq = [(rnd(140, 3 * 48, seed=s).to(torch.bfloat16).float() * 3, rnd(140, 80, seed=s + 10).to(torch.bfloat16).float()) for s in range(3)]
    want = [latent_plain(spec, w, *s)[0] for s in seq]
    at = [0, 0, 0]
    for counts in ((1, 5, 100), (2, 3, 20), (1, 1, 1), (16, 40, 3), (0, 80, 1), (0, 1, 1)):
        order = sorted((i for i in range(3) if counts[i]), key=lambda i: counts[i])
        got = r.rows([(i, at[i], seq[i][0][at[i]:at[i] + counts[i]], seq[i][1][at[i]:at[i] + counts[i]]) for i in order])
        exp = torch.cat([want[i][at[i]:at[i] + counts[i]] for i in order])
        assert (got.double() - exp).abs().max() < (2e-5 if dtype == torch.float32 else 0.03) * exp.abs().max()
        for i in range(3):
            at[i] += counts[i]


@pytest.mark.parametrize("device", DEVICES)
def test_rotation_is_exact_at_far_positions(device):
    """Scores depend on the difference of positions only, also a long way from the start."""
    spec, w = latent_case(1, 8, 8, 8, 16, base=1.5, scale=1.0)
    r = LatentRun(spec, w, torch.float32, device, slots=2, pages=9)
    kv, q = rnd(6, 24, seed=1), rnd(6, 16, seed=2)
    near = r.rows([(0, 0, q, kv)])
    far = torch.zeros_like(near)
    base = 500_000
    spec.bind(device)
    r.kv.page_table = torch.zeros(2, base // 64 + 2, dtype=torch.int32, device=device)
    r.kv.page_table[1, base // 64:] = 7                            # only the last page is looked at: the keys before it must not count
    r.kv.k[1, 0].zero_()
    r.kv.k[1, 0, :, :, :16] = 0
    if device == "cpu":
        at = torch.arange(6)
        s0 = spec.turn.turn(q[:, 8:], at) @ spec.turn.turn(kv[:, 16:], at).t()
        s1 = spec.turn.turn(q[:, 8:], at + base) @ spec.turn.turn(kv[:, 16:], at + base).t()
        assert (s0 - s1).abs().max() < 1e-5
        return
    from volta_engine_b200._lib import call, ptr
    D = spec.dims(r.kv.k[1])
    qs = []
    for p0 in (0, base):
        pos = (torch.arange(6) + p0).int().cuda()
        slot = torch.full((6,), 1, dtype=torch.int32, device="cuda")
        qo, kvd = torch.empty(6, 16, device="cuda"), kv.cuda()
        qd = q.cuda()
        call("latent_rope_store", "iiiiiiii" + "plplplii" + "ppf" + "pppip" + "ifi", *D, ptr(qd), 16, ptr(qo), 16, ptr(kvd), 24, 1, 1, ptr(r.norm),
             ptr(spec.turn.half_turns), 1.0, ptr(pos), ptr(slot), ptr(r.kv.page_table), r.kv.page_table.shape[1], ptr(r.kv.k[1]), 6, 1e-5, 1)
        page = 7 if p0 else 0
        off = p0 % 64
        qs.append(qo[:, 8:].cpu() @ r.kv.k[1, page, 0, off:off + 6, 16:24].cpu().t())
    assert (qs[0] - qs[1]).abs().max() < 1e-5
    assert near.shape == far.shape


@pytest.mark.gpu
@pytest.mark.parametrize("mode,H,dk,dv", [("hgrn2", 2, 128, 128), ("lightning", 3, 64, 32), ("hgrn2", 5, 24, 40)])
def test_chunked_recurrence_of_a_large_batch(mode, H, dk, dv):
    """Several sequences, portions longer than many chunks, values that are exact in bf16: then everything else of the chunked
    form keeps 32-bit quality."""
    base = lin_case(mode, H, dk, dv, seed=5)
    spec = on(base, "cuda")
    if mode == "lightning":
        base.decay = base.decay.clone()
    st = LinAttnState(spec, 4, "cuda")
    lens = [700, 16, 433, 17]
    rows = []
    for i, n in enumerate(lens):
        r = rnd(n, spec.cols, seed=30 + i, scale=1.5)
        v = r[:, 2 * H * dk:2 * H * dk + H * dv]
        v.copy_(v.to(torch.bfloat16))
        rows.append(r)
    want = [lin_plain(base, r) for r in rows]
    cut = [300, 0, 150, 0]
    for part in (0, 1):
        segs = [(i, 0 if part == 0 else cut[i], cut[i] if part == 0 else lens[i]) for i in range(4)]
        segs = [s for s in segs if s[2] > s[1]]
        pos = [p for i, a, b in segs for p in range(a, b)]
        slot = [3 - i for i, a, b in segs for _ in range(a, b)]
        batch = BatchRows.make(pos, pos, slot, "cuda")
        o = linattn_rows(torch.cat([rows[i][a:b] for i, a, b in segs]).cuda(), batch, st, spec).double().cpu()
        at = 0
        for i, a, b in segs:
            w = want[i][0]
            assert (o[at:at + b - a] - w[a:b]).abs().max() < (3e-3 if mode == "lightning" else 6e-5) * w.abs().max()
            at += b - a
    for i in range(4):
        S = want[i][1]
        assert (st.rec[3 - i].double().cpu() - S).abs().max() < (3e-3 if mode == "lightning" else 6e-5) * S.abs().max()
