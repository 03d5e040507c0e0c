"""Every mechanism of the Siditar decoder alone against the plain statement: position vectors, layer norm over read streams, stream
updates, the clamped gated unit, gated output norms, the decode linears that carry them, attention with its distance bias, sink and
temperature, gated linear attention. Inputs are made so that a missing key, a bucket one token off, a lost state or a sink that is
left out shows."""
import math

import pytest
import torch

import siditar_plain as plain
from listed_util import DEVICES, one_thread  # noqa: F401
from volta_engine_b200.ops.gqa import GqaSpec, distance_bias, gqa_attend
from volta_engine_b200.ops.linear import LinearBF16
from volta_engine_b200.ops.linear_attn import LinAttnSpec, LinAttnState, linattn_rows
from volta_engine_b200.ops.rowops import ClampedGlu, GroupRMS, SinusoidalPositions, StreamNorm, StreamWrite, embed_rows, gemv_rows
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
@pytest.mark.parametrize("width", [8, 75, 132])
def test_embedding_with_position_vectors(width, device):
    pos = torch.tensor([0, 1, 2, 63, 64, 1000, 131071, 1_000_003], dtype=torch.int32)
    ids = torch.tensor([3, 0, 29, 7, 7, 1, 2, 29], dtype=torch.int32)
    want = torch.stack([plain.position_vector(int(p), width) for p in pos])
    sp = SinusoidalPositions(width, 10000.0, device)
    for dtype in TYPES:
        t = rnd(30, width, seed=1).to(dtype)
        for streams in (1, 3):
            got = embed_rows(ids.to(device), t.to(device), pos.to(device), sp, streams).cpu()
            assert got.shape == (8, streams, width)
            for s in range(streams):
                assert (got[:, s].double() - t[ids.long()].double() - want).abs().max() < 1e-6


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows,streams,width", [(1, 1, 64), (5, 3, 75), (3, 2, 2052), (40, 2, 132), (2, 5, 100), (7, 8, 24), (2, 4, 4096), (3, 2, 8200)])
def test_streams_written_read_and_normed(rows, streams, width, dtype, device):
    h = rnd(rows, streams, width, seed=1) + 3.0                      # a mean that the variance must not contain
    w, read = rnd(width, seed=2), rnd(streams, seed=3)
    mix, out, part = rnd(streams, streams, seed=4), rnd(streams, seed=5), rnd(rows, width, seed=6, scale=2).to(dtype)
    n, wr = StreamNorm(w.to(device), 3e-4, read.to(device)), StreamWrite(mix.to(device), out.to(device))
    hd = h.clone().to(device)
    x = h.double().transpose(0, 1)
    close(n.rows(hd, dtype), plain.layer_norm(plain.read_streams(x, read.double()), w.double(), 3e-4), dtype, f32=2e-5)
    assert torch.equal(hd.cpu(), h)
    got = n.rows(hd, dtype, part.to(device), wr)
    x = plain.write_streams(x, mix.double(), out.double(), part.double())
    close(hd, x.transpose(0, 1), torch.float32)
    close(got, plain.layer_norm(plain.read_streams(x, read.double()), w.double(), 3e-4), dtype, f32=2e-5)


@pytest.mark.parametrize("device", DEVICES)
def test_layer_norm_of_small_rows_sees_eps_inside_the_root(device):
    h, w = rnd(4, 1, 96, seed=1, scale=1e-3), rnd(96, seed=2)
    got = StreamNorm(w.to(device), 1e-6, torch.ones(1, device=device)).rows(h.to(device), torch.float32)
    close(got, plain.layer_norm(h.double()[:, 0], w.double(), 1e-6), torch.float32, f32=1e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows,ff", [(1, 53), (7, 320), (30, 264)])
@pytest.mark.parametrize("limit", [0.3, 1.0, 7.0])
def test_clamped_gated_unit(rows, ff, limit, dtype, device):
    z = rnd(rows, 2 * ff, seed=6, scale=2).to(dtype)
    z[0, 0], z[0, ff] = -50.0, -50.0                                 # the gate has no lower bound, the other half has
    eye = torch.eye(ff, dtype=torch.float64)
    pick = {"gate": torch.cat([eye, 0 * eye], 1), "up": torch.cat([0 * eye, eye], 1), "down": eye}
    want = plain.clamped_ff(pick, "", {"limit": limit}, z.double())
    close(ClampedGlu(limit, 1.702).rows(z.to(device), dtype), want, dtype, f32=5e-6)
    if ff % 4 == 0:                                                  # the same with the halves in blocks, as a weight in blocks makes them
        zb = (z.float() @ ClampedGlu.interleave(pick["gate"].float(), pick["up"].float()).t()).to(dtype)
        assert not torch.equal(zb, z)
        close(ClampedGlu(limit, 1.702, True).rows(zb.to(device), dtype), want, dtype, f32=5e-6)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("groups,size", [(6, 20), (3, 130), (2, 9), (5, 512), (16, 128), (1, 1500)])
def test_output_norm_with_a_silu_gate_into_a_part_of_a_row(groups, size, dtype, device):
    cols = groups * size
    x, g, w = rnd(5, cols, seed=1, scale=0.01), rnd(5, cols + 3, seed=2, scale=4)[:, :cols], rnd(size, seed=3)
    want = plain.rms_norm(x.double().reshape(5, groups, size), w.double(), 3e-4).reshape(5, cols) * plain.silu(g.double())
    y = torch.full((5, cols + 16), 9.0, dtype=dtype, device=device)
    got = GroupRMS(w.to(device), 3e-4, size, silu=True).rows(x.to(device), dtype, gate=g.to(device), out=y[:, 16:])
    close(got, want, dtype, f32=5e-6)
    assert got.data_ptr() == y[:, 16:].data_ptr() and bool((y[:, :16] == 9.0).all())


@pytest.mark.gpu
@pytest.mark.parametrize("N,K,M", [(96, 64, 1), (1000, 2048, 1), (130, 75, 3), (2056, 1000, 8), (6000, 264, 5), (75, 4104, 4)])
def test_decode_linear_with_prologues(N, K, M):
    """y = W f(x) with stream norm, clamped unit, gated norm behind plain columns; streams rewritten in the epilogue."""
    dev = "cuda"
    W = (rnd(N, K, seed=1) * K ** -0.5).to(torch.bfloat16)
    lin, Wd = LinearBF16(W.to(dev)), W.double()

    def check(got, v, tol=6e-3):
        e = v.float().to(torch.bfloat16).double() @ Wd.t()
        assert (got.double().cpu() - e).abs().max() < tol * e.pow(2).mean().sqrt() + 1e-6
        return e
    for S in (1, 2, 5):
        h, w, read = rnd(M, S, K, seed=2) + 2.0, rnd(K, seed=3), rnd(S, seed=4)
        n = StreamNorm(w.to(dev), 1e-5, read.to(dev))
        v = plain.layer_norm(plain.read_streams(h.double().transpose(0, 1), read.double()), w.double(), 1e-5)
        check(gemv_rows(lin, M, out_f32=True, **n.prologue(h.to(dev))), v, 1e-2)
        z = rnd(M, 2 * K, seed=5, scale=2)
        eye = torch.eye(K, dtype=torch.float64)
        v = plain.clamped_ff({"gate": torch.cat([eye, 0 * eye], 1), "up": torch.cat([0 * eye, eye], 1), "down": eye}, "", {"limit": 0.8}, z.double())
        hs = rnd(M, S, N, seed=6)
        mix, out = rnd(S, S, seed=7), 1 + rnd(S, seed=8).abs()
        hd = hs.clone().to(dev)
        gemv_rows(lin, M, residual=(hd, StreamWrite(mix.to(dev), out.to(dev))), **ClampedGlu(0.8, 1.702).prologue(z.to(dev)))
        y = v.float().to(torch.bfloat16).double() @ Wd.t()
        want = plain.write_streams(hs.double().transpose(0, 1), mix.double(), out.double(), y).transpose(0, 1)
        assert (hd.double().cpu() - want).abs().max() < 1e-2 * want.pow(2).mean().sqrt()
    if N % 16 == 0:                                                   # the gated unit as the epilogue
        x, w = rnd(M, 1, K, seed=13), rnd(K, seed=14)
        n = StreamNorm(w.to(dev), 1e-5, torch.ones(1, device=dev))
        blk = LinearBF16(ClampedGlu.interleave(W[:N // 2], W[N // 2:]).to(dev))
        got = gemv_rows(blk, M, **n.prologue(x.to(dev)), **ClampedGlu(0.8, 1.702, True).epilogue())
        z = plain.layer_norm(x[:, 0].double(), w.double(), 1e-5).float().to(torch.bfloat16).double() @ Wd.t()
        eye = torch.eye(N // 2, dtype=torch.float64)
        v = plain.clamped_ff({"gate": torch.cat([eye, 0 * eye], 1), "up": torch.cat([0 * eye, eye], 1), "down": eye}, "", {"limit": 0.8}, z)
        assert got.shape == (M, N // 2) and (got.double().cpu() - v).abs().max() < 2e-2 * v.pow(2).mean().sqrt() + 2 ** -8 * v.abs().max()
    for G in (g for g in (8, 5, 1) if (K - 11) % g == 0 or K % 8 == 0):
        k0 = K % G + 2 * G
        a, x, gate, w = rnd(M, k0, seed=9), rnd(M, K - k0, seed=10), rnd(M, K - k0 + 2, seed=11)[:, 1:-1], rnd(G, seed=12)
        v = plain.rms_norm(x.double().reshape(M, -1, G), w.double(), 1e-4).reshape(M, -1) * plain.silu(gate.double())
        got = gemv_rows(lin, M, out_f32=True, **GroupRMS(w.to(dev), 1e-4, G, silu=True).prologue(x.to(dev), gate.to(dev), head=a.to(dev)))
        check(got, torch.cat([a.double(), v], 1))


# ------------------------------------------------------------------------------------------ attention
def test_distance_buckets():
    for B, D in ((32, 128), (6, 9), (2, 5), (16, 17), (32, 200), (8, 1000)):
        t = torch.arange(B * 2, dtype=torch.float32).reshape(B, 2)
        bias = distance_bias(t, D)
        assert bias[0, -1] == t[B - 1, 0] and bias[0, -2] != t[B - 1, 0]                    # as short as it can be
        for n in range(D + 40):
            assert bias[1, min(n, bias.shape[1] - 1)] == t[plain.distance_bucket(n, B, D), 1]
    for B, D in ((5, 20), (8, 4)):
        with pytest.raises(ValueError):
            distance_bias(torch.zeros(B, 1), D)


def attn_case(H, G, d, dv, B=8, D=50, coef=0.0, every=1, scale=None, seed=0, out_scale=1.0, norm=True, sink=0.0):
    """-> (spec on the CPU, the plain statement's mixer dictionary and weights: projections that select columns)."""
    rel, snk = rnd(B, H, seed=seed), torch.full((H,), sink) + rnd(H, seed=seed + 1)
    qn, kn = 1 + rnd(d, seed=seed + 2, scale=0.2), 1 + rnd(d, seed=seed + 3, scale=0.2)
    spec = GqaSpec(H, G, d, dv, scale or d ** -0.5, 1e-5, qn, kn, coef, every, distance_bias(rel, D), snk, out_scale)
    eye = torch.eye(spec.cols, dtype=torch.float64)
    W = {"q": eye[:H * d], "k": eye[H * d:(H + G) * d], "v": eye[(H + G) * d:], "q.norm": qn.double(), "k.norm": kn.double(), "rel": rel.double(),
         "sink": snk.double(), "o": torch.eye(H * dv, dtype=torch.float64) * out_scale}
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": spec.scale, "bias_max": D, "q_temp": {"coef": coef, "every": every}}
    return spec, W, m


def put(spec, device):
    move = lambda t: None if t is None else t.to(device)
    return GqaSpec(spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.scale, spec.eps, move(spec.q_norm), move(spec.k_norm), spec.temp_coef, spec.temp_every,
                   move(spec.bias), move(spec.sink), spec.out_scale)


class AttnRun:
    """A paged cache (its rows wider than this layer's, filled with an earlier request's rows) and batches through the operator."""

    def __init__(self, spec, dtype, device, slots=3, pages=24, extra=0, o32=False):
        self.spec, self.dtype, self.device, self.o32 = put(spec, device), dtype, device, o32
        kw, vw = spec.row_widths
        self.kv = PagedKVCache(2, 1, kw + extra, pages, slots, 1024, torch.device(device), dtype=dtype, v_head_dim=vw + extra)
        self.kv.k.fill_(3.0)
        self.kv.v.fill_(-3.0)

    def rows(self, parts):
        """parts: [(slot, first position, projection rows)] one batch, shortest first."""
        pos, slots = [], []
        for s, p0, x in parts:
            self.kv.reserve(s, p0 + x.shape[0])
            pos += range(p0, p0 + x.shape[0])
            slots += [s] * x.shape[0]
        b = BatchRows.make(pos, pos, slots, self.device)
        x = torch.cat([torch.nn.functional.pad(p[2], (0, 3)) for p in parts]).to(self.device)          # columns of something else behind it
        dt = torch.float32 if self.o32 and b.row_path else self.dtype
        w = self.spec.heads * self.spec.vdim
        y = torch.full((len(pos), w + 8), 5.0, dtype=dt, device=self.device)
        gqa_attend(self.spec, x, b, self.kv, self.kv.k[1], self.kv.v[1], y[:, :w])
        assert bool((y[:, w:] == 5.0).all())
        return y[:, :w].float().cpu()

    def walk(self, slot, x, cuts):
        at, got = 0, []
        for c in cuts:
            got.append(self.rows([(slot, at, x[at:at + c])]))
            at += c
        return torch.cat(got)


ATT = [(4, 2, 24, 40), (3, 3, 21, 13), (8, 2, 128, 128), (18, 1, 16, 8), (2, 1, 64, 136), (3, 1, 40, 16), (1, 1, 264, 24), (2, 2, 200, 128), (5, 5, 8, 64)]
CUT = [[210], [64, 64, 82], [1] * 10 + [60, 16, 2, 41, 1, 1, 15, 17] + [1] * 47, [130] + [2] * 40]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,G,d,dv", ATT)
def test_every_row_finds_its_key(H, G, d, dv, dtype, device):
    """A row's query is lined up with one key of its past (page borders, the first token, itself, the row before), so its output is
    almost that key's value."""
    T, (spec, W, m) = 210, attn_case(H, G, d, dv, seed=H + d, coef=0.3, every=40, sink=-1.0, out_scale=0.8)
    x = rnd(T, spec.cols, seed=5)
    pick = [max(0, min(t, [0, t, t - 1, 63, 64, 127, 128, t // 2, 1][t % 9])) for t in range(T)]
    spec.q_norm, spec.k_norm = torch.ones(d), torch.ones(d)
    W["q.norm"], W["k.norm"] = torch.ones(d).double(), torch.ones(d).double()
    spec.scale = m["scale"] = 26.0 / d                                # |q| |k| = d: score 26 for the key picked
    k = x[:, H * d:(H + G) * d].reshape(T, G, d).repeat_interleave(H // G, 1)
    x[:, :H * d] = torch.stack([k[pick[t]] for t in range(T)]).reshape(T, H * d)
    x = x.to(torch.bfloat16).float()
    want = plain.biased_attention(W, "", m, x.double(), spec.eps)
    if d >= 16:
        v = x[:, (H + G) * d:].reshape(T, G, dv).repeat_interleave(H // G, 1)
        near = torch.stack([v[pick[t]] for t in range(T)]).reshape(T, -1) * 0.8
        assert ((want - near).norm(dim=1) < 0.5 * near.norm(dim=1)).float().mean() > 0.9
    tol = 3e-5 if dtype == torch.float32 else 0.03
    for n, cuts in enumerate(CUT):
        if device == "cpu" and n % 2:
            continue
        got = AttnRun(spec, dtype, device, extra=40 * (n % 2), o32=n >= 2).walk(1, x, cuts)
        err = (got.double() - want[:got.shape[0]]).abs().max().item()
        assert err < tol * want.abs().max(), (n, err)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("B,D", [(8, 50), (16, 17), (32, 200), (6, 130)])
def test_the_edges_of_every_distance_bucket(B, D, dtype, device):
    """All scores alike but for the bias; one head per bucket, whose bias stands out there: a head's output is the mean of the values
    in its bucket, and changes when a bucket's edge is a token off."""
    T, G, d, dv = 300, 1, 8, 16
    H = B
    spec, W, m = attn_case(H, G, d, dv, B, D, sink=-3.0)
    rel = 20.0 * torch.eye(B, H) + rnd(B, H, seed=9)
    spec.bias = distance_bias(rel, D)
    W["rel"] = rel.double()
    x = torch.cat([torch.zeros(T, H * d), torch.ones(T, d), rnd(T, dv, seed=4)], 1).to(torch.bfloat16).float()
    want = plain.biased_attention(W, "", m, x.double(), spec.eps)
    tol = 2e-5 if dtype == torch.float32 else 0.01
    for cuts in ([300], [100, 64, 1, 1, 2, 90, 42]) if device == "cuda" or dtype == torch.float32 else ([300],):
        got = AttnRun(spec, dtype, device).walk(0, x, cuts)
        assert (got.double() - want).abs().max() < tol * want.abs().max()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("sink", [-60.0, 0.0, 12.0, 90.0])
def test_sinks_from_nothing_to_everything(sink, dtype, device):
    """The sink counts once, whatever the number of splits and streams: rows with few and many keys."""
    T, (spec, W, m) = 330, attn_case(4, 2, 32, 24, sink=sink, seed=2)
    x = rnd(T, spec.cols, seed=3).to(torch.bfloat16).float()
    want = plain.biased_attention(W, "", m, x.double(), spec.eps)
    for cuts in ([T], [1] * 3 + [300] + [1] * 27) if device == "cuda" or dtype == torch.float32 else ([T],):
        got = AttnRun(spec, dtype, device).walk(2, x, cuts)
        assert (got.double() - want).abs().max() < (2e-5 if dtype == torch.float32 else 0.02) * want.abs().max().clamp(min=1e-30)
    if sink == 90.0:
        assert want.abs().max() < 1e-20


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("coef,every", [(0.5, 1), (2.0, 7), (-0.15, 64), (1.0, 100000)])
def test_query_temperature_steps(coef, every, device):
    T, (spec, W, m) = 150, attn_case(2, 1, 16, 16, coef=coef, every=every, scale=0.5, seed=6)
    x = rnd(T, spec.cols, seed=7)
    want = plain.biased_attention(W, "", m, x.double(), spec.eps)
    got = AttnRun(spec, torch.float32, device).walk(0, x, [63, 1, 1, 85])
    assert (got.double() - want).abs().max() < 3e-5 * want.abs().max()
    if every == 7:
        assert plain.query_temperature(5, coef, every) != plain.query_temperature(6, coef, every) == plain.query_temperature(12, coef, every)


@pytest.mark.parametrize("device", DEVICES)
def test_attention_without_the_optional_terms(device):
    """No norms, temperature, bias or sink: plain causal grouped attention."""
    H, G, d, dv, T = 4, 2, 16, 24, 140
    spec = GqaSpec(H, G, d, dv, 0.3)
    x = rnd(T, spec.cols, seed=1).to(torch.bfloat16).float()
    q, k, v = (t.double() for t in (x[:, :H * d].reshape(T, H, d), x[:, H * d:(H + G) * d].reshape(T, G, d), x[:, (H + G) * d:].reshape(T, G, dv)))
    s = torch.einsum("thd,jhd->htj", q, k.repeat_interleave(2, 1)) * 0.3
    s = s.masked_fill(torch.ones(T, T).triu(1).bool(), -math.inf)
    want = torch.einsum("htj,jhv->thv", torch.softmax(s, -1), v.repeat_interleave(2, 1)).reshape(T, -1)
    for dtype in TYPES:
        got = AttnRun(spec, dtype, device).walk(0, x, [T] if dtype == torch.bfloat16 else [70, 70])
        assert (got.double() - want).abs().max() < (2e-5 if dtype == torch.float32 else 0.03) * want.abs().max()
    assert (AttnRun(spec, torch.bfloat16, device).walk(0, x, [100] + [1] * 40).double() - want).abs().max() < 0.03 * want.abs().max()


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
def test_attention_of_a_mixed_batch(dtype, device):
    spec, W, m = attn_case(6, 2, 40, 24, seed=9, coef=0.2, every=30)
    r = AttnRun(spec, dtype, device)
    seq = [(rnd(140, spec.cols, seed=s) * 1.5).to(torch.bfloat16).float() for s in range(3)]
    want = [plain.biased_attention(W, "", m, s.double(), spec.eps) for s in seq]
    at = [0, 0, 0]
    for counts in ((1, 5, 100), (2, 3, 20), (1, 1, 1), (16, 40, 3), (0, 80, 1), (0, 1, 1)):
        order = sorted((i for i in range(3) if counts[i]), key=lambda i: counts[i])
        got = r.rows([(i, at[i], seq[i][at[i]:at[i] + counts[i]]) for i in order])
        exp = torch.cat([want[i][at[i]:at[i] + counts[i]] for i in order])
        assert (got.double() - exp).abs().max() < (2e-5 if dtype == torch.float32 else 0.03) * exp.abs().max()
        for i in range(3):
            at[i] += counts[i]


@pytest.mark.gpu
@pytest.mark.parametrize("H,G,d,dv", [(4, 1, 128, 128), (3, 3, 64, 64), (2, 1, 256, 128), (6, 2, 40, 72)])
def test_prompt_of_many_pages_with_moving_references(H, G, d, dv):
    """Scores grow along the sequence, then fall: both streams, all ring stages and several query tiles."""
    spec, W, m = attn_case(H, G, d, dv, B=32, D=200, seed=3, coef=1.0, every=100, scale=2.0 / d ** 0.5)
    T = 700
    x = rnd(T, spec.cols, seed=5).to(torch.bfloat16).float()
    want = plain.biased_attention(W, "", m, x.double(), spec.eps)
    for cuts in ([T], [1, 399, 300], [129, 127, 444], [690] + [1] * 10):
        got = AttnRun(spec, torch.bfloat16, "cuda").walk(2, x, cuts)
        assert ((got.double() - want).abs().max() / want.abs().max()).item() < 0.03


@pytest.mark.gpu
def test_splits_leave_their_tickets_as_they_found_them():
    from volta_engine_b200.ops import gqa
    spec, W, m = attn_case(4, 2, 64, 64)
    x = rnd(1000, spec.cols, seed=5).to(torch.bfloat16).float()
    r = AttnRun(spec, torch.bfloat16, "cuda")
    first = [r.walk(s, x, [900] + [1] * 12)[900:] for s in (0, 0)]
    assert torch.equal(*first)                                        # the same rows again, bit by bit
    assert int(gqa._ticket_words(r.kv.page_table.device).abs().sum()) == 0


# ------------------------------------------------------------------------------------------ gated linear attention
def gla_case(H, dk, dv, rank, tau, seed=0):
    a2, b = rnd(H * dk, rank, seed=seed), rnd(H * dk, seed=seed + 1, scale=2)
    b[::3] += 8.0                                                     # channels that hardly forget
    b[1::3] -= 12.0                                                   # channels that forget fast
    spec = LinAttnSpec(H, dk, dv, bias=b, w2=a2, a_col=H * (2 * dk + 2 * dv), tau=tau, q_scale=dk ** -0.5)
    cols = spec.a_col + rank
    eye = torch.eye(cols, dtype=torch.float64)
    at = [0, H * dk, 2 * H * dk, 2 * H * dk + H * dv, spec.a_col, cols]
    W = {n: eye[i:j] for n, i, j in zip(("q", "k", "v", "g", "a1"), at, at[1:])}
    W.update({"a2": a2.double(), "a2.b": b.double(), "norm": torch.ones(dv).double(), "o": torch.eye(H * dv, dtype=torch.float64)})
    return spec, W, {"heads": H, "dim": dk, "vdim": dv, "tau": tau}


GLA = [(2, 32, 32, 16, 16.0), (3, 24, 40, 12, 8.0), (1, 128, 128, 16, 16.0), (2, 13, 7, 5, 1.0), (2, 64, 96, 40, 4.0), (1, 200, 33, 8, 2.0), (2, 16, 136, 33, 16.0)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("H,dk,dv,rank,tau", GLA)
def test_gated_linear_attention_in_portions(H, dk, dv, rank, tau, chunked, device):
    """One long sequence in portions of all kinds beside a second one, in slots that hold another sequence's state before."""
    base, W, m = gla_case(H, dk, dv, rank, tau)
    spec = LinAttnSpec(H, dk, dv, bias=base.bias.to(device), w2=base.w2.to(device), a_col=base.a_col, tau=tau, q_scale=base.q_scale)
    norm = GroupRMS(torch.ones(dv, device=device), 1e-6, dv, silu=True)
    st = LinAttnState(spec, 3, device)
    st.rec.fill_(7.0)                                                 # what an earlier request left behind
    cols = base.a_col + rank
    a, b = rnd(330, cols, seed=3), rnd(90, cols, seed=4)
    for t in (a, b):
        t[:, 2 * H * dk:2 * H * dk + H * dv] = t[:, 2 * H * dk:2 * H * dk + H * dv].to(torch.bfloat16).float()      # values that are exact in bf16
    a[37, base.a_col:] *= 30.0
    wa, wb = (plain.gated_linear_attention(W, "", m, t.double(), 1e-6) for t in (a, b))
    got_a, got_b, at, bt = [], [], 0, 0
    for na, nb in ((1, 0), (64, 1), (2, 0), (100, 40), (63, 3), (17, 16), (1, 1), (16, 0), (65, 29), (1, 0)):
        ids = list(range(at, at + na)) + list(range(bt, bt + nb))
        proj = torch.nn.functional.pad(torch.cat([a[at:at + na], b[bt:bt + nb]]), (4, 3)).to(device)[:, 4:]         # a part of wider rows
        o = linattn_rows(proj, BatchRows.make(ids, ids, [2] * na + [0] * nb, device), st, spec, chunked=chunked)
        y = norm.rows(o, torch.float32, gate=proj[:, spec.cols: spec.cols + H * dv])
        got_a.append(y[:na].cpu())
        got_b.append(y[na:].cpu())
        at, bt = at + na, bt + nb
    for got, want in ((torch.cat(got_a), wa), (torch.cat(got_b), wb)):
        assert (got.double() - want).abs().max() < 5e-4 * want.abs().max()
    assert bool((st.rec[1] == 7.0).all())                             # the slot nobody used


@pytest.mark.parametrize("device", DEVICES)
def test_a_far_token_survives_in_the_state(device):
    """One channel never forgets: a value written at the first token is read 300 tokens later, through portions and single rows."""
    H, dk, dv, rank = 1, 16, 16, 4
    base, W, m = gla_case(H, dk, dv, rank, 16.0)
    base.bias[:], base.w2[:] = -12.0, 0.0
    base.bias[5] = 30.0
    spec = LinAttnSpec(H, dk, dv, bias=base.bias.to(device), w2=base.w2.to(device), a_col=base.a_col, tau=16.0, q_scale=base.q_scale)
    T = 320
    x = rnd(T, base.a_col + rank, seed=1)
    x[:, dk + 5] = 0.0
    x[0, dk + 5] = 40.0
    x[-1, :dk] = 0.0
    x[-1, 5] = 4.0                                                    # the last query asks that channel alone
    for cuts in ([T], [70, 1, 129, 120], [300] + [1] * 20):
        st, at = LinAttnState(spec, 1, device), 0
        for c in cuts:
            ids = list(range(at, at + c))
            o = linattn_rows(x[at:at + c].to(device), BatchRows.make(ids, ids, [0] * c, device), st, spec)
            at += c
        want = 40.0 * x[0, 2 * dk:2 * dk + dv].double()
        assert (o[-1].double().cpu() - want).abs().max() < 5e-3 * want.abs().max()


@pytest.mark.parametrize("device", DEVICES)
def test_decays_at_both_ends(device):
    """sigmoid(z)^(1 / tau) where the sigmoid underflows or is one: through the step, and as the rows the chunks read."""
    z = torch.tensor([-200.0, -60.0, -5.0, 0.0, 5.0, 20.0, 200.0])
    want = torch.exp(torch.nn.functional.logsigmoid(z.double()) / 16.0)
    H, dk, dv = 1, z.numel(), 4
    spec = LinAttnSpec(H, dk, dv, bias=z.to(device), w2=torch.zeros(dk, 4, device=device), a_col=2 * dk + dv, tau=16.0)
    st = LinAttnState(spec, 1, device)
    st.rec.fill_(1.0)
    linattn_rows(torch.zeros(1, spec.a_col + 4, device=device), BatchRows.make([1], [1], [0], device), st, spec)
    close(st.rec[0, 0, :, 0], want, torch.float32)
    if device == "cuda":
        from volta_engine_b200._lib import call, ptr
        for rank in (4, 20, 70):
            dec, a, w2, zz = torch.empty(5, dk, device="cuda"), torch.zeros(5, rank, device="cuda"), torch.zeros(dk, rank, device="cuda"), z.cuda()
            call("linattn_decay", "plippp" + "iiif", ptr(a), rank, 1, ptr(w2), ptr(zz), ptr(dec), 5, dk, rank, 1.0 / 16.0)
            close(dec, want.expand(5, dk), torch.float32)
