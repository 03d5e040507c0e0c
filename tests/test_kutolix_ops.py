"""Every mechanism of the Kutolix decoder alone against the plain statement: rotations and their scaling, windowed attention with sink and
gate, latent attention with direct queries, routers and experts, norms on sublayer results, the decode linears that carry them, gated
units, soft caps, scaled embeddings. Inputs are made so that a wrong key, a window one token off, a sink that is left out or a wrong
expert shows."""
import math

import pytest
import torch

import kutolix_plain as plain
from listed_util import DEVICES, Rows, one_thread, vars_of  # noqa: F401
from volta_engine_b200.ops.gqa import GqaSpec, gqa_attend, gqa_store
from volta_engine_b200.ops.latent import LatentSpec, latent_rows
from volta_engine_b200.ops.linear import LinearBF16, LinearF32
from volta_engine_b200.ops.rotary import Rotation
from volta_engine_b200.ops.routed import ExpertWeights, Router, route, routed_few, routed_many, routed_reference
from volta_engine_b200.ops.rowops import ClampedGlu, NormedWrite, ResidualNorm, RoutedRows, embed_rows, gemv_rows, soft_cap_
from volta_engine_b200.runtime.kv_cache import PagedKVCache

TYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 3e-5, torch.bfloat16: 0.03}


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def close(got, want, dtype, f32=2e-6, bf16=2 ** -8):
    w = want.double()
    tol = f32 if dtype == torch.float32 else bf16
    assert got.shape == w.shape and bool(((got.double().cpu() - w).abs() <= tol * (w.abs() + w.pow(2).mean().sqrt())).all())


def apart(got, want):
    return ((got.double().cpu() - want.double()).abs().max() / want.double().abs().max()).item()


# ------------------------------------------------------------------------------------------ rotations
ROTS = [{"dims": 16, "base": 500.0}, {"dims": 64, "base": 1e6}, {"dims": 2, "base": 7.0}, {"dims": 10, "base": 90.0},
        {"dims": 16, "base": 300.0, "scaling": {"factor": 8.0, "original": 64, "fast": 6.0, "slow": 1.0}},
        {"dims": 64, "base": 1e4, "scaling": {"factor": 32.0, "original": 4096, "fast": 32.0, "slow": 1.0}},
        {"dims": 6, "base": 50.0, "scaling": {"factor": 2.0, "original": 20, "fast": 2.0, "slow": 2.0}},            # the ramp is one step
        {"dims": 8, "base": 10.0, "scaling": {"factor": 1.0, "original": 100, "fast": 9.0, "slow": 1.0}},
        {"dims": 12, "base": 1e5, "scaling": {"factor": 4.0, "original": 1e9, "fast": 64.0, "slow": 0.001}},          # both ends clipped
        {"dims": 128, "base": 2e4, "scaling": {"factor": 3.7, "original": 777, "fast": 11.0, "slow": 0.3}}]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("neighbours", [False, True])
@pytest.mark.parametrize("rot", ROTS, ids=lambda r: f"{r['dims']}{'s' if 'scaling' in r else ''}")
def test_rotations(rot, neighbours, device):
    """Near and far positions; the columns behind the rotated ones stay. On the GPU as the queries leave the attention's first kernel."""
    f, mul = plain.frequencies(rot)
    r = Rotation.from_config(rot, neighbours)
    assert torch.allclose(r.freq, torch.tensor(f, dtype=torch.float64), rtol=1e-12) and abs(r.mul - mul) < 1e-12
    pos = torch.tensor([0, 1, 2, 63, 64, 1000, 131071, 1_000_003], dtype=torch.int32)
    for wide in (rot["dims"], rot["dims"] + 8 - rot["dims"] % 8, rot["dims"] + 5):
        v = rnd(len(pos), 2, wide, seed=3)
        want = torch.stack([plain.rotate(v[i].double(), int(p), rot, neighbours) for i, p in enumerate(pos)])
        if device == "cpu":
            got = r.turn(v, pos)
        else:
            spec = GqaSpec(2, 1, wide, 8, 1.0, rot=Rotation.from_config(rot, neighbours).bind(device))
            kv = PagedKVCache(1, 1, spec.kw, 2, 1, 64, torch.device(device), dtype=torch.float32, v_head_dim=8)
            proj = torch.nn.functional.pad(v.reshape(len(pos), -1), (0, wide + 8)).to(device)
            hidden = torch.full((len(pos),), -1, dtype=torch.int32, device=device)                    # rows of no slot: queries only
            got = gqa_store(spec, proj, pos.to(device), hidden, kv, kv.k[0], kv.v[0])[0][:, :, :wide].cpu()
        assert (got.double() - want).abs().max() < 4e-6 * mul


def test_scaled_frequencies_keep_the_fast_and_slow_the_slow():
    rot = {"dims": 64, "base": 1e4, "scaling": {"factor": 32.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    plainly = Rotation(64, 1e4).freq
    f = Rotation.from_config(rot, True).freq
    assert f[0] == plainly[0] and torch.allclose(f[-1], plainly[-1] / 32.0) and bool((f[1:] < f[:-1]).all())
    with pytest.raises(ValueError):
        Rotation(7, 10.0)
    with pytest.raises(NotImplementedError):
        Rotation(1024, 10.0)


# ------------------------------------------------------------------------------------------ windowed attention
def att_case(H, G, d, dv, window, dims=None, base=500.0, scale=None, sink=0.0, seed=0):
    """-> (spec on the CPU, mixer dictionary, weights of the plain statement: projections that select columns)."""
    snk = torch.full((H,), sink) + rnd(H, seed=seed + 1)
    dims = d // 2 * 2 if dims is None else dims
    spec = GqaSpec(H, G, d, dv, scale or d ** -0.5, 1e-5, sink=snk, rot=Rotation(dims, base, False), unit=True, window=window, gated=True)
    eye = torch.eye(spec.cols, dtype=torch.float64)
    W = {"q": eye[:H * d], "k": eye[H * d:(H + G) * d], "v": eye[(H + G) * d: spec.gate_col], "g": eye[spec.gate_col:], "sink": snk.double(),
         "o": torch.eye(H * dv, dtype=torch.float64)}
    return spec, {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": spec.scale, "mask": {"size": window}, "rot": {"dims": dims, "base": base}}, W


class AttnRows(Rows):
    def __init__(self, spec, dtype, device, extra=0, x32=False):
        super().__init__(dtype, device, *spec.row_widths, extra)
        move = lambda t: None if t is None else t.to(device)
        self.spec, self.x32 = GqaSpec(**dict(vars_of(spec), sink=move(spec.sink), rot=Rotation(spec.rot.dims, spec.rot.base, False).bind(device))), x32

    def run(self, b, x):
        x = torch.nn.functional.pad(x, (0, 3)).to(self.device)                        # columns of something else behind it
        if self.dtype == torch.bfloat16 and not self.x32 and not b.row_path:
            x = x.to(torch.bfloat16)                                                  # as prompts bring it
        w = self.spec.heads * self.spec.vdim
        y = torch.full((b.n, w + 8), 5.0, dtype=self.dtype, device=self.device)
        gqa_attend(self.spec, x, b, self.kv, self.kv.k[1], self.kv.v[1], y[:, :w])
        assert bool((y[:, w:] == 5.0).all())
        return y[:, :w].float().cpu()


ATT = [(4, 2, 24, 40, 37, 16), (3, 3, 21, 13, 19, 10), (8, 2, 128, 128, 64, 128), (18, 1, 16, 8, 65, 2), (2, 1, 64, 136, 100, 64), (1, 1, 264, 24, 50, 100), (5, 5, 8, 64, 1, 8),
       (6, 3, 32, 24, 128, 12), (4, 1, 40, 16, 3, 24), (2, 2, 200, 128, 129, 8), (4, 2, 64, 64, 1000, 0)]
CUT = [[210], [64, 64, 82], [1] * 10 + [60, 16, 2, 41, 1, 1, 15, 17] + [1] * 47, [130] + [2] * 40]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,G,d,dv,window,dims", ATT)
def test_every_row_finds_its_key_inside_the_window_and_none_outside(H, G, d, dv, window, dims, dtype, device):
    """A row's query is lined up with one key: itself, the row before, the last key its window keeps, the first one that it does not, keys
    at page borders, the first token. Keys inside give their value, keys outside nothing."""
    T, (spec, m, W) = 210, att_case(H, G, d, dv, window, dims, seed=H + d, sink=-2.0)
    spec.scale = m["scale"] = 24.0 / d                                  # |q| |k| = d: score 24 for the key picked
    x = rnd(T, spec.cols, seed=5)
    choice = lambda t: [t, t - 1, t - window + 1, t - window, t // 64 * 64, t // 64 * 64 - 1, 0, t - window // 2, t - window - 1][t % 9]
    pick = [max(0, min(t, choice(t))) for t in range(T)]
    k = x[:, H * d:(H + G) * d].reshape(T, G, d).repeat_interleave(H // G, 1).double()
    q = torch.stack([plain.rotate(k[pick[t]], pick[t] - t, m["rot"], False) for t in range(T)])             # turned by the difference
    x[:, :H * d] = q.reshape(T, H * d).float()
    x = x.to(torch.bfloat16).float()
    want = plain.windowed_attention(W, "", m, x.double(), spec.eps)
    if d >= 16:
        v = x[:, (H + G) * d: spec.gate_col].reshape(T, G, dv).repeat_interleave(H // G, 1)
        near = torch.stack([v[pick[t]] for t in range(T)]).reshape(T, -1) * torch.sigmoid(x[:, spec.gate_col:])
        hit = (want - near).norm(dim=1) < 0.5 * near.norm(dim=1)
        inside = torch.tensor([t - pick[t] < window for t in range(T)])
        assert hit[inside].float().mean() > 0.9 and hit[~inside].float().mean() < 0.1 if (~inside).any() else hit.float().mean() > 0.9
    for n, cuts in enumerate(CUT):
        if device == "cpu" and n % 2:
            continue
        got = AttnRows(spec, dtype, device, extra=40 * (n % 2), x32=n >= 2).walk(1, x, cuts)
        assert apart(got, want[:got.shape[0]]) < TOL[dtype], n


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("sink", [-60.0, 0.0, 12.0, 90.0])
def test_sinks_from_nothing_to_everything(sink, dtype, device):
    """The sink counts once, whatever the number of splits, streams and keys."""
    T, (spec, m, W) = 330, att_case(4, 2, 32, 24, 200, sink=sink, seed=2)
    x = rnd(T, spec.cols, seed=3).to(torch.bfloat16).float()
    want = plain.windowed_attention(W, "", m, x.double(), spec.eps)
    for cuts in ([T], [1] * 3 + [300] + [1] * 27) if device == "cuda" or dtype == torch.float32 else ([T],):
        got = AttnRows(spec, dtype, device).walk(2, x, cuts)
        assert (got.double() - want).abs().max() < TOL[dtype] * want.abs().max().clamp(min=1e-30)
    if sink == 90.0:
        assert want.abs().max() < 1e-20


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("dv", [16, 12, 5])
def test_gates_open_and_shut(dv, dtype, device):
    """Every element has a gate of its own: open, half open, shut, in prompts (gate in bf16) and single rows (gate in fp32)."""
    T, (spec, m, W) = 150, att_case(3, 1, 16, dv, 64, seed=8)
    x = rnd(T, spec.cols, seed=1)
    gate = x[:, spec.gate_col:]
    gate[:] = torch.tensor([-90.0, -1.0, 0.0, 1.5, 40.0])[torch.randint(0, 5, gate.shape, generator=torch.Generator().manual_seed(2))]
    x = x.to(torch.bfloat16).float()
    want = plain.windowed_attention(W, "", m, x.double(), spec.eps)
    for cuts in ([T], [100] + [1] * 50, [20] * 7 + [10]):
        got = AttnRows(spec, dtype, device).walk(0, x, cuts)
        assert apart(got, want) < TOL[dtype]
        assert bool((got[gate < -50].abs() < 1e-20).all())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
def test_small_queries_and_keys_see_eps_inside_the_root(dtype, device):
    T, (spec, m, W) = 40, att_case(2, 1, 16, 8, 30, scale=0.7)
    x = rnd(T, spec.cols, seed=4)
    x[:, :3 * 16] *= 3e-3
    x = x.to(torch.bfloat16).float()
    want = plain.windowed_attention(W, "", m, x.double(), spec.eps)
    assert apart(AttnRows(spec, dtype, device).walk(0, x, [25, 1, 14]), want) < TOL[dtype]
    spec.eps = 1e-9                                                     # it matters here
    assert apart(AttnRows(spec, torch.float32, "cpu").walk(0, x, [T]), want) > 0.01


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
def test_attention_of_a_mixed_batch(dtype, device):
    spec, m, W = att_case(6, 2, 40, 24, 33, seed=9, scale=0.6)
    r = AttnRows(spec, dtype, device)
    seq = [(rnd(140, spec.cols, seed=s) * 1.5).to(torch.bfloat16).float() for s in range(3)]
    want = [plain.windowed_attention(W, "", m, s.double(), spec.eps) for s in seq]
    at = [0, 0, 0]
    for counts in ((1, 5, 100), (2, 3, 20), (1, 1, 1), (16, 40, 3), (0, 80, 1), (0, 1, 1)):
        order = sorted((i for i in range(3) if counts[i]), key=lambda i: counts[i])
        got = r.batch([(i, at[i], seq[i][at[i]:at[i] + counts[i]]) for i in order])
        assert apart(got, torch.cat([want[i][at[i]:at[i] + counts[i]] for i in order])) < TOL[dtype]
        for i in range(3):
            at[i] += counts[i]


@pytest.mark.gpu
@pytest.mark.parametrize("H,G,d,dv,window", [(4, 1, 128, 128, 300), (3, 3, 64, 64, 64), (2, 1, 256, 128, 511), (6, 2, 40, 72, 130), (4, 2, 128, 64, 5000)])
def test_prompt_of_many_pages(H, G, d, dv, window):
    """Windows of several pages: both streams, all ring stages, query tiles that start anywhere in their window; long decoding behind it."""
    spec, m, W = att_case(H, G, d, dv, window, seed=3, scale=3.0 / d ** 0.5, base=1e4)
    T = 700
    x = rnd(T, spec.cols, seed=5).to(torch.bfloat16).float()
    want = plain.windowed_attention(W, "", m, x.double(), spec.eps)
    for cuts in ([T], [1, 399, 300], [129, 127, 444], [400] + [1] * 300):
        assert apart(AttnRows(spec, torch.bfloat16, "cuda").walk(2, x, cuts), want) < 0.03


# ------------------------------------------------------------------------------------------ latent attention
def lat_case(H, d, rot, dv, kr, window, scaling=(4.0, 60, 5.0, 1.0), base=300.0, scale=None, seed=0):
    scaling = dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None
    spec = LatentSpec(H, d, rot, dv, kr, scale or (d + rot) ** -0.5, base, 1e-5, scaling, window)
    nq = H * (d + rot)
    eye = torch.eye(nq + kr + rot, dtype=torch.float64)
    W = {"q": eye[:nq], "dkv": eye[nq:], "dkv.norm": (1 + rnd(kr, seed=seed + 2, scale=0.2)).double(), "o": torch.eye(H * dv, dtype=torch.float64),
         "uk": (rnd(H * d, kr, seed=seed) * kr ** -0.5).to(torch.bfloat16).double(), "uv": (rnd(H * dv, kr, seed=seed + 1) * kr ** -0.5).to(torch.bfloat16).double()}
    m = {"heads": H, "dim": d, "rot_dim": rot, "vdim": dv, "kv_rank": kr, "scale": spec.scale, "mask": {"size": window} if window else None,
         "rot": {"base": base, "dims": rot, "scaling": scaling}}
    return spec, m, W


class LatentRows(Rows):
    def __init__(self, spec, W, dtype, device, extra=0):
        super().__init__(dtype, device, spec.width, 8, extra)
        self.spec = LatentSpec(**vars_of(spec)).bind(device)
        self.uk, self.uv, self.norm = W["uk"].to(device, dtype), W["uv"].to(device, dtype), W["dkv.norm"].float().to(device)
        self.ukv = LinearBF16(torch.cat([self.uk, self.uv], 0)) if dtype == torch.bfloat16 else None

    def run(self, b, x):
        x = x.to(self.device, torch.float32 if b.row_path or self.dtype == torch.float32 else torch.bfloat16)      # as the projection leaves it
        nq = self.spec.heads * (self.spec.dim + self.spec.rot)
        return latent_rows(self.spec, x[:, :nq], x[:, nq:], self.norm, self.uk, self.uv, self.ukv, b, self.kv, self.kv.k[1]).float().cpu()


LAT = [(3, 40, 8, 24, 72, 37), (2, 21, 6, 18, 50, 19), (2, 128, 64, 128, 512, 64), (17, 40, 24, 16, 64, 65), (1, 64, 32, 72, 136, 100), (2, 24, 16, 40, 544, 3),
       (2, 192, 64, 256, 256, 128), (1, 100, 24, 64, 320, 1), (3, 32, 16, 48, 40, 129), (2, 16, 8, 8, 24, 1000)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,d,rot,dv,kr,window", LAT)
def test_every_row_finds_its_latent_inside_the_window_and_none_outside(H, d, rot, dv, kr, window, dtype, device):
    T, (spec, m, W) = 210, lat_case(H, d, rot, dv, kr, window, seed=H)
    kv = rnd(T, kr + rot, seed=5).to(torch.bfloat16).float()
    choice = lambda t: [t, t - 1, t - window + 1, t - window, t // 64 * 64, t // 64 * 64 - 1, 0, t - window // 2, t - window - 1][t % 9]
    pick = [max(0, min(t, choice(t))) for t in range(T)]
    c = plain.rms_norm(kv[:, :kr].double(), W["dkv.norm"], spec.eps)
    k, v = (c @ W["uk"].T).reshape(T, H, d), (c @ W["uv"].T).reshape(T, H, dv)
    q = torch.zeros(T, H, d + rot, dtype=torch.float64)
    _, mul = plain.frequencies(m["rot"])
    for t in range(T):
        j = pick[t]
        turned = plain.rotate(kv[j, kr:].double(), j - t, m["rot"], True)              # the score sees the difference of positions,
        q[t] = torch.cat([k[j], turned.expand(H, rot)], -1)                           # and the factor of both turns
        q[t] *= 24.0 / spec.scale / ((k[j] * k[j]).sum(-1, keepdim=True) + mul * (turned * turned).sum())
    x = torch.cat([q.reshape(T, -1).float().to(torch.bfloat16).float(), kv], 1)
    want = plain.latent_attention(W, "", m, x.double(), spec.eps)
    near = torch.stack([v[pick[t]] for t in range(T)]).reshape(T, -1)
    hit = (want - near).norm(dim=1) < 0.5 * near.norm(dim=1)
    inside = torch.tensor([t - pick[t] < window for t in range(T)])
    assert hit[inside].float().mean() > 0.9 and ((~inside).sum() == 0 or hit[~inside].float().mean() < 0.1)
    for n, cuts in enumerate(CUT):
        if device == "cpu" and n % 2:
            continue
        got = LatentRows(spec, W, dtype, device, extra=64 * (n % 2)).walk(1, x, cuts)
        assert apart(got, want[:got.shape[0]]) < TOL[dtype], n


@pytest.mark.gpu
@pytest.mark.parametrize("H,d,rot,dv,kr,window", [c for c in LAT if c[1] % 8 == 0])
def test_windowed_latent_prompts_on_the_mma_kernel(H, d, rot, dv, kr, window, monkeypatch):
    from volta_engine_b200.ops import latent as L
    monkeypatch.setattr(L, "TC_PREFILL", False)
    test_every_row_finds_its_latent_inside_the_window_and_none_outside(H, d, rot, dv, kr, window, torch.bfloat16, "cuda")


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("scaling", [None, (1.0, 60, 5.0, 1.0), (16.0, 60, 5.0, 1.0), (40.0, 30, 2.0, 0.5)])
def test_the_factor_of_the_turns_is_on_the_turned_part_alone(scaling, dtype, device):
    T, (spec, m, W) = 90, lat_case(2, 16, 16, 24, 32, 50, scaling, seed=4, scale=0.5)
    x = rnd(T, 2 * 32 + 48, seed=6).to(torch.bfloat16).float()
    want = plain.latent_attention(W, "", m, x.double(), spec.eps)
    assert apart(LatentRows(spec, W, dtype, device).walk(0, x, [60, 2, 17, 1, 10]), want) < TOL[dtype]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
def test_latent_attention_of_a_mixed_batch(dtype, device):
    """Contexts of unequal sequences, cut to their windows, lie next to each other."""
    spec, m, W = lat_case(3, 40, 8, 24, 72, 33, seed=9)
    r = LatentRows(spec, W, dtype, device)
    seq = [(rnd(140, 3 * 48 + 80, seed=s) * 1.7).to(torch.bfloat16).float() for s in range(3)]
    want = [plain.latent_attention(W, "", m, s.double(), spec.eps) for s in seq]
    at = [0, 0, 0]
    for counts in ((1, 5, 100), (2, 3, 20), (1, 1, 1), (16, 40, 19), (0, 50, 1), (0, 1, 1)):
        order = sorted((i for i in range(3) if counts[i]), key=lambda i: counts[i])
        got = r.batch([(i, at[i], seq[i][at[i]:at[i] + counts[i]]) for i in order])
        assert apart(got, torch.cat([want[i][at[i]:at[i] + counts[i]] for i in order])) < TOL[dtype]
        for i in range(3):
            at[i] += counts[i]


@pytest.mark.gpu
@pytest.mark.parametrize("H,d,rot,dv,kr,window", [(2, 64, 32, 96, 64, 300), (1, 128, 64, 128, 512, 130), (2, 32, 16, 32, 40, 64)])
def test_latent_prompt_of_many_key_tiles(H, d, rot, dv, kr, window):
    spec, m, W = lat_case(H, d, rot, dv, kr, window, seed=3)
    T = 600
    x = (rnd(T, H * (d + rot) + kr + rot, seed=5) * 1.5).to(torch.bfloat16).float()
    want = plain.latent_attention(W, "", m, x.double(), spec.eps)
    for cuts in ([T], [1, 399, 200], [129, 127, 344], [400] + [1] * 200):
        assert apart(LatentRows(spec, W, torch.bfloat16, "cuda").walk(2, x, cuts), want) < 0.03


# ------------------------------------------------------------------------------------------ routers and experts
ROUTERS = [Router(18, 4, 3, 1), Router(12, 5, 3, 2), Router(7, 2), Router(40, 1, 8, 1), Router(64, 8, 8, 4), Router(5, 4, 5, 4), Router(6, 6, 2, 2), Router(300, 20, 10, 3),
           Router(1, 1), Router(1024, 32, 64, 7)]


def as_config(r):
    return {"experts": r.experts, "top": r.top, "groups": {"count": r.groups, "keep": r.keep}}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("r", ROUTERS, ids=lambda r: f"{r.top}of{r.experts}")
def test_routers(r, device):
    """Experts and weights of every row, best first; logits that reach far below and above."""
    z = rnd(37, r.experts, seed=r.experts, scale=2.0)
    z[5] *= 30.0
    z[6] += 500.0
    ids, w = route(r, z.to(device))
    for i in range(37):
        want = plain.choose(z[i].double(), as_config(r))
        live = [k for k, (_, s) in enumerate(want) if s > 1e-30]                    # scores that underflow are alike
        assert [int(ids[i, k]) for k in live] == [want[k][0] for k in live]
        assert all(abs(float(w[i, k]) - s) < 2e-6 * max(s, 1e-6) + 1e-9 for k, (_, s) in enumerate(want))
    assert int(ids.min()) >= 0 and int(ids.max()) < r.experts and all(len(set(row)) == r.top for row in ids.tolist())


@pytest.mark.parametrize("device", DEVICES)
def test_a_group_counts_by_its_best_member(device):
    """The group with the best expert wins against one whose sum is larger; an expert of a closed group is not taken however good."""
    z = torch.tensor([[5.0, 0.0, 0.0, 0.0, 4.9, 4.9, 4.9, 4.9], [1.0, 0.9, 0.8, 0.7, 3.0, -5.0, -5.0, -5.0]], device=device)
    ids, _ = route(Router(8, 2, 2, 1), z)
    assert int(ids[0, 0]) == 0 and set(ids[0].tolist()) <= {0, 1, 2, 3} and int(ids[1, 0]) == 4 and set(ids[1].tolist()) <= {4, 5, 6, 7}
    ids, w = route(Router(8, 2, 2, 1, best2=True, renorm=True, factor=2.5), z)
    assert set(ids[0].tolist()) <= {4, 5, 6, 7} and torch.allclose(w.sum(-1).cpu(), torch.tensor([2.5, 2.5]))


@pytest.mark.gpu
def test_a_row_of_nan_logits_still_gives_experts():
    z = torch.full((3, 24), float("nan"), device="cuda")
    z[1] = float("inf")
    z[2] = float("-inf")
    ids, _ = route(Router(24, 4, 4, 2), z)
    assert all(len(set(r)) == 4 and 0 <= min(r) and max(r) < 24 for r in ids.tolist())


def experts_case(r, width, ff, limit, seed=0):
    g, u, d = (rnd(r.experts, *s, seed=seed + i) * s[1] ** -0.5 for i, s in enumerate(((ff, width), (ff, width), (width, ff))))
    W = {"router": rnd(r.experts, width, seed=seed + 9) * 3.0 * width ** -0.5}
    for e in range(r.experts):
        W.update({f"e{e}.gate": g[e], f"e{e}.up": u[e], f"e{e}.down": d[e]})
    W = {n: t.to(torch.bfloat16).double() for n, t in W.items()}

    def pack(dtype, device):
        pad = lambda t: torch.nn.functional.pad(t, (0, -t.shape[-1] % 8)).to(device, dtype).contiguous()
        gu = torch.stack([torch.cat([W[f"e{e}.gate"], W[f"e{e}.up"]]) for e in range(r.experts)])
        return ExpertWeights(pad(gu), pad(torch.stack([W[f"e{e}.down"] for e in range(r.experts)])), ClampedGlu(limit, 1.702), ff)
    return W, {"expert": {"limit": limit}, "router": as_config(r)}, pack


EXP = [(Router(18, 4, 3, 1), 104, 40, 0.6), (Router(7, 2), 75, 19, 1.1), (Router(64, 8, 8, 4), 256, 88, 1.4), (Router(5, 4, 5, 4), 33, 130, 0.3), (Router(3, 3), 512, 8, 7.0),
       (Router(1, 1), 64, 64, 1.0), (Router(40, 1, 8, 1), 136, 264, 2.0), (Router(9, 8, 3, 3), 24, 6272, 1.0)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("r,width,ff,limit", EXP, ids=lambda v: f"{v.top}of{v.experts}" if isinstance(v, Router) else str(v))
def test_experts(r, width, ff, limit, dtype, device):
    """A few rows, and many; rows that all want the same expert; the router's logits are the plain statement's, so no close call differs."""
    W, m, pack = experts_case(r, width, ff, limit, seed=ff)
    ex = pack(dtype, device)
    for n in (1, 3, 16, 17, 45, 200):
        x = rnd(n, width, seed=n, scale=2.0)
        if n == 45:
            x[:] = x[0] + 0.01 * x
        x = x.to(torch.bfloat16)
        want = plain.routed_ff(W, "", m, x.double())
        z = (x.double() @ W["router"].T).float().to(device)
        xd = x.to(device, dtype)
        forms = {"fp32 out": lambda: routed_few(r, ex, z, xd.float(), torch.float32), "few": lambda: routed_few(r, ex, z, xd, dtype)} if device == "cuda" else \
            {"cpu": lambda: routed_reference(r, ex, z, xd, dtype)}
        if device == "cuda" and dtype == torch.bfloat16:
            forms["many"] = lambda: routed_many(r, ex, z, xd).tensor()
        for what, f in forms.items():
            assert apart(f(), want) < (1e-5 if dtype == torch.float32 else 0.02), (n, what)


# ------------------------------------------------------------------------------------------ row operators
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows,width", [(1, 64), (5, 75), (3, 2052), (40, 132), (2, 4096), (3, 8200), (17, 1024)])
@pytest.mark.parametrize("normed", [False, True])
def test_results_enter_the_residual_behind_their_norm(rows, width, normed, dtype, device):
    h, part = rnd(rows, width, seed=1, scale=3.0), rnd(rows, width, seed=2, scale=0.02).to(dtype)
    wa, wo = rnd(width, seed=3), rnd(width, seed=4)
    eps = 3e-4
    read = ResidualNorm(wo.to(device) if normed else None, eps)
    seen = lambda x: plain.rms_norm(x, wo.double(), eps) if normed else x
    hd = h.clone().to(device)
    close(read.rows(hd, dtype), seen(h.double()), dtype, f32=5e-6)
    assert torch.equal(hd.cpu(), h)
    x = h.double() + plain.rms_norm(part.double(), wa.double(), eps)
    close(read.rows(hd, dtype, part.to(device), NormedWrite(wa.to(device), eps)), seen(x), dtype, f32=5e-6)
    close(hd, x, torch.float32)


@pytest.mark.gpu
@pytest.mark.parametrize("rows,width,top", [(1, 64, 3), (30, 75, 1), (9, 1024, 8), (4, 2052, 5), (3, 8200, 2)])
def test_routed_results_are_summed_on_the_way_into_the_residual(rows, width, top):
    h, d = rnd(rows, width, seed=1), rnd(rows * top, width, seed=2).to(torch.bfloat16)
    inv, w = torch.randperm(rows * top, generator=torch.Generator().manual_seed(3)).reshape(rows, top).int(), rnd(rows, top, seed=4).abs()
    wa = rnd(width, seed=5)
    y = torch.stack([sum(w[i, k].double() * d[int(inv[i, k])].double() for k in range(top)) for i in range(rows)])
    x = h.double() + plain.rms_norm(y, wa.double(), 1e-5)
    hd = h.cuda()
    routed = RoutedRows(d.cuda(), inv.cuda(), w.cuda())
    close(ResidualNorm(None, 1e-5).rows(hd, torch.bfloat16, routed, NormedWrite(wa.cuda(), 1e-5)), x, torch.bfloat16)
    close(hd, x, torch.float32, f32=5e-6)
    close(routed.tensor(), y, torch.bfloat16)


@pytest.mark.gpu
@pytest.mark.parametrize("N,K,M", [(96, 64, 1), (1000, 2048, 1), (130, 75, 3), (2056, 1000, 8), (6000, 264, 5), (75, 4104, 4), (24, 320, 8)])
def test_decode_linear_that_adds_the_result_in_front(N, K, M):
    """y = W f(h + norm(result)) with the sum stored, as it is or normed; soft-capped; the gated unit behind it."""
    dev = "cuda"
    W = (rnd(N, K, seed=1) * K ** -0.5).to(torch.bfloat16)
    lin, Wd = LinearBF16(W.to(dev)), W.double()
    h, part, wa, wo = rnd(M, K, seed=2, scale=2.0), rnd(M, K, seed=3, scale=0.05), rnd(K, seed=4), rnd(K, seed=5)
    write = NormedWrite(wa.to(dev), 1e-4)

    def check(got, v, f=lambda e: e, tol=8e-3):
        e = f(v.float().to(torch.bfloat16).double() @ Wd.t())
        assert (got.double().cpu() - e).abs().max() < tol * e.pow(2).mean().sqrt() + 1e-6
    x = h.double() + plain.rms_norm(part.double(), wa.double(), 1e-4)
    for read, see in ((ResidualNorm(None, 1e-4), lambda v: v), (ResidualNorm(wo.to(dev), 1e-4), lambda v: plain.rms_norm(v, wo.double(), 1e-4))):
        check(gemv_rows(lin, M, out_f32=True, **read.prologue(h.to(dev))), see(h.double()))
        pro = read.prologue(h.to(dev), part.to(dev), write)
        check(gemv_rows(lin, M, out_f32=True, **pro), see(x))
        close(pro["h_out"], x, torch.float32, f32=5e-6)
        check(gemv_rows(lin, M, out_f32=True, cap=0.8, **read.prologue(h.to(dev), part.to(dev), write)), see(x), lambda e: plain.soft_cap(e, 0.8))
    if N % 16 == 0:
        blk = LinearBF16(ClampedGlu.interleave(W[:N // 2], W[N // 2:]).to(dev))
        got = gemv_rows(blk, M, **ResidualNorm(None, 1e-4).prologue(h.to(dev), part.to(dev), write), **ClampedGlu.silu(True).epilogue())
        z = x.float().to(torch.bfloat16).double() @ Wd.t()
        v = plain.dense_ff(pick_halves(N // 2), "", {}, z)
        assert got.shape == (M, N // 2) and (got.double().cpu() - v).abs().max() < 2e-2 * v.pow(2).mean().sqrt() + 2 ** -8 * v.abs().max()
    z = rnd(M, 2 * K, seed=6, scale=2)                                  # and in front of it
    v = plain.dense_ff(pick_halves(K), "", {}, z.double())
    check(gemv_rows(lin, M, out_f32=True, **ClampedGlu.silu().prologue(z.to(dev))), v)


def pick_halves(n):
    eye = torch.eye(n, dtype=torch.float64)
    return {"gate": torch.cat([eye, 0 * eye], 1), "up": torch.cat([0 * eye, eye], 1), "down": eye}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows,ff", [(1, 53), (7, 320), (30, 264)])
def test_gated_units(rows, ff, dtype, device):
    """silu(gate) up without bounds, and the clamped unit of the experts, from halves and from blocks."""
    z = rnd(rows, 2 * ff, seed=6, scale=4).to(dtype)
    z[0, 0], z[0, ff], z[-1, 1], z[-1, ff + 1] = -90.0, 50.0, 80.0, -70.0
    for unit, want in ((ClampedGlu.silu, plain.dense_ff(pick_halves(ff), "", {}, z.double())),
                       (lambda b=False: ClampedGlu(0.9, 1.702, b), plain.clamped_ff(pick_halves(ff), "", {"limit": 0.9}, z.double()))):
        close(unit().rows(z.to(device), dtype), want, dtype, f32=5e-6)
        if ff % 4 == 0:
            p = pick_halves(ff)
            zb = (z.float() @ ClampedGlu.interleave(p["gate"].float(), p["up"].float()).t()).to(dtype)
            close(unit(True).rows(zb.to(device), dtype), want, dtype, f32=5e-6)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("cap", [0.5, 7.0, 50.0])
def test_soft_caps(cap, device):
    x = rnd(5, 333, seed=1, scale=20.0)
    x[0, :4] = torch.tensor([0.0, 1e-4, -1e6, 1e6])
    close(soft_cap_(x.clone().to(device), cap), plain.soft_cap(x.double(), cap), torch.float32)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
def test_scaled_embeddings(dtype, device):
    t, ids = rnd(30, 75, seed=1).to(dtype), torch.tensor([3, 0, 29, 7, 7], dtype=torch.int32)
    for scale in (1.0, 12.0, 0.3):
        got = embed_rows(ids.to(device), t.to(device), scale=scale)
        assert got.dtype == torch.float32
        close(got, t[ids.long()].double() * scale, torch.float32)


def test_fp32_and_bf16_linears_of_a_tied_head_share_the_table():
    t = rnd(40, 64, seed=1)
    assert LinearF32(t).weight.data_ptr() == t.data_ptr() and LinearBF16(t.to(torch.bfloat16)).weight.shape == (40, 64)
    assert math.isinf(ClampedGlu.silu().limit)
