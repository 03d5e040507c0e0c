"""Every mechanism of the Vugipel decoder alone against the plain statement: attention with rotated values (one key per row that stands out:
just inside and just outside the window, among the first tokens and behind them, at page borders), soft caps, head factors, retention, the
gated recurrence per channel, sigmoid routers and experts weighed at their input, linears with biases, norms with offset weights."""
import pytest
import torch

import vugipel_plain as plain
from listed_util import DEVICES, Rows, one_thread, vars_of  # noqa: F401
from volta_engine_b200.ops.gqa import GqaSpec, gqa_attend
from volta_engine_b200.ops.linear import LinearBF16, LinearF32
from volta_engine_b200.ops.linear_attn import LinAttnSpec, LinAttnState, linattn_rows
from volta_engine_b200.ops.min_gru import MinGruState, min_gru_rows
from volta_engine_b200.ops.rotary import Rotation
from volta_engine_b200.ops.routed import ExpertWeights, Router, route, routed_few, routed_many, routed_reference
from volta_engine_b200.ops.rowops import ClampedGlu, GroupRMS, ResidualNorm, RoutedRows, gemv_rows
from volta_engine_b200.runtime.batch import BatchRows

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


# ------------------------------------------------------------------------------------------ attention
def att_case(H, G, d, dv, window, first, dims, base=500.0, scale=None, cap=18.0, seed=0):
    """-> (spec on the CPU, mixer dictionary, weights of the plain statement: projections that select columns)."""
    wq, wk, temp = (1.0 + 0.3 * rnd(n, seed=seed + i) for i, n in enumerate((d, d, H)))
    spec = GqaSpec(H, G, d, dv, scale or d ** -0.5, 1e-5, q_norm=wq, k_norm=wk, norm_first=True, head_mul=temp, softcap=cap, window=window, keep_first=first,
                   rot=Rotation(dims, base, True), v_rot=Rotation(dv, base, True))
    eye = torch.eye(spec.cols, dtype=torch.float64)
    W = {"q": eye[:H * d], "k": eye[H * d:(H + G) * d], "v": eye[(H + G) * d:], "q.norm": wq.double(), "k.norm": wk.double(), "temp": temp.double(),
         "o": torch.eye(H * dv, dtype=torch.float64)}
    W.update({n + ".b": torch.zeros(W[n].shape[0], dtype=torch.float64) for n in ("q", "k", "v", "o")})
    return spec, {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": spec.scale, "softcap": cap, "mask": {"size": window, "keep_first": first},
                  "rot": {"dims": dims, "base": base}}, W


class AttnRows(Rows):
    def __init__(self, spec, dtype, device, extra=0):
        super().__init__(dtype, device, *spec.row_widths, extra)
        move = lambda t: None if t is None else t.to(device)
        turn = lambda r: None if r is None else Rotation(r.dims, r.base, r.neighbours).bind(device)
        self.spec = GqaSpec(**dict(vars_of(spec), q_norm=move(spec.q_norm), k_norm=move(spec.k_norm), head_mul=move(spec.head_mul), rot=turn(spec.rot), v_rot=turn(spec.v_rot)))

    def run(self, b, x):
        x = torch.nn.functional.pad(x, (0, 3)).to(self.device)                        # columns of something else behind it
        w = self.spec.heads * self.spec.vdim
        y = torch.full((b.n, w + 8), 5.0, dtype=self.dtype, device=self.device)
        gqa_attend(self.spec, x, b, self.kv, self.kv.k[1], self.kv.v[1], y[:, :w])
        assert bool((y[:, w:] == 5.0).all())
        return y[:, :w].float().cpu()


ATT = [(4, 2, 24, 40, 37, 5, 16), (3, 3, 21, 14, 19, 0, 10), (8, 2, 128, 128, 64, 64, 128), (18, 1, 16, 8, 65, 1, 2), (2, 1, 64, 136, 100, 70, 64),
       (1, 1, 264, 24, 50, 3, 100), (5, 5, 8, 64, 1, 2, 8), (6, 3, 32, 24, 128, 4, 12), (4, 1, 40, 16, 3, 130, 24), (2, 2, 200, 128, 129, 63, 8),
       (4, 2, 64, 64, 1000, 9, 2), (12, 4, 72, 6, 16, 17, 72), (2, 1, 96, 100, 30, 8, 96)]
CUT = [[210], [64, 64, 82], [1] * 10 + [60, 16, 2, 41, 1, 1, 15, 17] + [1] * 47, [130] + [2] * 40]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("H,G,d,dv,window,first,dims", ATT)
def test_every_row_finds_its_key_in_sight_and_none_out_of_it(H, G, d, dv, window, first, dims, dtype, device):
    """A row's query is lined up with one key: itself, the row before, the last key its window keeps, the first one that it does not, the last
    of the first tokens that stay and the one behind it, keys at page borders. Keys in sight give their value, the others nothing."""
    T, (spec, m, W) = 210, att_case(H, G, d, dv, window, first, dims, seed=H + d)
    spec.scale = m["scale"] = 24.0 / d                                  # |q| |k| about d: a score that the cap leaves standing out
    spec.head_mul = torch.ones(H)
    spec.q_norm, spec.k_norm = torch.ones(d), 1.0 + 0.3 * rnd(d, seed=d)
    W.update({"temp": torch.ones(H).double(), "q.norm": torch.ones(d).double(), "k.norm": spec.k_norm.double()})
    x = rnd(T, spec.cols, seed=5)
    choice = lambda t: [t, first - 1, t - 1, t - window + 1, first, t - window, t // 64 * 64, 0, t // 64 * 64 - 1, t - window // 2, t - window - 1][t % 11]
    pick = [max(0, min(t, choice(t))) for t in range(T)]
    k = plain.over_rms(x[:, H * d:(H + G) * d].reshape(T, G, d).double(), 1e-5) * W["k.norm"]
    k = k.repeat_interleave(H // G, 1)
    x[:, :H * d] = plain.turn_pairs(k[pick], [p - t for t, p in enumerate(pick)], m["rot"]["base"], dims).reshape(T, H * d).float()      # turned by the difference
    x = x.to(torch.bfloat16).float()
    want = plain.rotated_value_attention(W, "", m, x.double(), spec.eps)
    if d >= 16:
        v = x[:, (H + G) * d:].reshape(T, G, dv).repeat_interleave(H // G, 1).double()
        near = plain.turn_pairs(v[pick], [p - t for t, p in enumerate(pick)], m["rot"]["base"], dv).reshape(T, -1)
        hit = (want - near).norm(dim=1) < 0.5 * near.norm(dim=1)
        inside = torch.tensor([t - pick[t] < window or pick[t] < first for t in range(T)])
        assert hit[inside].float().mean() > 0.9 and ((~inside).sum() == 0 or hit[~inside].float().mean() < 0.1)
    for n, cuts in enumerate(CUT):
        if device == "cpu" and n % 2:
            continue
        got = AttnRows(spec, dtype, device, extra=40 * (n % 2)).walk(1, x, cuts)
        assert apart(got, want[:got.shape[0]]) < TOL[dtype], n


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("cap,size", [(0.2, 1.0), (3.0, 1.0), (20.0, 30.0), (5.0, 3000.0), (1e4, 1.0)])
def test_soft_caps_of_scores(cap, size, dtype, device):
    """Scores far below the cap, around it and far above on both sides; heads whose factor is negative, zero or large."""
    T, (spec, m, W) = 150, att_case(4, 2, 32, 24, 90, 3, 16, seed=2, cap=cap, scale=size * 32 ** -0.5)
    spec.head_mul = torch.tensor([1.3, -0.7, 0.0, 6.0])
    W["temp"] = spec.head_mul.double()
    x = rnd(T, spec.cols, seed=3).to(torch.bfloat16).float()
    want = plain.rotated_value_attention(W, "", m, x.double(), spec.eps)
    for cuts in ([T], [1] * 3 + [100] + [1] * 47):
        got = AttnRows(spec, dtype, device).walk(2, x, cuts)
        # saturated scores flip with the sign of a product near zero: those rows are judged by their mean
        e = (got.double() - want).abs() / want.abs().max()
        assert (e.mean() if size > 1000 and dtype == torch.bfloat16 else e.max()) < (3e-4 if size > 1000 and dtype == torch.float32 else TOL[dtype])


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("dv", [24, 18, 72])
def test_values_turn_in_either_layout(dv, dtype, device):
    """Pairs half the width apart equal neighbouring pairs of shuffled columns; also without rotated queries and keys."""
    T, H, G, d = 160, 3, 1, 16
    halves = lambda n: torch.cat([torch.arange(0, n, 2), torch.arange(1, n, 2)])      # where a column of the halved layout comes from
    spec, m, W = att_case(H, G, d, dv, 40, 4, d, seed=7)
    x = rnd(T, spec.cols, seed=1).to(torch.bfloat16).float()
    want = plain.rotated_value_attention(W, "", m, x.double(), spec.eps)
    shuffle = torch.cat([i * d + halves(d) for i in range(H + G)] + [(H + G) * d + i * dv + halves(dv) for i in range(G)])
    other = GqaSpec(**dict(vars_of(spec), q_norm=spec.q_norm[halves(d)], k_norm=spec.k_norm[halves(d)], rot=Rotation(d, 500.0, False), v_rot=Rotation(dv, 500.0, False)))
    back = torch.cat([i * dv + halves(dv) for i in range(H)])
    for cuts in ([T], [100] + [1] * 60):
        got = AttnRows(other, dtype, device).walk(0, x[:, shuffle], cuts)
        assert apart(got, want[:, back]) < TOL[dtype]
    still = GqaSpec(**dict(vars_of(spec), rot=None))
    want = plain.rotated_value_attention(W, "", dict(m, rot={"dims": 0, "base": 500.0}), x.double(), spec.eps)
    assert apart(AttnRows(still, dtype, device).walk(0, x, [T]), want) < TOL[dtype]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
def test_small_queries_and_keys_see_eps_inside_the_root(dtype, device):
    T, (spec, m, W) = 40, att_case(2, 1, 16, 8, 30, 2, 16, scale=0.7)
    x = rnd(T, spec.cols, seed=4)
    x[:, :3 * 16] *= 3e-3
    x = x.to(torch.bfloat16).float()
    want = plain.rotated_value_attention(W, "", m, x.double(), spec.eps)
    assert apart(AttnRows(spec, dtype, device).walk(0, x, [25, 1, 14]), want) < TOL[dtype]
    spec.eps = 1e-9                                                     # it matters here
    assert apart(AttnRows(spec, torch.float32, "cpu").walk(0, x, [T]), want) > 0.01


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
def test_attention_of_a_mixed_batch(dtype, device):
    spec, m, W = att_case(6, 2, 40, 24, 33, 6, 40, seed=9, scale=0.6)
    r = AttnRows(spec, dtype, device)
    seq = [(rnd(140, spec.cols, seed=s) * 1.5).to(torch.bfloat16).float() for s in range(3)]
    want = [plain.rotated_value_attention(W, "", m, s.double(), spec.eps) for s in seq]
    at = [0, 0, 0]
    for counts in ((1, 5, 100), (2, 3, 20), (1, 1, 1), (16, 40, 3), (0, 80, 1), (0, 1, 1)):
        order = sorted((i for i in range(3) if counts[i]), key=lambda i: counts[i])
        got = r.batch([(i, at[i], seq[i][at[i]:at[i] + counts[i]]) for i in order])
        assert apart(got, torch.cat([want[i][at[i]:at[i] + counts[i]] for i in order])) < TOL[dtype]
        for i in range(3):
            at[i] += counts[i]


@pytest.mark.gpu
@pytest.mark.parametrize("H,G,d,dv,window,first", [(4, 1, 128, 128, 300, 70), (3, 3, 64, 64, 64, 128), (2, 1, 256, 128, 511, 1), (6, 2, 40, 72, 130, 200), (4, 2, 128, 64, 5000, 5)])
def test_prompt_of_many_pages(H, G, d, dv, window, first):
    """First tokens and windows of several pages: both streams, all ring stages, tiles that start anywhere; long decoding behind it."""
    spec, m, W = att_case(H, G, d, dv, window, first, d, seed=3, scale=3.0 / d ** 0.5, base=1e4)
    T = 700
    x = rnd(T, spec.cols, seed=5).to(torch.bfloat16).float()
    want = plain.rotated_value_attention(W, "", m, x.double(), spec.eps)
    for cuts in ([T], [1, 399, 300], [129, 127, 444], [400] + [1] * 300):
        assert apart(AttnRows(spec, torch.bfloat16, "cuda").walk(2, x, cuts), want) < 0.03


@pytest.mark.parametrize("device", DEVICES)
def test_cached_values_are_those_turned_by_their_position(device):
    """Far positions: angles are exact there too."""
    d, dv, at = 16, 24, 900
    spec, m, W = att_case(2, 1, d, dv, 16, 0, d, base=1e4)
    r = AttnRows(spec, torch.float32, device)
    x = rnd(3, spec.cols, seed=2)
    r.batch([(0, at, x)])
    page = int(r.kv.page_table[0, at // 64])
    v = r.kv.v[1][page].reshape(-1)[: 64 * dv].reshape(64, dv)[at % 64: at % 64 + 3]
    close(v, plain.turn_pairs(x[:, None, 3 * d:].double(), range(at, at + 3), 1e4, dv)[:, 0], torch.float32)


# ------------------------------------------------------------------------------------------ retention
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("H,dk,dv", [(4, 64, 64), (1, 16, 48), (3, 128, 80), (2, 9, 21), (2, 200, 33), (2, 96, 136), (5, 32, 32)])
def test_retention_in_portions(H, dk, dv, chunked, device):
    """A long sequence in portions of all kinds beside a second one, in slots that hold another sequence's state before; heads that never
    forget, and one that forgets at once."""
    decay = torch.tensor([1.0, 0.9, 0.0, 0.999, 0.5][:H])
    spec = LinAttnSpec(H, dk, dv, decay=decay.to(device), plain=True, q_scale=dk ** -0.5)
    st = LinAttnState(spec, 3, device)
    st.rec.fill_(7.0)
    a, b = (rnd(n, spec.cols + H * dv, seed=n, scale=1.5) for n in (330, 90))
    eye = torch.eye(spec.cols + H * dv, dtype=torch.float64)
    W = {"q": eye[:H * dk], "k": eye[H * dk:2 * H * dk], "v": eye[2 * H * dk:spec.cols], "g": eye[spec.cols:], "o": torch.eye(H * dv, dtype=torch.float64)}
    m = {"heads": H, "dim": dk, "vdim": dv, "decay": decay.tolist()}
    wa, wb = (plain.retention(W, "", m, x.double(), 1e-5) for x in (a, b))
    norm = GroupRMS(torch.ones(dv, device=device), 1e-5, dv, silu=True)
    got_a, got_b, at, bt = [], [], 0, 0
    for na, nb in ((1, 0), (64, 1), (2, 0), (100, 40), (63, 3), (17, 16), (1, 1), (16, 0), (65, 29), (1, 0)):
        ids = list(range(at, at + na)) + list(range(bt, bt + nb))
        batch = BatchRows.make(ids, ids, [2] * na + [0] * nb, device)
        proj = torch.cat([a[at:at + na], b[bt:bt + nb]]).to(device)
        o = norm.rows(linattn_rows(proj, batch, st, spec, chunked=chunked), torch.float32, gate=proj[:, spec.cols:])
        got_a.append(o[:na].cpu())
        got_b.append(o[na:].cpu())
        at, bt = at + na, bt + nb
    for got, want in ((torch.cat(got_a), wa), (torch.cat(got_b), wb)):
        e = (got.double() - want).abs() / (want.abs() + want.pow(2).mean().sqrt())
        # the chunked form rounds the values to bf16; a head without memory whose sum nearly vanishes is normed all the same
        assert (e.quantile(0.999) if chunked else e.max()) < (0.02 if chunked else 1e-3) and e.mean() < (3e-3 if chunked else 1e-5)
    assert bool((st.rec[1] == 7.0).all())         # the slot nobody used


# ------------------------------------------------------------------------------------------ the gated recurrence per channel
def gru_weights(width):
    eye = torch.eye(3 * width, dtype=torch.float64)
    zero = torch.zeros(width, dtype=torch.float64)
    return {"z": eye[:width], "x": eye[width:2 * width], "g": eye[2 * width:], "z.b": zero, "x.b": zero, "o": eye[:width, :width]}


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("width,pad", [(1, 0), (8, 8), (53, 3), (64, 0), (65, 7), (200, 0), (1030, 2)])
def test_recurrence_per_channel_in_portions(width, pad, dtype, device):
    """Portions of all kinds beside a second sequence, in slots with an earlier request's state; gates that are shut, open and in between,
    candidates on both sides of the bend and far out."""
    a, b = (rnd(n, 3 * width + 5, seed=n, scale=2.0) for n in (500, 90))
    a[:, :width:3] -= 9.0                         # channels that remember everything
    a[100:110, :width] = 90.0                     # rows that replace the state, rows that leave it alone
    a[200:210, :width] = -120.0
    a[300, width:2 * width], a[301, width:2 * width], a[302, width:2 * width] = 0.0, -100.0, 1e4
    W = gru_weights(width)
    wa, wb = (plain.min_gru(W, "", {"width": width}, x[:, :3 * width].double(), 1e-5) for x in (a, b))
    st = MinGruState(width, 3, device)
    st.rec.fill_(7.0)
    got_a, got_b, at, bt = [], [], 0, 0
    for na, nb in ((1, 0), (64, 1), (2, 0), (129, 40), (63, 3), (17, 16), (1, 1), (16, 0), (200, 29), (7, 0)):
        ids = list(range(at, at + na)) + list(range(bt, bt + nb))
        rows = sorted([(na, 2, at), (nb, 0, bt)])                                     # shortest first
        order = [(s, p0 + i) for n, s, p0 in rows for i in range(n)]
        batch = BatchRows.make([p for _, p in order], [p for _, p in order], [s for s, _ in order], device)
        proj = torch.cat([(a if s == 2 else b)[p0:p0 + n] for n, s, p0 in rows]).to(device)
        assert len(ids) == proj.shape[0]
        y = min_gru_rows(proj, batch, st, dtype, width + pad).cpu()
        assert y.shape[1] == width + pad and bool((y[:, width:] == 0).all())
        slot = torch.tensor([s for s, _ in order])
        got_a.append(y[slot == 2, :width])
        got_b.append(y[slot == 0, :width])
        at, bt = at + na, bt + nb
    for got, want in ((torch.cat(got_a), wa), (torch.cat(got_b), wb)):
        assert got.dtype == dtype
        e = (got.double() - want).abs() / (want.abs() + 1e-2)
        assert e.max() < (2e-5 if dtype == torch.float32 else 6e-3)
    assert bool((st.rec[1] == 7.0).all())


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("counts", [[2048], [1, 700], [40, 41, 300], [16, 16, 16], [5, 130]])
def test_long_portions_start_where_the_ones_before_ended(counts, device):
    """Chunks of every length, several segments in one batch: each goes on from its own slot's state, twice in a row."""
    width = 70
    W = gru_weights(width)
    st = MinGruState(width, len(counts), device)
    seqs = [rnd(2 * n, 3 * width, seed=i + 1, scale=1.5) for i, n in enumerate(counts)]
    want = [plain.min_gru(W, "", {"width": width}, s.double(), 1e-5) for s in seqs]
    for part in range(2):
        order = [(s, part * n + i) for s, n in enumerate(counts) for i in range(n)]
        batch = BatchRows.make([p for _, p in order], [p for _, p in order], [s for s, _ in order], device)
        y = min_gru_rows(torch.cat([s[part * n:(part + 1) * n] for s, n in zip(seqs, counts)]).to(device), batch, st, torch.float32)
        close(y, torch.cat([w[part * n:(part + 1) * n] for w, n in zip(want, counts)]), torch.float32, f32=1e-5)


@pytest.mark.gpu
def test_rows_of_no_slot_and_rows_of_one_slot_in_a_step():
    """Padding rows give zeros and touch no state; several rows of a slot in one step follow each other."""
    width, W = 40, gru_weights(40)
    x = rnd(9, 120, seed=3)
    st = MinGruState(width, 2, "cuda")
    st.rec.fill_(3.0)
    b = BatchRows.make([0] * 9, [0, 0, 1, 0, 2, 0, 3, 0, 4], [1, -1, 1, -1, 1, -1, 1, -1, 1], "cuda")
    y = min_gru_rows(x.cuda(), b, st, torch.float32).cpu()
    close(y[::2], plain.min_gru(W, "", {"width": width}, x[::2].double(), 1e-5), torch.float32, f32=1e-5)
    assert bool((y[1::2] == 0).all()) and bool((st.rec[0] == 3.0).all())


# ------------------------------------------------------------------------------------------ routers and experts
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("experts,top", [(13, 1), (7, 2), (40, 8), (1, 1), (6, 6), (300, 20), (1024, 32)])
def test_sigmoid_routers(experts, top, device):
    """Experts and weights of every row, best first; every weight is the sigmoid of its own logit, whatever the others are."""
    z = rnd(37, experts, seed=experts, scale=1.5)
    z[5] -= 20.0
    z[6] *= 0.1
    z[7] += 30.0                                                        # every sigmoid rounds to one: the logits still tell them apart
    ids, w = route(Router(experts, top, sigmoid=True, weigh_input=True), z.to(device))
    for i in range(37):
        want = plain.choose(z[i].double(), {"top": top})
        if i == 7:
            want = [(e, 1.0) for e in torch.sort(z[i], descending=True).indices[:top].tolist()]
        assert ids[i].tolist() == [e for e, _ in want]
        assert all(abs(float(w[i, k]) - s) < 2e-6 * s for k, (_, s) in enumerate(want))


@pytest.mark.gpu
def test_a_row_of_nan_logits_still_gives_experts():
    z = torch.full((3, 24), float("nan"), device="cuda")
    z[1] = float("inf")
    z[2] = float("-inf")
    ids, _ = route(Router(24, 4, sigmoid=True), z)
    assert all(len(set(r)) == 4 and 0 <= min(r) and max(r) < 24 for r in ids.tolist())


EXP = [(18, 4, 104, 40), (7, 2, 75, 19), (64, 8, 256, 88), (13, 1, 120, 264), (3, 3, 512, 8), (1, 1, 64, 64), (5, 4, 33, 130), (9, 8, 24, 6272)]


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("experts,top,width,ff", EXP)
def test_experts_weighed_at_their_input(experts, top, width, ff, dtype, device):
    """A few rows, and many; weights far below one, where the unit is not linear; rows that all want the same expert."""
    r = Router(experts, top, sigmoid=True, weigh_input=True)
    W = {"router": rnd(experts, width, seed=ff + 9) * 2.0 * width ** -0.5}
    for e in range(experts):
        W.update({f"e{e}.{n}": rnd(*s, seed=ff + 3 * e + i) * s[1] ** -0.5 for i, (n, s) in enumerate((("gate", (ff, width)), ("up", (ff, width)), ("down", (width, ff))))})
    W = {n: t.to(torch.bfloat16).double() for n, t in W.items()}
    pad = lambda t: torch.nn.functional.pad(t, (0, -t.shape[-1] % 8)).to(device, dtype).contiguous()
    gu = torch.stack([torch.cat([W[f"e{e}.gate"], W[f"e{e}.up"]]) for e in range(experts)])
    ex = ExpertWeights(pad(gu), pad(torch.stack([W[f"e{e}.down"] for e in range(experts)])), ClampedGlu.silu(), ff)
    m = {"router": {"top": top}}
    for n in (1, 3, 16, 17, 45, 200):
        x = rnd(n, width, seed=n, scale=2.0)
        if n == 45:
            x[:] = x[0] + 0.01 * x
        x = x.to(torch.bfloat16)
        want = plain.routed_ff(W, "", m, x.double())
        assert apart(plain.routed_ff({**W, **{k: 0 * v for k, v in W.items() if k.endswith(".up")}}, "", m, x.double()), want) > 0.5
        z = (x.double() @ W["router"].T).float().to(device)
        xd = x.to(device, dtype)
        base = rnd(n, width, seed=n + 1)

        def into_residual():
            h = base.clone().to(device)
            assert routed_few(r, ex, z, xd, residual=h) is None
            return h.cpu() - base
        forms = {"fp32 out": lambda: routed_few(r, ex, z, xd.float(), torch.float32), "few": lambda: routed_few(r, ex, z, xd, dtype), "residual": into_residual} \
            if device == "cuda" else {"cpu": lambda: routed_reference(r, ex, z, xd, dtype)}
        if device == "cuda" and dtype == torch.bfloat16:
            forms["many"] = lambda: routed_many(r, ex, z, xd).tensor()
        for what, f in forms.items():
            assert apart(f(), want) < (1e-5 if dtype == torch.float32 else 0.02), (n, what)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("ff", [53, 264])
def test_a_unit_of_weighed_rows(ff, dtype, device):
    z, w = rnd(30, 2 * ff, seed=6, scale=3).to(dtype), torch.rand(30, generator=torch.Generator().manual_seed(1))
    index = torch.randperm(30, generator=torch.Generator().manual_seed(2)).int()
    v = z.double() * w.double()[index.long()][:, None]
    want = plain.silu(v[:, :ff]) * v[:, ff:]
    close(ClampedGlu.silu().rows(z.to(device), dtype, (w.to(device), index.to(device))), want, dtype, f32=5e-6)


# ------------------------------------------------------------------------------------------ linears, norms
@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("N,K,M", [(96, 64, 1), (130, 75, 3), (1000, 2048, 8), (75, 4104, 4), (24, 320, 16), (256, 192, 200), (300, 104, 130), (77, 33, 1000), (64, 6600, 12)])
def test_linears_with_biases(N, K, M, device):
    """Few rows and many, in 16 and 32 bits; the bias is added before anything is rounded."""
    W, x, b = (rnd(N, K, seed=1) * K ** -0.5).to(torch.bfloat16), rnd(M, K, seed=2).to(torch.bfloat16), rnd(N, seed=3, scale=3.0)
    want = x.double() @ W.double().t() + b.double()
    lin = LinearBF16(W.to(device), b.to(device))
    close(lin.forward(x.to(device), out_f32=True), want, torch.float32, f32=1e-5)
    close(lin.forward(x.to(device)), want, torch.bfloat16)
    close(LinearF32(W.float().to(device), b.to(device)).forward(x.float().to(device)), want, torch.float32, f32=1e-5)
    if device == "cuda" and M <= 16:
        close(gemv_rows(lin, M, x=x.cuda(), out_f32=True), want, torch.float32, f32=1e-5)
        h = rnd(M, N, seed=4)
        hd = h.cuda()
        assert gemv_rows(lin, M, x=x.cuda(), residual=(hd, None)) is None
        close(hd, h.double() + want, torch.float32, f32=1e-5)


@pytest.mark.gpu
@pytest.mark.parametrize("N,K,M", [(96, 64, 1), (130, 75, 3), (2056, 1000, 8), (24, 320, 8), (600, 2048, 2)])
def test_decode_linear_behind_a_norm_keeps_the_row_it_read(N, K, M):
    """The normed row enters the product and is stored for whoever reads it next."""
    W, h, w, b = (rnd(N, K, seed=1) * K ** -0.5).to(torch.bfloat16), rnd(M, K, seed=2, scale=2.0), rnd(K, seed=5, scale=0.2), rnd(N, seed=6)
    x = plain.centred_norm(h.double(), w.double(), 1e-4)
    kept = torch.full((M, K), 9.0, dtype=torch.bfloat16, device="cuda")
    got = gemv_rows(LinearBF16(W.cuda(), b.cuda()), M, out_f32=True, x_out=kept, **ResidualNorm((1.0 + w).cuda(), 1e-4).prologue(h.cuda()))
    close(kept, x, torch.bfloat16)
    close(got, kept.double().cpu() @ W.double().t() + b.double(), torch.float32, f32=1e-5)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("dtype", TYPES)
@pytest.mark.parametrize("rows,width", [(1, 64), (5, 75), (3, 2052), (40, 132), (2, 4096), (3, 8200), (17, 1024)])
def test_results_enter_the_residual_as_they_are(rows, width, dtype, device):
    h, part, w = rnd(rows, width, seed=1, scale=3.0), rnd(rows, width, seed=2, scale=2.0).to(dtype), rnd(width, seed=4, scale=0.3)
    read = ResidualNorm((1.0 + w).to(device), 3e-4)
    hd = h.clone().to(device)
    close(read.rows(hd, dtype), plain.centred_norm(h.double(), w.double(), 3e-4), dtype, f32=5e-6)
    assert torch.equal(hd.cpu(), h)
    x = h.double() + part.double()
    close(read.rows(hd, dtype, part.to(device)), plain.centred_norm(x, w.double(), 3e-4), dtype, f32=5e-6)
    close(hd, x, torch.float32)
    tiny = 1e-3 * rnd(rows, width, seed=6)                              # eps counts inside the root
    close(read.rows(tiny.clone().to(device), dtype), plain.centred_norm(tiny.double(), w.double(), 3e-4), dtype, f32=5e-6)


@pytest.mark.parametrize("device", DEVICES)
@pytest.mark.parametrize("rows,width,top", [(1, 64, 1), (30, 75, 1), (9, 1024, 8), (4, 2052, 5), (3, 8200, 2)])
def test_routed_results_without_weights_are_summed_into_the_residual(rows, width, top, device):
    h, d = rnd(rows, width, seed=1), rnd(rows * top, width, seed=2).to(torch.bfloat16)
    inv = torch.randperm(rows * top, generator=torch.Generator().manual_seed(3)).reshape(rows, top).int()
    w = rnd(width, seed=5, scale=0.3)
    x = h.double() + torch.stack([sum(d[int(inv[i, k])].double() for k in range(top)) for i in range(rows)])
    hd = h.clone().to(device)
    got = ResidualNorm((1.0 + w).to(device), 1e-5).rows(hd, torch.bfloat16, RoutedRows(d.to(device), inv.to(device)))
    close(got, plain.centred_norm(x, w.double(), 1e-5), torch.bfloat16, bf16=2 ** -6)
    close(hd, x, torch.float32, f32=5e-6 if device == "cuda" else 2 ** -7)
