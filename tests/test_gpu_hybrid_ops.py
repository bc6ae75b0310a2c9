"""Every kernel of the hybrid stacks alone against the plain restatement, in fp32 and bf16, at sizes, page borders, window
edges, chunk edges and slot states where a mistake shows."""
import pytest
import torch

from oracle import hybrid_reference as R

pytestmark = pytest.mark.gpu
DEV = "cuda"
DT = {"f32": torch.float32, "bf16": torch.bfloat16}


def rnd(*shape, seed, dtype=torch.float32, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype)


def close(got, want, dtype, what="", factor=1.0):
    got, want = got.double().cpu(), want.double().cpu()
    err = (got - want).abs().max() / want.abs().max().clamp_min(1e-9)
    tol = factor * (3e-6 if dtype == torch.float32 else 1.2e-2)
    assert torch.isfinite(got).all() and err < tol, f"{what}: {float(err):.2e} > {tol:.2e}"


@pytest.fixture(scope="module")
def hops():
    from b200attn import hybrid_ops
    return hybrid_ops


class Batch:
    """What the recurrent kernels read of a packed batch."""

    def __init__(self, slots, starts, lengths):
        self.count, self.max_len = len(slots), max(lengths)
        self.cu = torch.tensor([0] + list(torch.tensor(lengths).cumsum(0)), dtype=torch.int32, device=DEV)
        self.slots = torch.tensor(slots, dtype=torch.int32, device=DEV)
        self.start = torch.tensor(starts, dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------------------------------------------------- streams
@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("s,width,true", [(1, 64, 64), (2, 192, 136), (3, 256, 256), (4, 2048, 2000), (5, 64, 7), (16, 128, 128),
                                          (2, 6144, 6144)])
def test_hyper_connect(hops, dt, s, width, true):
    dtype, rows, eps = DT[dt], 9, 1e-4
    x = rnd(rows, s, width, seed=1)
    y = rnd(rows, width, seed=2, dtype=dtype)
    x[..., true:] = 0
    y[:, true:] = 0
    mix, out, into, gain = rnd(s, s, seed=3), rnd(s, seed=4), rnd(s, seed=5), torch.tensor([1.7])
    weights = torch.cat((mix.flatten(), out, into, gain)).to(DEV)
    w = {"in": torch.zeros(s).double(), "out": out.double(), "mix": mix.double()}
    want = R.hyper_connect(x.double().transpose(0, 1), w, "", lambda u: y.double())
    u = torch.einsum("s,stw->tw", into.double(), want)
    h_want = R.rms(u[:, :true], eps) * 1.7
    streams = x.to(DEV)
    h = hops.hyper_connect(streams, weights, true, eps, dtype, y=y.to(DEV))
    close(streams.transpose(0, 1), want, torch.float32, "streams")
    close(h[:, :true], h_want, dtype, "read-out")
    assert not h[:, true:].any()
    # embedding form, int32 and int64 ids
    table = rnd(11, width, seed=6, dtype=dtype)
    for idt in (torch.int32, torch.int64):
        ids = torch.tensor([3, 10, 0, 3, 5, 1, 2, 9, 7], dtype=idt, device=DEV)
        streams = torch.full((rows, s, width), 9.0, device=DEV)
        hops.hyper_connect(streams, weights, true, eps, dtype, ids=ids, table=table.to(DEV))
        assert torch.equal(streams.cpu(), table.float()[ids.cpu().long()][:, None].expand(rows, s, width))


def test_swiglu_f32(hops):
    gu = rnd(5, 2 * 136, seed=1, scale=4.0)
    got = hops.swiglu_f32(gu.to(DEV), 136)
    close(got, R.silu(gu[:, :136].double()) * gu[:, 136:].double(), torch.float32)


# -------------------------------------------------------------------------------------------------------- recurrences
def _mingru_want(zxg, bias, width, state0):
    z = R.sigmoid(zxg[:, :width].double() + bias[:width].double())
    u = zxg[:, width: 2 * width].double() + bias[width:].double()
    c = torch.where(u >= 0, u + 0.5, R.sigmoid(u))
    s, out = state0.double(), []
    for t in range(zxg.shape[0]):
        s = (1 - z[t]) * s + z[t] * c[t]
        out.append(s)
    return torch.stack(out) * R.silu(zxg[:, 2 * width:].double()), s


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("lengths", [[1], [2, 15, 16, 17], [127, 128, 129], [128, 1, 300], [4097]])
@pytest.mark.parametrize("segments", [None, (10 ** 6, 1), (64, 65), (256, 17)])
def test_mingru_prefill(hops, dt, lengths, segments):
    dtype, width = DT[dt], 68
    zxg = rnd(sum(lengths), 3 * width, seed=5, dtype=dtype, scale=2.0)
    zxg[:, :width] -= 3.0                                   # gates that keep most of the state: far tokens matter
    bias = rnd(2 * width, seed=6)
    slots = [3, 0, 5, 1][: len(lengths)]
    starts = [0, 7, 0, 40][: len(lengths)]
    before = rnd(6, width, seed=7, scale=3.0)
    state = before.to(DEV)
    out = hops.mingru_prefill(zxg.to(DEV), bias.to(DEV), state, Batch(slots, starts, lengths), segments=segments)
    row = 0
    for slot, start, n in zip(slots, starts, lengths):
        want, last = _mingru_want(zxg[row: row + n], bias, width, before[slot] if start else torch.zeros(width))
        close(out[row: row + n], want, dtype, f"length {n}", 2.0)
        close(state[slot], last, torch.float32, f"state after {n}", 1.0 if dt == "f32" else 4.0)
        row += n
    for slot in set(range(6)) - set(slots):
        assert torch.equal(state[slot].cpu(), before[slot])


@pytest.mark.parametrize("dt", DT)
def test_mingru_decode(hops, dt):
    dtype, width, rows = DT[dt], 132, 5
    zxg, bias, before = rnd(rows, 3 * width, seed=1, dtype=dtype), rnd(2 * width, seed=2), rnd(rows, width, seed=3)
    pos = torch.tensor([0, 5, 1, 9, 3], device=DEV)
    active = torch.tensor([1, 1, 0, 1, 1], device=DEV)
    state = before.to(DEV)
    out = hops.mingru_decode(zxg.to(DEV), bias.to(DEV), state, pos, active)
    for b in range(rows):
        want, last = _mingru_want(zxg[b: b + 1], bias, width, before[b] if pos[b] else torch.zeros(width))
        if active[b]:
            close(out[b: b + 1], want, dtype)
            close(state[b], last, torch.float32, factor=4.0)
        else:
            assert torch.equal(state[b].cpu(), before[b])


def _hgrn2_want(qfv, lower, bias, norm, heads, dim, vdim, state0, eps, true_vdim):
    hd = heads * dim
    q = R.silu(qfv[:, :hd].double()).view(-1, heads, dim)
    f = (lower.double() + (1 - lower.double()) * R.sigmoid(qfv[:, hd: 2 * hd].double() + bias.double())).view(-1, heads, dim)
    v = qfv[:, 2 * hd:].double().view(-1, heads, vdim)
    s, out = state0.double(), []
    for t in range(qfv.shape[0]):
        s = f[t][:, :, None] * s + (1 - f[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", s, q[t]))
    o = torch.stack(out)
    o = o / torch.sqrt(o.pow(2).sum(-1, keepdim=True) / true_vdim + eps) * norm.double()
    return o.flatten(1), s


def _hgrn2_inputs(tokens, heads, dim, vdim, dtype, seed):
    qfv = rnd(tokens, 2 * heads * dim + heads * vdim, seed=seed, dtype=dtype)
    bias = rnd(heads * dim, seed=seed + 1, scale=3.0)
    bias[::5] = 30.0            # f = 1: a channel that keeps its state for ever
    bias[1::7] = -90.0          # f = the floor
    lower = torch.rand(heads * dim, generator=torch.Generator().manual_seed(seed + 2))
    lower[1::14] = 0.0          # ... which may be zero
    return qfv, lower, bias, 1.0 + rnd(vdim, seed=seed + 3, scale=0.3)


HGRN2_SIZES = [(3, 32, 48), (1, 16, 16), (2, 48, 144), (4, 112, 64), (2, 128, 128), (5, 64, 32), (2, 208, 80), (1, 256, 512)]


@pytest.mark.parametrize("form", ["f32", "bf16", "bf16-serial"])
@pytest.mark.parametrize("heads,dim,vdim", HGRN2_SIZES)
def test_hgrn2_prefill(hops, form, heads, dim, vdim):
    dtype, eps = DT[form.split("-")[0]], 1e-5
    lengths, slots, starts = [1, 15, 16, 33, 70], [2, 0, 4, 5, 1], [0, 3, 0, 16, 0]
    qfv, lower, bias, norm = _hgrn2_inputs(sum(lengths), heads, dim, vdim, dtype, 11)
    before = rnd(6, heads, dim, vdim, seed=17)
    state = before.to(DEV)
    dev = [t.to(DEV) for t in (qfv, lower, bias, norm)]
    out = hops.hgrn2_prefill(*dev, state, Batch(slots, starts, lengths), vdim, eps, serial=form.endswith("serial"))
    row = 0
    for slot, start, n in zip(slots, starts, lengths):
        want, last = _hgrn2_want(qfv[row: row + n], lower, bias, norm, heads, dim, vdim,
                                 before[slot] if start else torch.zeros(heads, dim, vdim), eps, vdim)
        close(out[row: row + n], want, dtype, f"length {n}", 2.0)
        close(state[slot], last, torch.float32, f"state after {n}", 4.0)
        row += n
    assert torch.equal(state[3].cpu(), before[3])


@pytest.mark.parametrize("heads,dim,vdim", [(2, 128, 128), (1, 48, 144), (3, 32, 48)])
@pytest.mark.parametrize("segments", [None, (16, 40), (64, 10), (320, 2)])
def test_hgrn2_segments(hops, heads, dim, vdim, segments):
    """Sequences cut into segments that run side by side: unequal lengths (some with a single segment), carried states,
    gates that never forget across segments."""
    lengths, slots, starts, eps = [600, 16, 33, 320, 1], [2, 0, 4, 5, 1], [0, 3, 0, 16, 9], 1e-5
    qfv, lower, bias, norm = _hgrn2_inputs(sum(lengths), heads, dim, vdim, torch.bfloat16, 41)
    before = rnd(6, heads, dim, vdim, seed=42)
    state = before.to(DEV)
    out = hops.hgrn2_prefill(*[t.to(DEV) for t in (qfv, lower, bias, norm)], state, Batch(slots, starts, lengths), vdim, eps,
                             segments=segments)
    row = 0
    for slot, start, n in zip(slots, starts, lengths):
        want, last = _hgrn2_want(qfv[row: row + n], lower, bias, norm, heads, dim, vdim,
                                 before[slot] if start else torch.zeros(heads, dim, vdim), eps, vdim)
        close(out[row: row + n], want, torch.bfloat16, f"length {n}", 2.0)
        close(state[slot], last, torch.float32, f"state after {n}", 8.0)
        row += n
    assert torch.equal(state[3].cpu(), before[3])


@pytest.mark.parametrize("serial", [False, True])
def test_hgrn2_wide_batch(hops, serial):
    """A batch of many heads (the wide-column form of the token-serial kernel among them)."""
    heads, dim, vdim, lengths = 16, 128, 128, [20 + i for i in range(9)]
    qfv, lower, bias, norm = _hgrn2_inputs(sum(lengths), heads, dim, vdim, torch.bfloat16, 3)
    state = torch.zeros(9, heads, dim, vdim, device=DEV)
    out = hops.hgrn2_prefill(*[t.to(DEV) for t in (qfv, lower, bias, norm)], state, Batch(list(range(9)), [0] * 9, lengths), vdim, 1e-5,
                             serial=serial)
    row = 0
    for i, n in enumerate(lengths):
        want, last = _hgrn2_want(qfv[row: row + n], lower, bias, norm, heads, dim, vdim, torch.zeros(heads, dim, vdim), 1e-5, vdim)
        close(out[row: row + n], want, torch.bfloat16, f"length {n}", 2.0)
        close(state[i], last, torch.float32, factor=4.0)
        row += n


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("heads,dim,vdim", HGRN2_SIZES)
def test_hgrn2_decode(hops, dt, heads, dim, vdim):
    dtype, rows, eps = DT[dt], 4, 1e-5
    qfv, lower, bias, norm = _hgrn2_inputs(rows, heads, dim, vdim, dtype, 23)
    before = rnd(rows, heads, dim, vdim, seed=29)
    pos = torch.tensor([4, 0, 7, 1], device=DEV)
    active = torch.tensor([1, 1, 0, 1], device=DEV)
    state = before.to(DEV)
    out = hops.hgrn2_decode(*[t.to(DEV) for t in (qfv, lower, bias, norm)], state, pos, active, vdim, eps)
    for b in range(rows):
        if not active[b]:
            assert torch.equal(state[b].cpu(), before[b])
            continue
        want, last = _hgrn2_want(qfv[b: b + 1], lower, bias, norm, heads, dim, vdim,
                                 before[b] if pos[b] else torch.zeros(heads, dim, vdim), eps, vdim)
        close(out[b: b + 1], want, dtype, factor=2.0)
        close(state[b], last, torch.float32, factor=4.0)


# --------------------------------------------------------------------------------------------------- latent attention
def test_rope_interleaved(hops):
    from b200attn.mixers import Rotation
    rot = {"base": 300.0, "dims": 24, "scaling": {"factor": 3.0, "original": 40, "fast": 8.0, "slow": 1.0}}
    x = rnd(6, 3, 64 + 32, seed=1)
    pos = torch.tensor([0, 1, 999, 17, 500, 64], dtype=torch.int32)
    want = x.double().clone()
    want[..., 64: 88] = R.rotate(x[..., 64: 88].double(), rot, pos)
    got = x.to(DEV)
    hops.rope_interleaved(got, 64, pos.to(DEV), Rotation.from_config(rot).table(1000, DEV))
    close(got, want, torch.float32)


@pytest.mark.parametrize("repeat,q_rank", [(1, 128), (1, 2944), (200, 128), (200, 640), (200, 1152), (200, 1792)])
@pytest.mark.parametrize("dt", DT)
def test_latent_prep_writes_pages(hops, dt, repeat, q_rank):
    """A few rows and prompt-sized batches (the same six rows over and over), narrow and wide query latents."""
    from b200attn.mixers import Rotation
    dtype, eps = DT[dt], 1e-5
    rot = {"base": 300.0, "dims": 24}
    true_q, rank, true_rank, rotw = q_rank - 40, 64, 40, 64
    pos = torch.tensor([0, 15, 16, 31, 47, 5], dtype=torch.int32)
    slot = torch.tensor([1, 1, 1, 0, 0, 2], dtype=torch.int32)
    fused = rnd(6, q_rank + rank + rotw, seed=1, dtype=dtype)
    fused[:, true_q: q_rank] = 0
    fused[:, q_rank + true_rank: q_rank + rank] = 0
    fused[:, q_rank + rank + 24:] = 0
    qw, kw = rnd(q_rank, seed=2), rnd(rank, seed=3)
    table = torch.tensor([[7, 2, 4], [0, 5, 1], [6, 3, 8]], dtype=torch.int32, device=DEV)
    cache = torch.full((9, 16, rank + rotw), 5.0, dtype=dtype, device=DEV)
    active = torch.tensor([1, 1, 0], device=DEV)
    angles = Rotation.from_config(rot).table(64, DEV)
    cq = hops.latent_prep(fused.repeat(repeat, 1).to(DEV), qw.to(DEV), kw.to(DEV), pos.repeat(repeat).to(DEV),
                          slot.repeat(repeat).to(DEV), active, table, angles, cache, true_q, rank, true_rank, eps)
    assert torch.equal(cq[:6].repeat(repeat, 1), cq)
    cq = cq[:6]
    f = fused.double()
    close(cq[:, :true_q], R.rms(f[:, :true_q], eps) * qw[:true_q].double(), dtype)
    want = torch.full((9, 16, rank + rotw), 5.0, dtype=torch.float64)
    for i in range(6):
        if slot[i] == 2:
            continue                                       # idle
        r = torch.zeros(rank + rotw, dtype=torch.float64)
        r[:true_rank] = R.rms(f[i, q_rank: q_rank + true_rank], eps) * kw[:true_rank].double()
        r[rank: rank + 24] = R.rotate(f[i: i + 1, q_rank + rank: q_rank + rank + 24], rot, pos[i: i + 1])[0]
        want[table[slot[i], pos[i] // 16].item(), pos[i] % 16] = r
    close(cache, want, dtype)


def _portions(hops, lengths, starts, window, heads, dim, rot, vdim, rank, dtype, seed, true_dim=None, true_rot=None, plant=None):
    """Packed queries of portions, their packed visible keys, and the wanted outputs."""
    q = rnd(sum(lengths), heads, dim + rot, seed=seed, dtype=dtype)
    first = [max(0, s - window + 1) for s in starts]
    counts = [s + n - f for s, n, f in zip(starts, lengths, first)]
    kv = rnd(sum(counts), heads * (dim + vdim), seed=seed + 1, dtype=dtype)
    ctx = rnd(sum(counts), rank + rot, seed=seed + 2, dtype=dtype)
    if true_dim is not None:                               # padding columns carry zeros on both sides
        q[..., true_dim: dim] = 0
        q[..., dim + true_rot:] = 0
        kv[:, : heads * dim].view(-1, heads, dim)[..., true_dim:] = 0
        ctx[:, rank + true_rot:] = 0
    scale = (dim + rot) ** -0.5
    if plant is not None:
        plant(q, kv, ctx, lengths, starts, first, counts)
    want, r, c = [], 0, 0
    for n, s, f, m in zip(lengths, starts, first, counts):
        k = torch.cat((kv[c: c + m, : heads * dim].double().view(m, heads, dim),
                       ctx[c: c + m, None, rank:].double().expand(m, heads, rot)), -1)
        v = kv[c: c + m, heads * dim:].double().view(m, heads, vdim)
        score = torch.einsum("ihd,jhd->hij", q[r: r + n].double(), k) * scale
        gap = (s + torch.arange(n))[:, None] - (f + torch.arange(m))[None, :]
        score = score.masked_fill(~((gap >= 0) & (gap < window))[None], float("-inf"))
        want.append(torch.einsum("hij,jhd->ihd", score.softmax(-1), v).flatten(1))
        r, c = r + n, c + m
    i32 = dict(dtype=torch.int32, device=DEV)
    cu_q = torch.tensor([0] + torch.tensor(lengths).cumsum(0).tolist(), **i32)
    cu_k = torch.tensor([0] + torch.tensor(counts).cumsum(0).tolist(), **i32)
    args = (q.to(DEV), kv.to(DEV), ctx.to(DEV), cu_q, cu_k, torch.tensor(starts, **i32), torch.tensor(first, **i32), max(lengths),
            true_dim or dim, true_rot or rot, vdim, rank, window, scale)
    return args, torch.cat(want)


PREFILL_SIZES = [(3, 64, 64, 64, 64), (2, 128, 64, 128, 128), (1, 192, 64, 256, 64), (2, 64, 128, 192, 64), (2, 64, 64, 256, 64)]


@pytest.mark.parametrize("form", ["f32", "bf16", "bf16-simple"])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank", PREFILL_SIZES)
@pytest.mark.parametrize("window", [1, 2, 50, 128, 129, 10 ** 9])
def test_latent_prefill(hops, form, heads, dim, rot, vdim, rank, window):
    dtype = torch.float32 if form == "f32" else torch.bfloat16
    args, want = _portions(hops, [1, 2, 130, 300], [500, 0, 90, 0], window, heads, dim, rot, vdim, rank, dtype, 7)
    got = hops.latent_prefill(*args, simple=form.endswith("simple"))
    close(got, want, dtype)
    import b200attn
    assert b200attn.load().b200_wait_timed_out() == 0


def test_latent_prefill_padded_heads(hops):
    args, want = _portions(hops, [140, 5], [0, 60], 33, 3, 64, 64, 64, 64, torch.bfloat16, 9, true_dim=40, true_rot=24)
    close(hops.latent_prefill(*args), want, torch.bfloat16)


@pytest.mark.parametrize("form", ["f32", "bf16", "bf16-simple"])
@pytest.mark.parametrize("distance", ["inside", "outside"])
@pytest.mark.parametrize("window", [96, 128, 130, 257])
def test_latent_prefill_window_edge(hops, form, distance, window):
    """One key stands out for one query: just inside the window it takes all the weight, just outside it takes none."""
    dtype = torch.float32 if form == "f32" else torch.bfloat16
    back = window - 1 if distance == "inside" else window
    heads, dim, rot, vdim, rank = 2, 64, 64, 64, 64
    spots = []

    def plant(q, kv, ctx, lengths, starts, first, counts):
        r, c = 0, 0
        for n, s, f, m in zip(lengths, starts, first, counts):
            for i in (0, 1, n // 2, n - 2, n - 1):
                j = s + i - back - f
                if 0 <= j < m and i >= 0:
                    d = torch.randn(dim, generator=torch.Generator().manual_seed(100 + i))
                    d = d / d.norm() * 40
                    q[r + i, :, :dim] = d.to(q.dtype)
                    kv[c + j, : heads * dim].view(heads, dim)[:] = d.to(kv.dtype)
                    spots.append((r + i, c + j))
            r, c = r + n, c + m

    args, want = _portions(hops, [400, 70], [0, 333], window, heads, dim, rot, vdim, rank, dtype, 21, plant=plant)
    assert len(spots) >= 4
    got = hops.latent_prefill(*args, simple=form.endswith("simple"))
    close(got, want, dtype)
    v = args[1].cpu()[:, heads * dim:].double()
    for row, key in spots[:1]:
        near = (want[row] - v[key]).abs().max() < 0.05
        assert near == (distance == "inside")


def _decode_case(hops, positions, heads, rank, rot, window, splits, dtype, seed, batch_active=None):
    pitch, batch = rank + rot, len(positions)
    per = max(p // 16 + 1 for p in positions)
    pages = batch * per + 3
    order = torch.randperm(pages, generator=torch.Generator().manual_seed(seed))
    table = order[: batch * per].view(batch, per).to(torch.int32)
    cache = rnd(pages, 16, pitch, seed=seed + 1, dtype=dtype)
    q = rnd(batch, heads, pitch, seed=seed + 2, dtype=dtype)
    scale = pitch ** -0.5 * 2
    want = torch.zeros(batch, heads, rank, dtype=torch.float64)
    for b, p in enumerate(positions):
        lo = max(0, p - window + 1)
        rows = torch.stack([cache[table[b, j // 16].item(), j % 16] for j in range(lo, p + 1)]).double()
        w = torch.softmax(q[b].double() @ rows.T * scale, -1)
        want[b] = w @ rows[:, :rank]
        visible = torch.zeros(pages, 16, dtype=torch.bool)
        for j in range(lo, p + 1):
            visible[table[b, j // 16].item(), j % 16] = True
        own = torch.zeros(pages, dtype=torch.bool)
        own[table[b].long()] = True
        cache[own[:, None] & ~visible] = float("nan")      # nothing else of its pages may matter
    ws = hops.latent_decode_workspace(batch, heads, rank, splits, DEV)
    ws[1].fill_(float("nan"))
    active = None if batch_active is None else torch.tensor(batch_active, device=DEV)
    args = (q.to(DEV), cache.to(DEV), table.to(DEV), torch.tensor(positions, device=DEV), active, ws, window, scale)
    return args, want


@pytest.mark.parametrize("form", ["f32", "bf16", "bf16-simple"])
@pytest.mark.parametrize("heads,rank,rot,splits", [(1, 64, 64, 1), (5, 128, 64, 3), (16, 512, 64, 4), (17, 192, 64, 2), (40, 64, 64, 7),
                                                   (3, 1024, 64, 2), (16, 320, 128, 5)])
@pytest.mark.parametrize("window", [1, 2, 33, 10 ** 9])
def test_latent_decode(hops, form, heads, rank, rot, splits, window):
    dtype = torch.float32 if form == "f32" else torch.bfloat16
    positions = [0, 1, 15, 16, 31, 32, 33, 200]
    args, want = _decode_case(hops, positions, heads, rank, rot, window, splits, dtype, 31)
    hops.latent_decode(*args, simple=form.endswith("simple"))
    eye = torch.eye(rank).to(dtype).expand(heads, rank, rank).contiguous().to(DEV)      # W_uv = identity: the merge alone
    got = hops.latent_value(args[5], eye, dtype).view(len(positions), heads, rank)
    close(got, want, dtype)
    import b200attn
    assert b200attn.load().b200_wait_timed_out() == 0


def test_latent_decode_idle_slots(hops):
    args, want = _decode_case(hops, [20, 40, 7], 4, 64, 64, 100, 2, torch.bfloat16, 5, batch_active=[1, 0, 1])
    hops.latent_decode(*args)
    eye = torch.eye(64).to(torch.bfloat16).expand(4, 64, 64).contiguous().to(DEV)
    got = hops.latent_value(args[5], eye, torch.bfloat16).view(3, 4, 64)
    close(got[[0, 2]], want[[0, 2]], torch.bfloat16)
    assert not got[1].any()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("batch,heads,dim,rank,rot", [(1, 3, 64, 64, 64), (5, 2, 128, 512, 64), (33, 4, 192, 128, 64)])
def test_latent_absorb_and_value(hops, dt, batch, heads, dim, rank, rot):
    from b200attn.mixers import Rotation
    dtype = DT[dt]
    rotation = {"base": 100.0, "dims": 48}
    q = rnd(batch, heads, dim + rot, seed=1, dtype=dtype)
    uk = rnd(heads, dim, rank, seed=2, dtype=dtype, scale=dim ** -0.5)
    pos = torch.arange(batch, device=DEV) * 7
    got = hops.latent_absorb(q.to(DEV), uk.to(DEV), pos, Rotation.from_config(rotation).table(300, DEV))
    close(got[..., :rank], torch.einsum("bhd,hdr->bhr", q[..., :dim].double(), uk.double()), dtype)
    want = q[..., dim:].double().clone()
    want[..., :48] = R.rotate(want[..., :48], rotation, pos.cpu())
    close(got[..., rank:], want, dtype)
    # merge of splits (one of them empty) and W_uv
    vdim = 128
    uv = rnd(heads, vdim, rank, seed=3, dtype=dtype, scale=rank ** -0.5)
    ml = torch.stack((rnd(batch, heads, 3, seed=4), rnd(batch, heads, 3, seed=5).abs() + 0.1), -1)
    o = rnd(batch, heads, 3, rank, seed=6)
    ml[:, :, 1] = torch.tensor([float("-inf"), 0.0])
    o[:, :, 1] = float("nan")
    m = ml[..., 0].double()
    w = torch.exp(m - m.max(-1, keepdim=True)[0])
    w = w / (w * ml[..., 1].double()).sum(-1, keepdim=True)
    merged = sum(w[..., s, None] * o[..., s, :].double() for s in (0, 2))
    got = hops.latent_value((ml.to(DEV), o.to(DEV)), uv.to(DEV), dtype).view(batch, heads, vdim)
    close(got, torch.einsum("bhr,hvr->bhv", merged, uv.double()), dtype)


def test_latent_gather(hops):
    cache = rnd(8, 16, 128, seed=1).to(DEV)
    table = torch.tensor([[3, 1, 6], [0, 7, 2]], dtype=torch.int32, device=DEV)
    i32 = dict(dtype=torch.int32, device=DEV)
    out = hops.latent_gather(cache, table, torch.tensor([1, 0], **i32), torch.tensor([0, 20, 25], **i32), torch.tensor([9, 30], **i32),
                             25, 20)
    rows = [cache[table[1, j // 16], j % 16] for j in range(9, 29)] + [cache[table[0, j // 16], j % 16] for j in range(30, 35)]
    assert torch.equal(out, torch.stack(rows))
