"""Kernels of the cores (windowed attention with grouped heads, state space, gated linear attention, gated feed-forward, norm
weights, soft cap) alone against the plain restatement, in fp32 and bf16, at sizes, page borders, window edges, chunk
edges and slot states where a mistake shows."""
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


def wide(t, extra, seed=0):
    """t as the leading columns of a wider matrix on the device (rows further apart than they are long)."""
    full = torch.cat((t, rnd(t.shape[0], extra, seed=seed, dtype=t.dtype)), dim=1).to(DEV)
    return full[:, : t.shape[1]]


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


# ------------------------------------------------------------------------------------------------------- element-wise
@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("width,true", [(64, 64), (192, 136), (2048, 2000)])
def test_norm_weights_on_a_plain_residual(hops, dt, width, true):
    dtype, rows, eps = DT[dt], 7, 1e-3
    x, y, gain = rnd(rows, 1, width, seed=1), rnd(rows, width, seed=2, dtype=dtype), rnd(width, seed=3)
    x[..., true:], y[:, true:], gain[true:] = 0, 0, 0
    streams = x.to(DEV)
    h = hops.hyper_connect(streams, torch.ones(4, device=DEV), true, eps, dtype, y=y.to(DEV), gains=gain.to(DEV))
    total = x[:, 0].double() + y.double()
    close(streams[:, 0], total, torch.float32)
    close(h[:, :true], R.rms(total[:, :true], eps) * gain[:true].double(), dtype)
    assert not h[:, true:].any()


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("rows,width", [(3, 64), (1030, 192), (1, 8), (5, 2048)])
def test_gated_act(hops, dt, rows, width):
    dtype = DT[dt]
    gu = rnd(rows, 2 * width, seed=1, dtype=dtype, scale=3.0)
    gu[0, :4] = torch.tensor([40.0, -40.0, 0.0, -5.0]).to(dtype)
    for act, fn in ((hops.ACT_SILU, R.silu), (hops.ACT_GELU_TANH, R.gelu_tanh)):
        out = torch.full((rows, width + 8), 7.0, dtype=dtype, device=DEV)
        hops.gated_act(wide(gu, 24), width, out[:, :width], act)
        close(out[:, :width], fn(gu[:, :width].double()) * gu[:, width:].double(), dtype)
        assert (out[:, width:] == 7).all()


def test_softcap(hops):
    x = rnd(5, 336, seed=1, scale=60.0)
    got = hops.softcap(x.to(DEV).clone(), 331, 12.5)
    close(got[:, :331], 12.5 * torch.tanh(x[:, :331].double() / 12.5), torch.float32)
    assert torch.isneginf(got[:, 331:]).all()


# -------------------------------------------------------------------------------------------------- windowed attention
class Attention:
    """One layer's sizes, random projections of sequences, and what the restatement makes of them."""

    def __init__(self, heads, kv_heads, dim, vdim, dims, window, dtype, lengths, seed=0, scale=None):
        from b200attn.mixers import Rotation, round_up
        self.heads, self.kv_heads, self.dim, self.vdim, self.window, self.dtype = heads, kv_heads, dim, vdim, window, dtype
        self.dim_p, self.vdim_p = round_up(dim, 32), round_up(vdim, 64)
        self.pitch = round_up(self.dim_p + self.vdim_p, 64)
        self.rot, self.scale, self.out_scale = {"base": 500.0, "dims": dims}, scale or dim ** -0.5, 0.7
        self.angles = Rotation(dims, 500.0).table(max(lengths) + 1, DEV)
        self.qkv = [(rnd(n, heads, dim, seed=seed + 5 * i, dtype=dtype), rnd(n, kv_heads, dim, seed=seed + 5 * i + 1, dtype=dtype),
                     rnd(n, kv_heads, vdim, seed=seed + 5 * i + 2, dtype=dtype), rnd(n, heads, vdim, seed=seed + 5 * i + 3, dtype=dtype))
                    for i, n in enumerate(lengths)]
        self.biases = rnd(heads, dim, seed=90, scale=0.5), rnd(kv_heads, dim, seed=91, scale=0.5), rnd(kv_heads, vdim, seed=92, scale=0.5)

    def _pad(self, t, size):
        out = torch.zeros(*t.shape[:-1], size, dtype=t.dtype)
        out[..., : t.shape[-1]] = t
        return out.flatten(-2)

    def rows(self, seq, lo, hi):
        """[q | k | v | gate] projection rows lo..hi-1 of a sequence, padded."""
        q, k, v, g = (t[lo:hi] for t in self.qkv[seq])
        return torch.cat((self._pad(q, self.dim_p), self._pad(k, self.dim_p), self._pad(v, self.vdim_p), self._pad(g, self.vdim_p)), dim=1)

    def bias(self):
        q, k, v = self.biases
        return torch.cat((self._pad(q, self.dim_p), self._pad(k, self.dim_p), self._pad(v, self.vdim_p))).to(DEV)

    @property
    def gate_at(self):
        return (self.heads + self.kv_heads) * self.dim_p + self.kv_heads * self.vdim_p

    def rotated(self, seq):
        q, k, v, _ = (t.double() for t in self.qkv[seq])
        at = torch.arange(q.shape[0])
        bq, bk, bv = (b.double() for b in self.biases)
        return R.rotate_halves(q + bq, self.rot, at), R.rotate_halves(k + bk, self.rot, at), v + bv

    def want(self, seq):
        q, k, v = self.rotated(seq)
        if self.dtype == torch.bfloat16:
            q, k, v = (t.to(torch.bfloat16).double() for t in (q, k, v))
        owner = torch.arange(self.heads) // (self.heads // self.kv_heads)
        o = R.window_attention(q, k[:, owner], v[:, owner], self.scale, self.window)
        return o * R.sigmoid(self.qkv[seq][3].double()) * self.out_scale

    def head_columns(self, out):
        return out.view(out.shape[0], self.heads, self.vdim_p)[..., : self.vdim]


def run_prefill(hops, a, slots, starts, ends, table, cache, simple=False):
    """Sequences' tokens starts..ends-1 through prep, gather and prefill; earlier positions are in the cache."""
    from b200attn.hybrid import PackedBatch
    b = PackedBatch(slots, starts, [[0] * (e - s) for s, e in zip(starts, ends)], DEV)
    x = wide(torch.cat([a.rows(i, s, e) for i, (s, e) in enumerate(zip(starts, ends))]), 40)
    span = b.context(a.window)
    ctx = torch.full((span.keys, a.kv_heads, a.pitch), float("nan"), dtype=a.dtype, device=DEV)
    hops.window_prep(x, a.bias(), b.pos, b.slot_of, None, table, a.angles, cache, a.heads, a.dim_p, a.vdim_p, ctx=ctx, ctx_row=span.rows)
    if span.max_old:
        hops.window_gather(cache, ctx, table, b.slots, span.cu, span.first, span.max_old)
    out = torch.full((x.shape[0], a.heads * a.vdim_p + 8), 5.0, dtype=a.dtype, device=DEV)
    hops.window_prefill(x, ctx, x[:, a.gate_at:], out[:, :-8], b.cu, span.cu, b.start, span.first, b.max_len, a.heads, a.dim_p, a.dim, a.vdim_p,
                        a.window, a.scale, a.out_scale, simple=simple)
    assert (out[:, -8:] == 5).all()
    o = out[:, :-8].reshape(-1, a.heads, a.vdim_p)
    assert not o[..., a.vdim:].any()
    return o[..., : a.vdim].split([e - s for s, e in zip(starts, ends)])


def pages(slots, context, seed=3):
    per = -(-context // 16)
    perm = torch.randperm(slots * per + 2, generator=torch.Generator().manual_seed(seed))[: slots * per]
    return perm.view(slots, per).to(torch.int32).to(DEV), slots * per + 2


SIZES = [(4, 2, 32, 64, 32), (6, 3, 20, 24, 12), (5, 1, 72, 136, 72), (2, 2, 160, 192, 48), (17, 1, 128, 128, 64), (2, 1, 256, 256, 256),
         (2, 1, 264, 264, 40), (3, 3, 64, 64, 2)]


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("simple", [False, True])
@pytest.mark.parametrize("sizes", SIZES)
def test_window_prefill_sizes(hops, dt, simple, sizes):
    if simple and dt == "f32":
        pytest.skip("fp32 has one form")
    dtype = DT[dt]
    a = Attention(*sizes, window=33, dtype=dtype, lengths=[150, 1, 70])
    table, n = pages(4, 160)
    cache = hops.allocate_window_cache(n, a.kv_heads, a.pitch, dtype, device=DEV)
    got = run_prefill(hops, a, [2, 0, 3], [0, 0, 0], [150, 1, 70], table, cache, simple)
    for i in range(3):
        close(got[i], a.want(i), dtype, f"sequence {i}", 1.0 if dt == "f32" else 0.8)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 127, 128, 129, 200, 1000])
def test_window_prefill_portions(hops, dt, window):
    """The second portion of three sequences reads keys of the first from the pages; lengths straddle 128-token tiles."""
    dtype = DT[dt]
    a = Attention(4, 2, 40, 72, 24, window=window, dtype=dtype, lengths=[300, 140, 33], seed=40)
    table, n = pages(4, 304)
    cache = hops.allocate_window_cache(n, a.kv_heads, a.pitch, dtype, device=DEV)
    cuts = [(0, 0, 0), (131, 2, 31), (133, 140, 33), (300, 140, 33)]
    for lo, hi in zip(cuts, cuts[1:]):
        live = [i for i in range(3) if hi[i] > lo[i]]
        if live != list(range(len(live))):
            live = [0]
        sub = [[2, 0, 3][i] for i in live]
        got = run_prefill(hops, a, sub, [lo[i] for i in live], [hi[i] for i in live], table, cache)
        for i, g in zip(live, got):
            close(g, a.want(i)[lo[i]: hi[i]], dtype, f"sequence {i} from {lo[i]}", 1.0 if dt == "f32" else 0.8)


def standout(a, query, keys, gain):
    """Makes the scores of one query with some keys stand far out: the keys are set to the query's direction (undoing rotation
    and biases), so attention weighs what is visible of them and little else."""
    q, k, _, _ = a.qkv[0]
    d = torch.zeros(a.dim).double()
    d[: a.rot["dims"] // 2] = 1.0
    d = d / d.norm()

    def raw(pos, size, bias):                       # rotate(raw + bias) = size * d
        x = (size * d).view(1, 1, -1)
        n = a.rot["dims"] // 2
        freqs, _ = R.rotary_frequencies(a.rot)
        ang = pos * freqs
        u, w = x[..., :n].clone(), x[..., n: 2 * n].clone()
        un = torch.cat((u * ang.cos() + w * ang.sin(), w * ang.cos() - u * ang.sin(), x[..., 2 * n:]), -1)
        return un.view(-1) - bias

    for h in range(a.heads):
        q[query, h] = raw(query, gain, a.biases[0][h].double()).to(q.dtype)
    for j in keys:
        for h in range(a.kv_heads):
            k[j, h] = raw(j, gain, a.biases[1][h].double()).to(k.dtype)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("window,query", [(37, 90), (16, 64), (128, 300), (130, 257), (1, 50)])
def test_window_edges_in_prompts_and_decoding(hops, dt, window, query):
    """A key that stands out just inside the window takes the row; one just outside must not be seen."""
    dtype = DT[dt]
    inside, outside = query - window + 1, query - window
    for at in (inside, outside):
        a = Attention(4, 2, 40, 72, 24, window=window, dtype=dtype, lengths=[query + 5], seed=70, scale=0.5)
        a.qkv[0][2][at] = 30.0                                 # its value is unmistakable
        standout(a, query, [at], 8.0)
        want = a.want(0)
        seen = want[query].abs().max() > 5
        assert bool(seen) == (at == inside)
        table, n = pages(2, query + 16)
        cache = hops.allocate_window_cache(n, a.kv_heads, a.pitch, dtype, device=DEV)
        got = run_prefill(hops, a, [1], [0], [query + 5], table, cache)[0]
        close(got, want, dtype, "prompt", 2.0)
        # the same query decoded after a prompt
        cache.zero_()
        run_prefill(hops, a, [1], [0], [query], table, cache)
        got = run_decode(hops, a, table, cache, [0, query], [False, True], [None, 0])
        close(got[1], want[query], dtype, "decoded", 2.0)


def run_decode(hops, a, table, cache, pos, active, seqs, splits=None, simple=False):
    batch = len(pos)
    x = wide(torch.cat([a.rows(s, p, p + 1) if s is not None else a.rows(0, 0, 1) for s, p in zip(seqs, pos)]), 24)
    pos, active = torch.tensor(pos, device=DEV), torch.tensor(active, device=DEV).long()
    hops.window_prep(x, a.bias(), pos, None, active, table, a.angles, cache, a.heads, a.dim_p, a.vdim_p)
    ws = hops.latent_decode_workspace(batch, a.heads, a.vdim_p, splits or 3, DEV)
    ws[1].fill_(float("nan"))
    hops.window_decode(x, cache, table, pos, active, ws, a.dim_p, a.window, a.scale, simple=simple)
    out = torch.full((batch, a.heads * a.vdim_p + 8), 5.0, dtype=a.dtype, device=DEV)
    hops.window_merge(ws, x[:, a.gate_at:], out[:, :-8], a.out_scale)
    assert (out[:, -8:] == 5).all()
    o = out[:, :-8].reshape(batch, a.heads, a.vdim_p)
    assert not o[..., a.vdim:].any()
    return o[..., : a.vdim]


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("simple", [False, True])
@pytest.mark.parametrize("sizes", SIZES)
def test_window_decode_sizes(hops, dt, simple, sizes):
    if simple and dt == "f32":
        pytest.skip("fp32 has one form")
    dtype = DT[dt]
    lengths = [150, 1, 17, 64]
    a = Attention(*sizes, window=100, dtype=dtype, lengths=lengths, seed=11)
    table, n = pages(5, 160)
    cache = hops.allocate_window_cache(n, a.kv_heads, a.pitch, dtype, device=DEV)
    for i, length in enumerate(lengths):
        if length > 1:
            one = Attention(*sizes, window=100, dtype=dtype, lengths=[150], seed=11 + 5 * i)
            run_prefill(hops, one, [i], [0], [length - 1], table, cache)
    before = cache[table[4].long()].clone()
    got = run_decode(hops, a, table, cache, [n - 1 for n in lengths] + [3], [True] * 4 + [False], [0, 1, 2, 3, None], simple=simple)
    for i, length in enumerate(lengths):
        close(got[i], a.want(i)[length - 1], dtype, f"slot {i}", 1.0 if dt == "f32" else 0.8)
    assert torch.equal(cache[table[4].long()], before)          # the idle slot wrote nothing


@pytest.mark.parametrize("splits", [1, 2, 7, 64])
@pytest.mark.parametrize("window", [3, 16, 90, 500])
def test_window_decode_reads_nothing_it_must_not(hops, splits, window):
    """NaN in every cache row outside the window, and in the rows of the last page behind the token."""
    dtype, length = torch.bfloat16, 230
    a = Attention(6, 2, 64, 64, 64, window=window, dtype=dtype, lengths=[length], seed=21)
    table, n = pages(1, 240)
    cache = hops.allocate_window_cache(n, a.kv_heads, a.pitch, dtype, device=DEV)
    run_prefill(hops, a, [0], [0], [length - 1], table, cache)
    for p in list(range(0, max(0, length - window))) + list(range(length, 240)):
        cache[table[0, p // 16].long(), :, p % 16] = float("nan")
    got = run_decode(hops, a, table, cache, [length - 1], [True], [0], splits=splits)
    close(got[0], a.want(0)[length - 1], dtype, factor=0.8)


# --------------------------------------------------------------------------------------------------------- state space
@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 8, 11, 16])
def test_convolution(hops, dt, taps):
    """Whole prompts and portions of every small size, through the ring, against one pass; another slot is left alone."""
    dtype, channels, length = DT[dt], 72, 90
    T = hops.conv_taps(taps)
    x, w, b = rnd(length, channels, seed=1, dtype=dtype), rnd(channels, taps, seed=2), rnd(channels, seed=3)
    want = R.silu(R.causal_conv(x.double(), w.double(), b.double()))
    weight = torch.zeros(T, channels)
    weight[:taps] = w.flip(1).t()
    weight, bias = weight.to(DEV).contiguous(), b.to(DEV)
    for sizes in ([length], [1], [2], [3, 1], [16, 17], [5, 40, 2]):
        ring = torch.full((3, T, channels), 9.0, device=DEV)
        got, at, k = [], 0, 0
        while at < length:
            n = min(sizes[min(k, len(sizes) - 1)], length - at)
            got.append(hops.conv_prefill(wide(x[at: at + n], 16), weight, bias, ring, Batch([1], [at], [n])))
            at, k = at + n, k + 1
        close(torch.cat(got), want, dtype, f"portions {sizes}")
        assert (ring[::2] == 9).all()


def ssd_inputs(heads, groups, dim, vdim, length, dtype, seed=0):
    xbc = rnd(length, heads * vdim + 2 * groups * dim, seed=seed, dtype=dtype)
    dt = rnd(length, heads, seed=seed + 1, dtype=dtype, scale=2.0)
    return xbc, dt, rnd(heads, seed=seed + 2) - 2.0, rnd(heads, seed=seed + 3, scale=1.5) - 1.0, rnd(heads, seed=seed + 4)


def ssd_want(xbc, dt, dt_bias, a_log, skip, heads, groups, dim, vdim, state0):
    """The recurrence from a state [heads, dim, vdim], and the state it leaves."""
    xbc, dt = xbc.double(), R.softplus(dt.double() + dt_bias.double())
    x, B, C = xbc.split([heads * vdim, groups * dim, groups * dim], dim=1)
    owner = torch.arange(heads) // (heads // groups)
    x, B, C = x.view(-1, heads, vdim), B.view(-1, groups, dim)[:, owner], C.view(-1, groups, dim)[:, owner]
    S, out = state0.double(), []
    for t in range(x.shape[0]):
        S = torch.exp(-torch.exp(a_log.double()) * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, C[t]) + skip.double()[:, None] * x[t])
    return torch.stack(out).flatten(1), S


SSD_SIZES = [(4, 2, 64, 32), (6, 3, 32, 48), (8, 1, 16, 16), (8, 2, 128, 64), (2, 1, 48, 144), (1, 1, 128, 128), (2, 2, 208, 32)]


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("sizes", SSD_SIZES)
@pytest.mark.parametrize("lengths", [[1, 2, 31], [32, 33, 70], [150]])
def test_state_space_prefill(hops, dt, sizes, lengths):
    dtype, (heads, groups, dim, vdim) = DT[dt], sizes
    slots, starts = [3, 0, 4][: len(lengths)], [0, 9, 5][: len(lengths)]
    xbc, step, dt_bias, a_log, skip = ssd_inputs(heads, groups, dim, vdim, sum(lengths), dtype)
    before = rnd(5, heads, dim, vdim, seed=8)
    state = before.to(DEV)
    dev = [t.to(DEV) for t in (dt_bias, a_log, skip)]
    y = hops.ssd_prefill(wide(xbc, 8), wide(step, 24), *dev, state, groups, Batch(slots, starts, lengths))
    row = 0
    for slot, start, n in zip(slots, starts, lengths):
        first = before[slot] if start else torch.zeros(heads, dim, vdim)
        want, last = ssd_want(xbc[row: row + n], step[row: row + n], dt_bias, a_log, skip, heads, groups, dim, vdim, first)
        close(y[row: row + n], want, dtype, f"length {n}")
        close(state[slot], last, torch.float32, f"state after {n}", 2.0 if dt == "f32" else 20.0)
        row += n
    for slot in set(range(5)) - set(slots):
        assert torch.equal(state[slot].cpu(), before[slot])


@pytest.mark.parametrize("segments", [(64, 8), (32, 16), (256, 2), (512, 1)])
@pytest.mark.parametrize("sizes", [(4, 2, 64, 32), (2, 1, 48, 144)])
def test_state_space_segments(hops, segments, sizes):
    """Sequences cut into segments that run side by side give what one pass gives, also with slow decays: far tokens matter."""
    heads, groups, dim, vdim = sizes
    lengths, starts, slots = [500, 64, 300], [0, 3, 0], [1, 2, 0]
    xbc, step, dt_bias, a_log, skip = ssd_inputs(heads, groups, dim, vdim, sum(lengths), torch.bfloat16, seed=30)
    a_log = a_log - 4.0
    before = rnd(3, heads, dim, vdim, seed=8)
    state = before.to(DEV)
    y = hops.ssd_prefill(xbc.to(DEV), step.to(DEV), *(t.to(DEV) for t in (dt_bias, a_log, skip)), state, groups,
                         Batch(slots, starts, lengths), segments=segments)
    row = 0
    for slot, start, n in zip(slots, starts, lengths):
        first = before[slot] if start else torch.zeros(heads, dim, vdim)
        want, last = ssd_want(xbc[row: row + n], step[row: row + n], dt_bias, a_log, skip, heads, groups, dim, vdim, first)
        close(y[row: row + n], want, torch.bfloat16, f"length {n}")
        close(state[slot], last, torch.float32, f"state after {n}", 20.0)
        row += n


@pytest.mark.parametrize("dt", DT)
def test_state_space_extreme_steps(hops, dt):
    """Steps that wipe the state and steps of almost nothing inside one chunk."""
    dtype, (heads, groups, dim, vdim) = DT[dt], (2, 1, 32, 32)
    xbc, step, dt_bias, a_log, skip = ssd_inputs(heads, groups, dim, vdim, 100, dtype, seed=50)
    step[:] = torch.where(torch.rand(100, heads, generator=torch.Generator().manual_seed(1)) < 0.2, 60.0, -14.0).to(dtype)
    a_log[:] = torch.tensor([3.0, -3.0])
    state = torch.zeros(1, heads, dim, vdim, device=DEV)
    y = hops.ssd_prefill(xbc.to(DEV), step.to(DEV), *(t.to(DEV) for t in (dt_bias, a_log, skip)), state, groups, Batch([0], [0], [100]))
    want, last = ssd_want(xbc, step, dt_bias, a_log, skip, heads, groups, dim, vdim, torch.zeros(heads, dim, vdim))
    close(y, want, dtype, factor=2.0)
    close(state[0], last, torch.float32, factor=4.0 if dt == "f32" else 20.0)


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("sizes", SSD_SIZES)
@pytest.mark.parametrize("taps", [1, 4, 6])
def test_state_space_decode(hops, dt, sizes, taps):
    """Several decoded tokens in slots at different positions, one idle: convolution, ring and state run on."""
    dtype, (heads, groups, dim, vdim), T = DT[dt], sizes, hops.conv_taps(taps)
    channels, n, batch = heads * vdim + 2 * groups * dim, 7, 3
    seqs = [ssd_inputs(heads, groups, dim, vdim, n, dtype, seed=60 + 7 * b) for b in range(batch)]
    _, _, dt_bias, a_log, skip = seqs[0]
    w, bias = rnd(channels, taps, seed=1), rnd(channels, seed=2, scale=0.3)
    weight = torch.zeros(T, channels)
    weight[:taps] = w.flip(1).t()
    ring, state = torch.full((batch, T, channels), 4.0, device=DEV), rnd(batch, heads, dim, vdim, seed=3).to(DEV)
    idle = ring[2].clone(), state[2].clone()
    dev = [t.to(DEV).contiguous() for t in (dt_bias, a_log, skip, weight, bias)]
    for t in range(n):
        x = wide(torch.stack([seqs[b][0][t] for b in range(batch)]), 8)
        step = wide(torch.stack([seqs[b][1][t] for b in range(batch)]), 8)
        y = hops.ssd_decode(x, step, *dev, ring, state, groups, torch.tensor([t, t, 2], device=DEV), torch.tensor([1, 1, 0], device=DEV))
        for b in range(2):
            conv = R.silu(R.causal_conv(seqs[b][0][: t + 1].double(), w.double(), bias.double()))
            want, last = ssd_want(conv, seqs[b][1][: t + 1], dt_bias, a_log, skip, heads, groups, dim, vdim, torch.zeros(heads, dim, vdim))
            close(y[b], want[-1], torch.float32, f"token {t}", 2.0 if dt == "f32" else 10.0)
            close(state[b], last, torch.float32, f"state after {t}", 2.0 if dt == "f32" else 10.0)
    assert torch.equal(ring[2], idle[0]) and torch.equal(state[2], idle[1])


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("rows", [3, 1100])
@pytest.mark.parametrize("heads,vdim,true,groups", [(4, 32, 32, 2), (6, 32, 20, 5), (3, 16, 16, 1), (8, 64, 64, 1), (16, 64, 64, 16), (40, 64, 64, 1),
                                                    (2, 48, 48, 12), (3, 16, 9, 27)])
def test_gated_group_norm(hops, dt, rows, heads, vdim, true, groups):
    dtype, eps = DT[dt], 1e-3
    if rows > 100 and heads * vdim > 2000:
        rows = 130
    for y_dtype in {dtype, torch.float32}:
        y, z, w = (torch.zeros(n, heads, vdim) for n in (rows, rows, 1))
        y[..., :true], z[..., :true], w[..., :true] = rnd(rows, heads, true, seed=1), rnd(rows, heads, true, seed=2, scale=2.0), rnd(1, heads, true, seed=3)
        y[..., true:] = 3.0                                    # padding is not read
        y, z, w = y.flatten(1).to(y_dtype), z.flatten(1).to(dtype), w.flatten()
        out = torch.full((rows, heads * vdim + 8), 5.0, dtype=dtype, device=DEV)
        hops.gated_group_norm(y.to(DEV), wide(z, 16), w.to(DEV), out[:, :-8], heads, true, groups, eps)
        f = (y.double() * R.silu(z.double())).view(rows, heads, vdim)[..., :true].reshape(rows, -1)
        want = R.grouped_rms(f, groups, eps) * w.view(heads, vdim)[:, :true].reshape(-1).double()
        got = out[:, :-8].reshape(rows, heads, vdim)
        close(got[..., :true].reshape(rows, -1), want, dtype)
        assert not got[..., true:].any() and (out[:, -8:] == 5).all()


# ----------------------------------------------------------------------------------------------- gated linear attention
def gla_inputs(heads, dim, vdim, length, dtype, seed=0):
    return (rnd(length, heads * (2 * dim + vdim), seed=seed, dtype=dtype), rnd(length, heads * dim, seed=seed + 1, scale=2.0),
            rnd(length, heads * vdim, seed=seed + 2, dtype=dtype))


def gla_want(qkv, z, gate, bias, norm, heads, dim, vdim, true, q_scale, tau, eps, state0):
    q, k, v = (t.double().view(-1, heads, n) for t, n in zip(qkv.split([heads * dim, heads * dim, heads * vdim], 1), (dim, dim, vdim)))
    keep = torch.exp(-R.softplus(-(z.double() + bias.double())) / tau).view(-1, heads, dim)
    S, out = state0.double(), []
    for t in range(q.shape[0]):
        S = keep[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t] * q_scale))
    o = torch.stack(out)
    o = o / torch.sqrt(o.pow(2).sum(-1, keepdim=True) / true + eps) * norm.double()
    return o.flatten(1) * R.silu(gate.double()), S


GLA_SIZES = [(2, 32, 32, 32), (3, 24, 40, 40), (1, 64, 128, 100), (2, 128, 128, 128), (2, 48, 208, 208), (1, 200, 64, 64), (4, 8, 4, 3)]


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("serial", [False, True])
@pytest.mark.parametrize("heads,dim,vdim,true", GLA_SIZES)
def test_gla_prefill(hops, dt, serial, heads, dim, vdim, true):
    dtype, lengths, slots, starts, eps = DT[dt], [1, 15, 16, 90], [2, 0, 4, 1], [0, 6, 2, 0], 1e-4
    if serial and dt == "f32":
        pytest.skip("fp32 has one form")
    if dt == "bf16" and vdim % 8:
        serial = True                                          # the chunked form takes whole 16-byte vectors
    qkv, z, gate = gla_inputs(heads, dim, vdim, sum(lengths), dtype)
    for t in (qkv.view(sum(lengths), -1)[:, 2 * heads * dim:], gate):
        t.view(sum(lengths), heads, vdim)[..., true:] = 0
    bias, norm, before = rnd(heads * dim, seed=5) + 1.0, rnd(vdim, seed=6), rnd(5, heads, dim, vdim, seed=7)
    before[..., true:] = 0
    state, out = before.to(DEV), torch.full((sum(lengths), heads * vdim + 8), 5.0, dtype=dtype, device=DEV)
    if heads * vdim % 8:
        out = torch.full((sum(lengths), heads * vdim), 5.0, dtype=dtype, device=DEV)
    hops.gla_prefill(wide(qkv, 24), z.to(DEV), bias.to(DEV), norm.to(DEV), wide(gate, 8), state, out[:, : heads * vdim], Batch(slots, starts, lengths),
                     true, dim ** -0.5, 4.0, eps, serial=serial)
    row = 0
    for slot, start, n in zip(slots, starts, lengths):
        first = before[slot] if start else torch.zeros(heads, dim, vdim)
        want, last = gla_want(qkv[row: row + n], z[row: row + n], gate[row: row + n], bias, norm, heads, dim, vdim, true, dim ** -0.5, 4.0, eps, first)
        close(out[row: row + n, : heads * vdim], want, dtype, f"length {n}", 2.0)
        close(state[slot], last, torch.float32, f"state after {n}", 2.0 if dt == "f32" else 20.0)
        row += n
    assert torch.equal(state[3].cpu(), before[3])


@pytest.mark.parametrize("segments", [(64, 8), (128, 4), (512, 1)])
@pytest.mark.parametrize("tau", [1.0, 30.0])
def test_gla_segments(hops, segments, tau):
    """Also with gates near one (far tokens matter) and gates that forget at once."""
    heads, dim, vdim, lengths, slots, starts, eps = 2, 64, 96, [500, 40, 260], [0, 2, 1], [0, 4, 0], 1e-5
    qkv, z, gate = gla_inputs(heads, dim, vdim, sum(lengths), torch.bfloat16, seed=20)
    z[:, ::7] = -90.0
    bias, norm, before = torch.full((heads * dim,), 3.0), rnd(vdim, seed=6), rnd(3, heads, dim, vdim, seed=7)
    state, out = before.to(DEV), torch.empty(sum(lengths), heads * vdim, dtype=torch.bfloat16, device=DEV)
    hops.gla_prefill(qkv.to(DEV), z.to(DEV), bias.to(DEV), norm.to(DEV), gate.to(DEV), state, out, Batch(slots, starts, lengths), vdim,
                     dim ** -0.5, tau, eps, segments=segments)
    row = 0
    for slot, start, n in zip(slots, starts, lengths):
        first = before[slot] if start else torch.zeros(heads, dim, vdim)
        want, last = gla_want(qkv[row: row + n], z[row: row + n], gate[row: row + n], bias, norm, heads, dim, vdim, vdim, dim ** -0.5, tau, eps, first)
        close(out[row: row + n], want, torch.bfloat16, f"length {n}", 2.0)
        close(state[slot], last, torch.float32, f"state after {n}", 20.0)
        row += n


@pytest.mark.parametrize("dt", DT)
@pytest.mark.parametrize("heads,dim,vdim,true", GLA_SIZES)
def test_gla_decode(hops, dt, heads, dim, vdim, true):
    dtype, batch, rank, eps = DT[dt], 4, 24, 1e-4
    width = heads * (2 * dim + vdim)
    x = rnd(batch, width + rank, seed=1, dtype=dtype)
    x[:, 2 * heads * dim: width].view(batch, heads, vdim)[..., true:] = 0
    gate, w_low = rnd(batch, heads * vdim, seed=2, dtype=dtype), rnd(heads * dim, rank, seed=3, dtype=dtype, scale=0.5)
    bias, norm, before = rnd(heads * dim, seed=5), rnd(vdim, seed=6), rnd(batch, heads, dim, vdim, seed=7)
    before[..., true:] = 0
    state, out = before.to(DEV), torch.empty(batch, heads * vdim, dtype=dtype, device=DEV)
    pos, active = torch.tensor([0, 3, 5, 2], device=DEV), torch.tensor([1, 1, 0, 1], device=DEV)
    xd = wide(x, 8 - (width + rank) % 8 if (width + rank) % 8 else 8)
    if width % 8:                                              # the low-rank part must start on a 16-byte boundary
        pytest.skip("projection layout is padded by the caller")
    hops.gla_decode(xd[:, :width], xd[:, width:], w_low.to(DEV), bias.to(DEV), norm.to(DEV), gate.to(DEV), state, out, pos, active, true, dim ** -0.5,
                    4.0, eps)
    z = x[:, width:].double() @ w_low.double().T
    for b in range(batch):
        if not active[b]:
            assert torch.equal(state[b].cpu(), before[b])
            continue
        first = before[b] if pos[b] else torch.zeros(heads, dim, vdim)
        want, last = gla_want(x[b: b + 1, :width], z[b: b + 1], gate[b: b + 1], bias, norm, heads, dim, vdim, true, dim ** -0.5, 4.0, eps, first)
        close(out[b: b + 1], want, dtype, f"slot {b}", 2.0)
        close(state[b], last, torch.float32, f"state {b}", 2.0 if dt == "f32" else 4.0)
