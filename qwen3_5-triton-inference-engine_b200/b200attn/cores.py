"""Sublayers as cores between two shared products: windowed attention with grouped heads, state space, gated linear attention,
gated feed-forward.  A core turns columns of one input projection into columns of one activation matrix, so that everything
which reads the same normed input (mixers side by side, a mixer and a feed-forward) costs one product in and one out
(`FusedUnit`): the weights are stacked when they are loaded, and scales of the parts live in the cores' last steps.

    in_size, out_size                    columns a core takes and gives (padded layout)
    shapes(width), measure(shapes)       its tensors; sizes that only a tensor's shape tells
    load(get, width_p, dtype, device)    -> (input rows [in_size, width_p], output columns [width_p, out_size])
    allocate(engine)                     cache or state, indexed by page or by slot
    prefill(x, out, batch, engine, state)          packed tokens; x and out are column ranges of the unit's matrices
    decode(x, out, engine, state, first, last)     one token per slot, no host value that changes from step to step; first and
                                                   last: overlap flags of its first and its last kernel
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from . import hybrid_ops as hops
from . import ops
from .mixers import Rotation, _fp32, padded, round_up


def _by_head(w, heads: int, size: int, size_p: int, *rest: int):
    """Rows of w in heads of `size`, every head padded to size_p (and the other dimension to rest)."""
    return padded(w.view(heads, size, *w.shape[1:]), heads, size_p, *rest).flatten(0, 1)


def _out_by_head(w, heads: int, size: int, size_p: int, width_p: int):
    return padded(w.view(w.shape[0], heads, size), width_p, heads, size_p).flatten(1, 2)


def one_kernel(first: int, last: int) -> int:
    """Overlap flags of a kernel that is both: starts as the first, triggers as the last."""
    return (first & ops.OVERLAP_START) | (last & ops.OVERLAP_TRIGGER)


class Core:
    def __init__(self, prefix: str, scale: float):
        self.prefix, self.scale = prefix, float(scale)

    def measure(self, shape_of) -> None:
        """shape_of(name): shape of one of the core's tensors in a checkpoint."""


# -------------------------------------------------------------------------------------------------- windowed attention
class WindowAttention(Core):
    """Grouped query heads over a sliding window, biases on q, k and v, halves of the heads rotated against one another, outputs
    times sigmoid of a gate.  Keys and values may differ in size; a cache row is [key | value]."""

    def __init__(self, mixer: dict, eps: float, prefix: str = "", scale: float = 1.0):
        super().__init__(prefix, scale)
        self.heads, self.kv_heads, self.dim, self.vdim = (int(mixer[n]) for n in ("heads", "kv_heads", "dim", "vdim"))
        self.score_scale, self.window = float(mixer["scale"]), int(mixer["mask"]["size"])
        self.rotation = Rotation.from_config(mixer["rot"])
        assert self.heads % self.kv_heads == 0 and self.window >= 1
        assert self.rotation.dims % 2 == 0 and self.rotation.dims <= self.dim
        self.dim_p, self.vdim_p = round_up(self.dim, 32), round_up(self.vdim, 64)
        self.pitch = round_up(self.dim_p + self.vdim_p, 64)
        self.out_size = self.heads * self.vdim_p
        self.qkv = (self.heads + self.kv_heads) * self.dim_p + self.kv_heads * self.vdim_p
        self.in_size = self.qkv + self.out_size

    def shapes(self, width: int) -> dict:
        h, g = self.heads, self.kv_heads
        sizes = {"q": h * self.dim, "k": g * self.dim, "v": g * self.vdim}
        out = {n: (rows, width) for n, rows in sizes.items()} | {f"{n}.b": (rows,) for n, rows in sizes.items()}
        return out | {"g": (h * self.vdim, width), "o": (width, h * self.vdim)}

    def load(self, get, width_p: int, dtype, device):
        parts = {"q": (self.heads, self.dim, self.dim_p), "k": (self.kv_heads, self.dim, self.dim_p),
                 "v": (self.kv_heads, self.vdim, self.vdim_p), "g": (self.heads, self.vdim, self.vdim_p)}
        self.bias = torch.cat([_fp32(_by_head(get(f"{n}.b"), *parts[n]), device) for n in ("q", "k", "v")])
        return (torch.cat([_by_head(get(n), *sizes, width_p) for n, sizes in parts.items()]),
                _out_by_head(get("o"), self.heads, self.vdim, self.vdim_p, width_p))

    def allocate(self, engine) -> dict:
        splits = hops.window_decode_splits(engine.batch, self.heads, self.kv_heads, min(self.window, engine.max_context), engine.sm_count)
        return {"angles": engine.rotation_table(self.rotation),
                "cache": hops.allocate_window_cache(engine.num_pages, self.kv_heads, self.pitch, engine.dtype, device=engine.device),
                "workspace": engine.shared_workspace(self.heads, self.vdim_p, splits)}

    def prefill(self, x, out, batch, engine, state) -> None:
        span, cache = batch.context(self.window), state["cache"]
        ctx = torch.empty((span.keys, self.kv_heads, self.pitch), dtype=engine.dtype, device=engine.device)
        hops.window_prep(x, self.bias, batch.pos, batch.slot_of, None, engine.block_table, state["angles"], cache, self.heads, self.dim_p,
                         self.vdim_p, ctx=ctx, ctx_row=span.rows)
        if span.max_old:
            hops.window_gather(cache, ctx, engine.block_table, batch.slots, span.cu, span.first, span.max_old)
        hops.window_prefill(x, ctx, x[:, self.qkv:], out, batch.cu, span.cu, batch.start, span.first, batch.max_len, self.heads, self.dim_p,
                            self.dim, self.vdim_p, self.window, self.score_scale, self.scale)

    def decode(self, x, out, engine, state, first: int, last: int) -> None:
        then = engine.then(True)
        hops.window_prep(x, self.bias, engine.pos, None, engine.active, engine.block_table, state["angles"], state["cache"], self.heads,
                         self.dim_p, self.vdim_p, overlap=first)
        hops.window_decode(x, state["cache"], engine.block_table, engine.pos, engine.active, state["workspace"], self.dim_p, self.window,
                           self.score_scale, overlap=then)
        hops.window_merge(state["workspace"], x[:, self.qkv:], out, self.scale, overlap=last)


# --------------------------------------------------------------------------------------------------------- state space
class StateSpace(Core):
    """State space with one decay per head and token (Mamba-2): a short convolution over [x | B | C], B and C shared by groups of
    heads, gate before the norm over equal parts of the channels."""

    def __init__(self, mixer: dict, eps: float, prefix: str = "", scale: float = 1.0):
        super().__init__(prefix, scale)
        self.eps = eps
        self.heads, self.vdim, self.dim, self.groups = (int(mixer[n]) for n in ("heads", "vdim", "state", "groups"))
        self.taps, self.norm_groups = int(mixer["conv"]), int(mixer["norm_groups"])
        assert self.heads % self.groups == 0 and self.heads * self.vdim % self.norm_groups == 0
        self.dim_p, self.vdim_p, self.taps_p = round_up(self.dim, 16), round_up(self.vdim, 16), hops.conv_taps(self.taps)
        self.out_size = self.heads * self.vdim_p
        self.channels = self.out_size + 2 * self.groups * self.dim_p
        self.dt_at = self.out_size + self.channels
        self.in_size = self.dt_at + round_up(self.heads, 8)

    def shapes(self, width: int) -> dict:
        inner, bc, h = self.heads * self.vdim, self.groups * self.dim, self.heads
        return {"in": (2 * inner + 2 * bc + h, width), "conv": (inner + 2 * bc, self.taps), "conv.b": (inner + 2 * bc,),
                "dt_bias": (h,), "A_log": (h,), "D": (h,), "norm": (inner,), "o": (width, inner)}

    def _channels(self, w, *rest: int):
        """Rows of w, one per channel of [x | B | C], in the padded order."""
        inner, bc = self.heads * self.vdim, self.groups * self.dim
        x, b, c = w.split([inner, bc, bc])
        return torch.cat((_by_head(x, self.heads, self.vdim, self.vdim_p, *rest), _by_head(b, self.groups, self.dim, self.dim_p, *rest),
                          _by_head(c, self.groups, self.dim, self.dim_p, *rest)))

    def load(self, get, width_p: int, dtype, device):
        inner, bc = self.heads * self.vdim, self.groups * self.dim
        z, xbc, dt = get("in").split([inner, inner + 2 * bc, self.heads])
        taps = self._channels(get("conv"), self.taps).flip(1).t()               # the current token's weights first
        self.conv = _fp32(padded(taps.contiguous(), self.taps_p, self.channels), device)
        self.conv_bias = _fp32(self._channels(get("conv.b")), device)
        self.dt_bias, self.a_log, self.skip = (_fp32(get(n), device) for n in ("dt_bias", "A_log", "D"))
        self.norm = _fp32(_by_head(get("norm") * self.scale, self.heads, self.vdim, self.vdim_p), device)
        return (torch.cat((_by_head(z, self.heads, self.vdim, self.vdim_p, width_p), self._channels(xbc, width_p),
                           padded(dt, round_up(self.heads, 8), width_p))),
                _out_by_head(get("o"), self.heads, self.vdim, self.vdim_p, width_p))

    def allocate(self, engine) -> dict:
        f32 = dict(dtype=torch.float32, device=engine.device)
        return {"state": torch.zeros(engine.batch, self.heads, self.dim_p, self.vdim_p, **f32),
                "ring": torch.zeros(engine.batch, self.taps_p, self.channels, **f32)}

    def prefill(self, x, out, batch, engine, state) -> None:
        xbc = hops.conv_prefill(x[:, self.out_size: self.dt_at], self.conv, self.conv_bias, state["ring"], batch)
        y = hops.ssd_prefill(xbc, x[:, self.dt_at:], self.dt_bias, self.a_log, self.skip, state["state"], self.groups, batch)
        hops.gated_group_norm(y, x[:, : self.out_size], self.norm, out, self.heads, self.vdim, self.norm_groups, self.eps)

    def decode(self, x, out, engine, state, first: int, last: int) -> None:
        y = hops.ssd_decode(x[:, self.out_size: self.dt_at], x[:, self.dt_at:], self.dt_bias, self.a_log, self.skip, self.conv,
                            self.conv_bias, state["ring"], state["state"], self.groups, engine.pos, engine.active, overlap=first)
        hops.gated_group_norm(y, x[:, : self.out_size], self.norm, out, self.heads, self.vdim, self.norm_groups, self.eps,
                              overlap=last)


# ----------------------------------------------------------------------------------------------- gated linear attention
class GatedLinear(Core):
    """Gated linear attention: a decay per key channel, sigmoid(z)^(1/tau) with z from a low-rank projection; head norm, silu
    gate.  The rank is the checkpoint's."""
    RANK = 16                                    # of random weights

    def __init__(self, mixer: dict, eps: float, prefix: str = "", scale: float = 1.0):
        super().__init__(prefix, scale)
        self.eps, self.tau = eps, float(mixer["tau"])
        self.heads, self.dim, self.vdim = (int(mixer[n]) for n in ("heads", "dim", "vdim"))
        self.dim_p, self.vdim_p = round_up(self.dim, 16), round_up(self.vdim, 16)
        self.out_size = self.heads * self.vdim_p
        self.gate_at = 2 * self.heads * self.dim_p + self.out_size
        self.low_at = self.gate_at + self.out_size
        self._set_rank(self.RANK)

    def _set_rank(self, rank: int) -> None:
        self.rank, self.rank_p = rank, round_up(rank, 8)
        self.in_size = self.low_at + self.rank_p

    def measure(self, shape_of) -> None:
        self._set_rank(int(shape_of("a1")[0]))

    def shapes(self, width: int) -> dict:
        n, m = self.heads * self.dim, self.heads * self.vdim
        return {"q": (n, width), "k": (n, width), "v": (m, width), "g": (m, width), "a1": (self.rank, width), "a2": (n, self.rank),
                "a2.b": (n,), "norm": (self.vdim,), "o": (width, m)}

    def load(self, get, width_p: int, dtype, device):
        keys, values = (self.heads, self.dim, self.dim_p), (self.heads, self.vdim, self.vdim_p)
        self.w_low = _by_head(get("a2"), *keys, self.rank_p).to(device, dtype)
        self.bias = _fp32(_by_head(get("a2.b"), *keys), device)
        self.norm = _fp32(padded(get("norm") * self.scale, self.vdim_p), device)
        return (torch.cat((_by_head(get("q"), *keys, width_p), _by_head(get("k"), *keys, width_p), _by_head(get("v"), *values, width_p),
                           _by_head(get("g"), *values, width_p), padded(get("a1"), self.rank_p, width_p))),
                _out_by_head(get("o"), *values, width_p))

    def allocate(self, engine) -> dict:
        return {"state": torch.zeros(engine.batch, self.heads, self.dim_p, self.vdim_p, dtype=torch.float32, device=engine.device)}

    def _split(self, x):
        return x[:, : self.gate_at], x[:, self.gate_at: self.low_at], x[:, self.low_at:]

    def prefill(self, x, out, batch, engine, state) -> None:
        qkv, gate, low = self._split(x)
        z = F.linear(low, self.w_low) if x.dtype == torch.float32 else torch.mm(low, self.w_low.t(), out_dtype=torch.float32)
        hops.gla_prefill(qkv, z, self.bias, self.norm, gate, state["state"], out, batch, self.vdim, self.dim ** -0.5, self.tau, self.eps)

    def decode(self, x, out, engine, state, first: int, last: int) -> None:
        qkv, gate, low = self._split(x)
        hops.gla_decode(qkv, low, self.w_low, self.bias, self.norm, gate, state["state"], out, engine.pos, engine.active, self.vdim,
                        self.dim ** -0.5, self.tau, self.eps, overlap=one_kernel(first, last))


# -------------------------------------------------------------------------------------------------------- feed-forward
class GatedMLP(Core):
    ACTIVATIONS = {"silu": hops.ACT_SILU, "gelu_tanh": hops.ACT_GELU_TANH}

    def __init__(self, mlp: dict, activation: str):
        super().__init__("", 1.0)
        self.ff, self.act = int(mlp["ff"]), self.ACTIVATIONS[activation]
        self.out_size = round_up(self.ff, 64)
        self.in_size = 2 * self.out_size

    def shapes(self, width: int) -> dict:
        return {"gate": (self.ff, width), "up": (self.ff, width), "down": (width, self.ff)}

    def load(self, get, width_p: int, dtype, device):
        return (torch.cat([padded(get(n), self.out_size, width_p) for n in ("gate", "up")]), padded(get("down"), width_p, self.out_size))

    def allocate(self, engine) -> dict:
        return {}

    def prefill(self, x, out, batch, engine, state) -> None:
        hops.gated_act(x, self.out_size, out, self.act)

    def decode(self, x, out, engine, state, first: int, last: int) -> None:
        hops.gated_act(x, self.out_size, out, self.act, overlap=one_kernel(first, last))


# ---------------------------------------------------------------------------------------------------- layers from cores
class CoreMixer:
    """A layer's mixer made of cores that read the same input and add their outputs."""

    def __init__(self, cores: list):
        self.cores = cores

    def check(self, stack: list) -> None:
        pass

    def measure(self, shape_of) -> None:
        for core in self.cores:
            core.measure(lambda n, core=core: shape_of(core.prefix + n))

    def shapes(self, width: int) -> dict:
        return {core.prefix + n: shape for core in self.cores for n, shape in core.shapes(width).items()}


class SideBySide(CoreMixer):
    """left_scale * windowed attention + right_scale * state space."""
    kind = "parallel"

    def __init__(self, mixer: dict, eps: float, index: int):
        super().__init__([WindowAttention(mixer["left"], eps, "left.", mixer["left_scale"]),
                          StateSpace(mixer["right"], eps, "right.", mixer["right_scale"])])


class GatedLinearMixer(CoreMixer):
    kind = "gla"

    def __init__(self, mixer: dict, eps: float, index: int):
        super().__init__([GatedLinear(mixer, eps)])


class FusedUnit:
    """Cores that read one input: one product in, the cores on column ranges of its result, one product out."""

    def __init__(self, layer: int, parts: list):
        """parts: (prefix of the tensors, core)"""
        self.layer, self.parts = layer, parts

    def load(self, get, width_p: int, dtype, device) -> None:
        rows, cols = zip(*(core.load(lambda n, pre=pre: get(pre + n), width_p, dtype, device) for pre, core in self.parts))
        self.ins = [r.shape[0] for r in rows]
        self.outs = [c.shape[1] for c in cols]
        # the product out, in parts along K that the weight-streaming kernel splits over pairs of CTAs
        used = sum(self.outs)
        parts = -(-used // ops.SKINNY_GEMM_PAIR_MAX_K)
        part = next((n for n in range(round_up(-(-used // parts), 128), ops.SKINNY_GEMM_PAIR_MAX_K + 1, 128)
                     if ops.skinny_gemm_supports(1, width_p, n)), round_up(-(-used // parts), 128))
        size = part * parts
        self.pad = size - used
        self.w_in = torch.cat(rows).to(device, dtype)
        self.w_out = padded(torch.cat(cols, dim=1), width_p, size).to(device, dtype)
        self.part = part
        self.w_parts = list(self.w_out.split(part, dim=1))

    def keys(self):
        """Where the cores' caches and states live in the engine's table."""
        return [(self.layer, j) for j in range(len(self.parts))]

    def allocate(self, engine) -> dict:
        return {key: core.allocate(engine) for key, (_, core) in zip(self.keys(), self.parts)}

    def _ranges(self, fused, act):
        return zip(self.keys(), self.parts, fused.split(self.ins, dim=1), act.split([*self.outs, self.pad], dim=1))

    def prefill(self, h, batch, engine, states):
        fused = engine.linear(h, self.w_in)
        act = torch.empty((h.shape[0], sum(self.outs) + self.pad), dtype=h.dtype, device=h.device)
        if self.pad:
            act[:, -self.pad:].zero_()
        for key, (_, core), x, out in self._ranges(fused, act):
            core.prefill(x, out, batch, engine, states[key])
        return engine.linear(act, self.w_out)

    def starts_own(self, engine) -> bool:
        """Whether the product in runs on the weight-streaming kernel: its form for inputs of up to 1280 takes any number of
        outputs, the split one meets after every 16 outputs and is for few."""
        n, k = self.w_in.shape
        return engine.streams_weight(self.w_in) and (k <= ops.SKINNY_GEMM_MAX_K or n <= 8192)

    def out_parts(self, engine):
        """(weight, first and last column) of the product's parts in a decode step, or None: one library product."""
        if not all(engine.streams_weight(w) for w in self.w_parts):
            return None
        return [(w, n * self.part, (n + 1) * self.part) for n, w in enumerate(self.w_parts)]

    def decode(self, h, engine, states, nxt: bool):
        """Several cores: the first runs on the current stream, the others beside it on a second one."""
        own, side = engine.then(True), len(self.parts) > 1
        outs = self.out_parts(engine)
        own_out = outs is not None
        fused = engine.proj(h, self.w_in, not side) if self.starts_own(engine) else F.linear(h, self.w_in)
        act = engine.zero_scratch(sum(self.outs), self.pad)      # padding columns stay zero
        ranges = list(self._ranges(fused, act))
        plain = own & ~ops.OVERLAP_START                          # behind a kernel of another stream
        if side:
            with torch.cuda.stream(engine.fork()):
                for n, (key, (_, core), x, out) in enumerate(ranges[1:]):
                    core.decode(x, out, engine, states[key], own if n else plain, own if n + 2 < len(ranges) else own & ~ops.OVERLAP_TRIGGER)
        key, (_, core), x, out = ranges[0]
        core.decode(x, out, engine, states[key], plain if side else own, engine.then(own_out and not side))
        if side:
            engine.join()
        if not own_out:
            return F.linear(act, self.w_out)
        y = torch.empty((len(outs), act.shape[0], self.w_out.shape[0]), dtype=act.dtype, device=act.device)
        for n, (weight, lo, hi) in enumerate(outs):
            flags = engine.then(nxt or n + 1 < len(outs))
            ops.skinny_gemm_part(act[:, lo:hi], weight, y[n], overlap=flags & ~ops.OVERLAP_START if side and n == 0 else flags)
        return y
