"""Sequence mixers of hybrid stacks: latent attention, minGRU, HGRN2.  Each class holds one layer's sizes and weights in the
padded layout of the kernels (feature sizes rounded up with zero rows and columns, so that a kernel never sees a ragged
edge) and knows what a slot keeps for it:

    allocate(engine)                        the layer's cache or state, indexed by page or by slot
    prefill(h, batch, engine, states)       packed tokens of several sequences (`hybrid.PackedBatch`)
    decode(h, engine, states, nxt)          one token per slot; no host value changes from step to step.  Kernels of this
                                            package that follow one another start early (`engine.then(own)`: whether the
                                            kernel behind is one of them); nxt: what follows the mixer

`shapes(width)` lists a layer's tensors (name -> shape) for loading and for random initialisation.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import hybrid_ops as hops
from . import ops

def round_up(n: int, to: int) -> int:
    return -(-n // to) * to


def padded(w: torch.Tensor, *sizes: int) -> torch.Tensor:
    """w with every dimension zero-padded at its end to `sizes`."""
    assert w.dim() == len(sizes) and all(a <= b for a, b in zip(w.shape, sizes))
    if tuple(w.shape) == sizes:
        return w
    out = w.new_zeros(sizes)
    out[tuple(slice(0, n) for n in w.shape)] = w
    return out


def _fp32(w, device):
    return w.to(device=device, dtype=torch.float32).contiguous()


# ------------------------------------------------------------------------------------------------------------ rotation
@dataclass(frozen=True)
class Rotation:
    """Interleaved rotary positions on the first `dims` dimensions, optionally YaRN-scaled."""
    dims: int
    base: float
    scaling: tuple | None = None          # (factor, original, fast, slow)

    @classmethod
    def from_config(cls, rot: dict) -> "Rotation":
        s = rot.get("scaling")
        return cls(int(rot["dims"]), float(rot["base"]),
                   None if s is None else (float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"])))

    def frequencies(self) -> torch.Tensor:
        i = torch.arange(self.dims // 2, dtype=torch.float64)
        f = self.base ** (-2.0 * i / self.dims)
        if self.scaling is None:
            return f
        factor, original, fast, slow = self.scaling

        def dim_of(turns: float) -> float:
            return self.dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(self.base))

        lo, hi = max(math.floor(dim_of(fast)), 0), min(math.ceil(dim_of(slow)), self.dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / factor * ramp + f * (1.0 - ramp)

    def amplitude(self) -> float:
        return 1.0 if self.scaling is None else 0.1 * math.log(self.scaling[0]) + 1.0

    def table(self, positions: int, device) -> torch.Tensor:
        """fp32 (cos, sin) [positions, dims/2, 2] with the amplitude inside, from float64 angles."""
        angle = torch.arange(positions, dtype=torch.float64)[:, None] * self.frequencies()[None, :]
        return (torch.stack((angle.cos(), angle.sin()), dim=-1) * self.amplitude()).to(torch.float32).to(device).contiguous()


# ---------------------------------------------------------------------------------------------------- latent attention
class LatentAttention:
    kind = "latent_attention"

    def __init__(self, mixer: dict, eps: float, index: int):
        self.index, self.eps = index, eps
        self.heads, self.dim, self.vdim = mixer["heads"], mixer["dim"], mixer["vdim"]
        self.rank, self.rot_dim, self.q_rank = mixer["kv_rank"], mixer["rot_dim"], mixer["q_rank"]
        self.scale, self.window = float(mixer["scale"]), int(mixer["mask"]["size"])
        self.rotation = Rotation.from_config(mixer["rot"])
        self.kv_from = mixer.get("kv_from")          # layer whose latents this one reads, None = its own
        self.source = index if self.kv_from is None else int(self.kv_from)
        assert self.rotation.dims % 2 == 0 and self.rotation.dims <= self.rot_dim and self.window >= 1
        self.dim_p, self.vdim_p, self.rank_p, self.rot_p, self.q_rank_p = (
            round_up(n, 64) for n in (self.dim, self.vdim, self.rank, self.rot_dim, self.q_rank))

    def check(self, stack: list) -> None:
        """A shared latent must come from an earlier latent layer that has its own, of the same shape and rotation."""
        if self.kv_from is None:
            return
        assert 0 <= self.source < self.index, f"layer {self.index}: kv_from must name an earlier layer"
        other = stack[self.source]
        assert isinstance(other, LatentAttention) and other.kv_from is None, f"layer {self.source} keeps no latent of its own"
        assert (other.rank, other.rot_dim, other.rotation) == (self.rank, self.rot_dim, self.rotation), (
            f"layer {self.index}: latent shape or rotation differs from layer {self.source}")

    def shapes(self, width: int) -> dict:
        own = {"dkv": (self.rank + self.rot_dim, width), "dkv.norm": (self.rank,)} if self.kv_from is None else {}
        return {"dq": (self.q_rank, width), "dq.norm": (self.q_rank,),
                "uq": (self.heads * (self.dim + self.rot_dim), self.q_rank), **own,
                "uk": (self.heads * self.dim, self.rank), "uv": (self.heads * self.vdim, self.rank),
                "o": (width, self.heads * self.vdim)}

    def load(self, get, width_p: int, dtype, device) -> None:
        h = self.heads
        down = [padded(get("dq"), self.q_rank_p, width_p)]
        self.q_norm = _fp32(padded(get("dq.norm"), self.q_rank_p), device)
        self.kv_norm = None
        if self.kv_from is None:
            dkv = get("dkv")
            down += [padded(dkv[: self.rank], self.rank_p, width_p), padded(dkv[self.rank:], self.rot_p, width_p)]
            self.kv_norm = _fp32(padded(get("dkv.norm"), self.rank_p), device)
        self.down = torch.cat(down).to(device, dtype)
        uq = get("uq").view(h, self.dim + self.rot_dim, self.q_rank)
        self.uq = torch.cat((padded(uq[:, : self.dim], h, self.dim_p, self.q_rank_p),
                             padded(uq[:, self.dim:], h, self.rot_p, self.q_rank_p)), dim=1).flatten(0, 1).to(device, dtype)
        uk = padded(get("uk").view(h, self.dim, self.rank), h, self.dim_p, self.rank_p)
        uv = padded(get("uv").view(h, self.vdim, self.rank), h, self.vdim_p, self.rank_p)
        self.ukv = torch.cat((uk.flatten(0, 1), uv.flatten(0, 1))).to(device, dtype)        # one expansion product
        cut = h * self.dim_p
        self.uk = self.ukv[:cut].view(h, self.dim_p, self.rank_p)
        self.uv = self.ukv[cut:].view(h, self.vdim_p, self.rank_p)
        o = get("o")
        self.o = padded(o.view(o.shape[0], h, self.vdim), width_p, h, self.vdim_p).flatten(1, 2).to(device, dtype)

    def allocate(self, engine) -> dict:
        state = {"angles": engine.rotation_table(self.rotation)}
        if self.kv_from is None:
            state["cache"] = hops.allocate_latent_cache(engine.num_pages, self.rank_p + self.rot_p, engine.dtype,
                                                        device=engine.device)
        splits = hops.latent_decode_splits(engine.batch, self.heads, min(self.window, engine.max_context), engine.sm_count)
        state["workspace"] = engine.shared_workspace(self.heads, self.rank_p, splits)
        return state

    def prefill(self, h, batch, engine, states):
        state, cache = states[self.index], states[self.source]["cache"]
        own = self.kv_from is None
        fused = engine.linear(h, self.down)
        cq = hops.latent_prep(fused, self.q_norm, self.kv_norm, batch.pos, batch.slot_of, None, engine.block_table,
                              state["angles"], cache if own else None, self.q_rank, self.rank_p, self.rank, self.eps)
        q = engine.linear(cq, self.uq).view(-1, self.heads, self.dim_p + self.rot_p)
        hops.rope_interleaved(q, self.dim_p, batch.pos, state["angles"])
        span = batch.context(self.window)
        ctx = batch.kept.get((self.source, self.window))
        if ctx is None:
            ctx = hops.latent_gather(cache, engine.block_table, batch.slots, span.cu, span.first, span.keys, span.max_keys)
            batch.kept[self.source, self.window] = ctx
        kv = engine.linear(ctx[:, : self.rank_p], self.ukv)
        out = hops.latent_prefill(q, kv, ctx, batch.cu, span.cu, batch.start, span.first, batch.max_len, self.dim,
                                  self.rot_dim, self.vdim_p, self.rank_p, self.window, self.scale)
        return engine.linear(out, self.o)

    def first_weight(self):
        return self.down

    def decode(self, h, engine, states, nxt: bool):
        state, cache, then = states[self.index], states[self.source]["cache"], engine.then
        own = self.kv_from is None
        fused = engine.proj(h, self.down, True)
        cq = hops.latent_prep(fused, self.q_norm, self.kv_norm, engine.pos, None, engine.active, engine.block_table,
                              state["angles"], cache if own else None, self.q_rank, self.rank_p, self.rank, self.eps,
                              overlap=then(engine.streams_weight(self.uq)))
        q = engine.proj(cq, self.uq, True).view(-1, self.heads, self.dim_p + self.rot_p)
        q = hops.latent_absorb(q, self.uk, engine.pos, state["angles"], overlap=then(True))
        hops.latent_decode(q, cache, engine.block_table, engine.pos, engine.active, state["workspace"], self.window, self.scale,
                           overlap=then(True))
        out = hops.latent_value(state["workspace"], self.uv, engine.dtype, overlap=then(engine.streams_weight(self.o)))
        return engine.proj(out, self.o, nxt)


# -------------------------------------------------------------------------------------------------------------- minGRU
class MinGRU:
    kind = "mingru"

    def __init__(self, mixer: dict, eps: float, index: int):
        self.index, self.size = index, mixer["width"]
        self.size_p = round_up(self.size, 64)

    def check(self, stack: list) -> None:
        pass

    def shapes(self, width: int) -> dict:
        n = self.size
        return {"z": (n, width), "z.b": (n,), "x": (n, width), "x.b": (n,), "g": (n, width), "o": (width, n)}

    def load(self, get, width_p: int, dtype, device) -> None:
        self.zxg = torch.cat([padded(get(n), self.size_p, width_p) for n in ("z", "x", "g")]).to(device, dtype)
        self.bias = torch.cat([_fp32(padded(get(n), self.size_p), device) for n in ("z.b", "x.b")])
        self.o = padded(get("o"), width_p, self.size_p).to(device, dtype)

    def allocate(self, engine) -> dict:
        return {"state": torch.zeros(engine.batch, self.size_p, dtype=torch.float32, device=engine.device)}

    def prefill(self, h, batch, engine, states):
        out = hops.mingru_prefill(engine.linear(h, self.zxg), self.bias, states[self.index]["state"], batch)
        return engine.linear(out, self.o)

    def first_weight(self):
        return self.zxg

    def decode(self, h, engine, states, nxt: bool):
        out = hops.mingru_decode(engine.proj(h, self.zxg, True), self.bias, states[self.index]["state"], engine.pos,
                                 engine.active, overlap=engine.then(engine.streams_weight(self.o)))
        return engine.proj(out, self.o, nxt)


# --------------------------------------------------------------------------------------------------------------- HGRN2
class HGRN2:
    kind = "hgrn2"

    def __init__(self, mixer: dict, eps: float, index: int):
        self.index, self.eps = index, eps
        self.heads, self.dim, self.vdim = mixer["heads"], mixer["dim"], mixer["vdim"]
        self.dim_p, self.vdim_p = round_up(self.dim, 16), round_up(self.vdim, 16)

    def check(self, stack: list) -> None:
        pass

    def shapes(self, width: int) -> dict:
        n = self.heads * self.dim
        return {"q": (n, width), "f": (n, width), "f.b": (n,), "lower": (n,), "v": (self.heads * self.vdim, width),
                "norm": (self.vdim,), "o": (width, self.heads * self.vdim)}

    def _by_head(self, w, size: int, size_p: int, width_p: int):
        return padded(w.view(self.heads, size, w.shape[1]), self.heads, size_p, width_p).flatten(0, 1)

    def load(self, get, width_p: int, dtype, device) -> None:
        self.qfv = torch.cat((self._by_head(get("q"), self.dim, self.dim_p, width_p),
                              self._by_head(get("f"), self.dim, self.dim_p, width_p),
                              self._by_head(get("v"), self.vdim, self.vdim_p, width_p))).to(device, dtype)
        self.bias, self.lower = (_fp32(padded(get(n).view(self.heads, self.dim), self.heads, self.dim_p), device).flatten()
                                 for n in ("f.b", "lower"))
        self.norm = _fp32(padded(get("norm"), self.vdim_p), device)
        o = get("o")
        self.o = padded(o.view(o.shape[0], self.heads, self.vdim), width_p, self.heads, self.vdim_p).flatten(1, 2).to(device, dtype)

    def allocate(self, engine) -> dict:
        return {"state": torch.zeros(engine.batch, self.heads, self.dim_p, self.vdim_p, dtype=torch.float32,
                                     device=engine.device)}

    def prefill(self, h, batch, engine, states):
        out = hops.hgrn2_prefill(engine.linear(h, self.qfv), self.lower, self.bias, self.norm, states[self.index]["state"],
                                 batch, self.vdim, self.eps)
        return engine.linear(out, self.o)

    def first_weight(self):
        return self.qfv

    def decode(self, h, engine, states, nxt: bool):
        out = hops.hgrn2_decode(engine.proj(h, self.qfv, True), self.lower, self.bias, self.norm, states[self.index]["state"],
                                engine.pos, engine.active, self.vdim, self.eps,
                                overlap=engine.then(engine.streams_weight(self.o)))
        return engine.proj(out, self.o, nxt)


# -------------------------------------------------------------------------------------------------------- feed-forward
class SwiGLU:
    def __init__(self, ff: int):
        self.ff, self.ff_p = ff, round_up(ff, 64)

    def shapes(self, width: int) -> dict:
        return {"gate": (self.ff, width), "up": (self.ff, width), "down": (width, self.ff)}

    def load(self, get, width_p: int, dtype, device) -> None:
        self.gate_up = torch.cat([padded(get(n), self.ff_p, width_p) for n in ("gate", "up")]).to(device, dtype)
        self.down = padded(get("down"), width_p, self.ff_p).to(device, dtype)

    def _act(self, gate_up, overlap: int = 0):
        if gate_up.dtype == torch.float32:
            return hops.swiglu_f32(gate_up, self.ff_p)
        return ops.swiglu_fused(gate_up, self.ff_p, overlap=overlap)

    def prefill(self, h, engine):
        return engine.linear(self._act(engine.linear(h, self.gate_up)), self.down)

    def decode(self, h, engine, nxt: bool):
        flags = engine.then(engine.streams_weight(self.down))
        if engine.streams_weight(self.gate_up, swiglu=True):
            act = ops.skinny_gemm(h, self.gate_up, swiglu=True, overlap=flags)
        else:
            act = self._act(F.linear(h, self.gate_up), overlap=flags)
        return engine.proj(act, self.down, nxt)


MIXERS = {cls.kind: cls for cls in (LatentAttention, MinGRU, HGRN2)}
FEED_FORWARDS = {"dense": lambda mlp: SwiGLU(mlp["ff"])}
