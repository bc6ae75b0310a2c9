"""Decoder stacks whose layers are listed one by one in config.json: any order of the mixers of `mixers.py` and `cores.py`, an
optional feed-forward per layer.  What a family of such stacks fixes is its `Design`: several residual streams joined by
hyper-connections or one plain residual, norms with a single gain or a weight per channel, the feed-forward behind the mixer
or beside it on the same norm.  Served by `HybridEngine` through the same slots, pages, graph capture and batcher as every
other engine of the package.

config.json:  architecture, vocab, width, norm.eps, layers = [{type, mixer, mlp | null}, ...]; hyper-connected: streams;
optional: logit_softcap.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import numpy as np
import torch
import torch.nn.functional as F

from . import hybrid_ops as hops
from . import ops
from . import cores
from .cores import CoreMixer, FusedUnit, GatedMLP
from .mixers import FEED_FORWARDS, MIXERS, padded, round_up
from .slots import SlotEngine

MIXERS = MIXERS | {cls.kind: cls for cls in (cores.SideBySide, cores.GatedLinearMixer)}


@dataclass(frozen=True)
class Design:
    """What config.json does not say."""
    hyper: bool            # hyper-connected streams and norms with a single gain; else one residual and norm weights
    parallel: bool         # mixer and feed-forward read one norm and are added together; else one behind the other
    activation: str        # of the feed-forward's gate


DESIGNS = {"Tofilorn": Design(hyper=True, parallel=False, activation="silu"),
           "Dugilorn": Design(hyper=False, parallel=True, activation="gelu_tanh")}


@dataclass(frozen=True)
class HybridConfig:
    vocab: int
    width: int
    streams: int
    eps: float
    layers: tuple          # of the raw layer dictionaries
    design: Design
    softcap: float | None = None

    @classmethod
    def from_config(cls, config: dict) -> "HybridConfig":
        design, cap = DESIGNS[config["architecture"]], config.get("logit_softcap")
        return cls(int(config["vocab"]), int(config["width"]), int(config["streams"]) if design.hyper else 1,
                   float(config["norm"]["eps"]), tuple(config["layers"]), design, None if cap is None else float(cap))


# Units: what runs between two joints.  prefill(h, batch, engine, states) and decode(h, engine, states, nxt) give the
# sublayer's output; starts_own(engine): whether its first decode-step kernel is one of this package.
class MixerUnit:
    def __init__(self, layer: int, mixer):
        self.layer, self.mixer = layer, mixer

    def load(self, get, width_p, dtype, device) -> None:
        self.mixer.load(lambda n: get(f"mix.{n}"), width_p, dtype, device)

    def allocate(self, engine) -> dict:
        return {self.mixer.index: self.mixer.allocate(engine)}

    def prefill(self, h, batch, engine, states):
        return self.mixer.prefill(h, batch, engine, states)

    def starts_own(self, engine) -> bool:
        return engine.streams_weight(self.mixer.first_weight())

    def decode(self, h, engine, states, nxt: bool):
        return self.mixer.decode(h, engine, states, nxt)


class FeedForwardUnit:
    def __init__(self, layer: int, mlp):
        self.layer, self.mlp = layer, mlp

    def load(self, get, width_p, dtype, device) -> None:
        self.mlp.load(lambda n: get(f"mlp.{n}"), width_p, dtype, device)

    def allocate(self, engine) -> dict:
        return {}

    def prefill(self, h, batch, engine, states):
        return self.mlp.prefill(h, engine)

    def starts_own(self, engine) -> bool:
        return engine.streams_weight(self.mlp.gate_up, swiglu=True)

    def decode(self, h, engine, states, nxt: bool):
        return self.mlp.decode(h, engine, nxt)


class HybridWeights:
    """The layers of one stack with their weights on the device, in the kernels' padded layout."""

    def __init__(self, cfg: HybridConfig):
        self.cfg = cfg
        self.width_p, self.vocab_p = round_up(cfg.width, 64), round_up(cfg.vocab, 8)
        self.mixers, self.mlps = [], []
        for i, layer in enumerate(cfg.layers):
            if layer["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer '{layer['type']}' (known: {', '.join(sorted(MIXERS))})")
            self.mixers.append(MIXERS[layer["type"]](layer["mixer"], cfg.eps, i))
            mlp = layer["mlp"]
            if mlp is not None and mlp["kind"] not in FEED_FORWARDS:
                raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
            fused = cfg.design.parallel or cfg.design.activation != "silu"
            self.mlps.append(None if mlp is None else GatedMLP(mlp, cfg.design.activation) if fused else FEED_FORWARDS[mlp["kind"]](mlp))
        for mixer in self.mixers:
            mixer.check(self.mixers)
        self.units = [unit for i in range(len(self.mixers)) for unit in self._layer_units(i)]

    def _layer_units(self, i: int) -> list:
        mixer, mlp = self.mixers[i], self.mlps[i]
        ff = [("mlp.", mlp)] if mlp is not None else []
        if not isinstance(mixer, CoreMixer):
            if self.cfg.design.parallel and ff:
                raise ValueError(f"layer {i}: this mixer cannot share its norm with a feed-forward")
            return [MixerUnit(i, mixer)] + [FusedUnit(i, ff) if isinstance(mlp, GatedMLP) else FeedForwardUnit(i, mlp) for _ in ff]
        mix = [("mix." + core.prefix, core) for core in mixer.cores]
        if self.cfg.design.parallel:
            return [FusedUnit(i, mix + ff)]
        return [FusedUnit(i, mix)] + [FeedForwardUnit(i, mlp) if not isinstance(mlp, GatedMLP) else FusedUnit(i, ff) for _ in ff]

    def sublayers(self):
        """(layer, 1 = mixer, with the feed-forward where they share a norm / 2 = feed-forward) in the order they run."""
        for k, unit in enumerate(self.units):
            yield unit.layer, 2 if k and self.units[k - 1].layer == unit.layer else 1

    def shapes(self) -> dict:
        """name -> shape of every tensor of the checkpoint."""
        cfg, s = self.cfg, self.cfg.streams
        out = {"embed": (cfg.vocab, cfg.width)}
        for i, (mixer, mlp) in enumerate(zip(self.mixers, self.mlps)):
            out |= {f"l{i}.mix.{n}": shape for n, shape in mixer.shapes(cfg.width).items()}
            if mlp is not None:
                out |= {f"l{i}.mlp.{n}": shape for n, shape in mlp.shapes(cfg.width).items()}
        gain = () if cfg.design.hyper else (cfg.width,)
        for i, q in self.sublayers():
            out[f"l{i}.norm{q}"] = gain
            if cfg.design.hyper:
                out |= {f"l{i}.hc{q}.in": (s,), f"l{i}.hc{q}.out": (s,), f"l{i}.hc{q}.mix": (s, s)}
        return out | {"final.norm": gain, "head": (cfg.vocab, cfg.width)}

    def load(self, tensors: dict, dtype, device) -> "HybridWeights":
        for i, mixer in enumerate(self.mixers):
            if isinstance(mixer, CoreMixer):
                mixer.measure(lambda n, i=i: tensors[f"l{i}.mix.{n}"].shape)
        want = self.shapes()
        missing = sorted(set(want) - set(tensors))
        if missing:
            raise KeyError(f"the checkpoint lacks {missing}")
        for name, shape in want.items():
            if tuple(tensors[name].shape) != tuple(shape):
                raise ValueError(f"{name} has shape {tuple(tensors[name].shape)}, the configuration says {tuple(shape)}")
        cfg, width_p = self.cfg, self.width_p
        self.dtype = dtype

        def wide(name):
            return tensors[name].to(torch.float32)

        self.embed = padded(wide("embed"), cfg.vocab, width_p).to(device, dtype)
        self.head = padded(wide("head"), self.vocab_p, width_p).to(device, dtype)
        for unit in self.units:
            unit.load(lambda n, i=unit.layer: wide(f"l{i}.{n}"), width_p, dtype, device)
        # joints: what happens to the streams between two sublayers, as one fp32 vector [mix | out | in | gain] each, and the
        # norm weights where a norm has more than a single gain
        steps = list(self.sublayers())
        norms = [f"l{i}.norm{q}" for i, q in steps] + ["final.norm"]
        s = cfg.streams
        if not cfg.design.hyper:
            plain = torch.ones(4, device=device)
            self.joints = [plain] * len(norms)
            self.gains = [padded(wide(n), width_p).to(device).contiguous() for n in norms]
            return self
        none = [torch.zeros(s * s), torch.zeros(s)]
        after = [[wide(f"l{i}.hc{q}.mix").flatten(), wide(f"l{i}.hc{q}.out")] for i, q in steps]
        before = [[wide(f"l{i}.hc{q}.in"), wide(n).view(1)] for (i, q), n in zip(steps, norms)]
        before.append([torch.ones(s), wide("final.norm").view(1)])
        self.joints = [torch.cat([t.cpu() for t in a + b]).to(device) for a, b in zip([none] + after, before)]
        self.gains = [None] * len(norms)
        return self


def random_tensors(weights: HybridWeights, seed: int, device="cpu", std: float = 0.02) -> dict:
    """Random checkpoint of a stack's shapes: N(0, std) projections, unit norm weights, forget-gate floors in [0, 1),
    streams mixed by a matrix near the identity, decays that forget within tens to hundreds of tokens."""
    gen = torch.Generator(device=device).manual_seed(seed)
    out = {}
    for name, shape in weights.shapes().items():
        leaf = name.rsplit(".", 1)[-1]
        noise = torch.randn(shape, generator=gen, device=device) * std
        if leaf.startswith("norm"):
            noise = noise + 1.0
        elif leaf == "lower":
            noise = torch.rand(shape, generator=gen, device=device) * 0.9
        elif leaf == "mix":
            noise = noise + torch.eye(shape[0], device=device)
        elif leaf == "in" and len(shape) == 1:
            noise = noise + 1.0 / shape[0]
        elif leaf == "out":
            noise = noise + 1.0
        elif leaf == "dt_bias":
            noise = noise * 50.0 - 3.0
        out[name] = noise.to(torch.bfloat16)
    return out


@dataclass
class KeySpan:
    """Cached positions a packed batch's queries can see: packed row offsets and the first position per sequence, the row of
    every token of the batch itself, the most positions of a sequence that earlier passes wrote."""
    cu: torch.Tensor
    first: torch.Tensor
    rows: torch.Tensor
    keys: int
    max_keys: int
    max_old: int


class PackedBatch:
    """Portions of several sequences in one buffer, with what the kernels need to know about every row."""

    def __init__(self, slots, starts, portions, device):
        self.lengths, self.starts, self.device = [len(p) for p in portions], list(starts), device
        self.count, self.tokens, self.max_len = len(portions), sum(self.lengths), max(self.lengths)
        lens = np.asarray(self.lengths, dtype=np.int32)
        ends = np.cumsum(lens, dtype=np.int32)
        n, total = self.count, self.tokens
        host = np.empty(3 * total + 3 * n + 1, dtype=np.int32)
        host[:total] = np.fromiter((t for p in portions for t in p), dtype=np.int32, count=total)
        host[total: 2 * total] = np.arange(total) - np.repeat(ends - lens - np.asarray(starts, dtype=np.int32), lens)
        host[2 * total: 3 * total] = np.repeat(np.asarray(slots, dtype=np.int32), lens)
        tail = host[3 * total:]
        tail[:n], tail[n: 2 * n], tail[2 * n], tail[2 * n + 1:] = slots, starts, 0, ends
        self.ids, self.pos, self.slot_of, rest = torch.from_numpy(host).to(device).split([total, total, total, 3 * n + 1])
        self.slots, self.start, self.cu = rest.split([n, n, n + 1])
        self.kept: dict = {}              # gathered contexts: layers that share a latent and a window share the rows too
        self._spans: dict[int, KeySpan] = {}

    def context(self, window: int) -> KeySpan:
        span = self._spans.get(window)
        if span is None:
            first = [max(0, s - window + 1) for s in self.starts]
            counts = [s + n - f for s, n, f in zip(self.starts, self.lengths, first)]
            cu = np.concatenate(([0], np.cumsum(counts)))
            old = [s - f for s, f in zip(self.starts, first)]
            ends = np.cumsum(self.lengths)
            rows = np.arange(self.tokens) + np.repeat(cu[:-1] + old - (ends - self.lengths), self.lengths)
            host = torch.from_numpy(np.concatenate((cu, first, rows)).astype(np.int32)).to(self.device)
            cu, pos, rows = host.split([self.count + 1, self.count, self.tokens])
            span = self._spans[window] = KeySpan(cu, pos, rows, sum(counts), max(counts), max(old))
        return span


class HybridEngine(SlotEngine):
    """One replica of a hybrid stack: caches and states per slot, packed prefill (whole prompts or portions of them) and
    the batched decode step."""

    def __init__(self, weights: HybridWeights, batch: int, max_context: int, device, page_seed: int = 0,
                 on_demand_pages: bool = False, num_pages: int | None = None, prefill_chunk: int | None = None):
        """prefill_chunk: longest portion of one sequence that a prefill runs at once (None: whole prompts); longer prompts
        are run portion by portion against the caches, which bounds the memory of a pass."""
        super().__init__(batch, max_context, device, page_seed, on_demand_pages, num_pages)
        self.w, self.cfg, self.dtype = weights, weights.cfg, weights.dtype
        self.prefill_chunk = prefill_chunk
        self.sm_count = torch.cuda.get_device_properties(self.device).multi_processor_count
        # 32-bit means 32-bit: no TF32 products, no 16-bit partial sums
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        self._tables, self._workspaces, self._scratch, self._side = {}, {}, {}, None
        self.states: dict = {}               # caches and states of the units, by the unit's own keys (a mixer's: its layer)
        for unit in weights.units:
            self.states |= unit.allocate(self)
        self.streams = torch.zeros(batch, self.cfg.streams, weights.width_p, dtype=torch.float32, device=self.device)
        self.trace: list | None = None       # a list: the residual (sum of the streams) after every layer is appended

    # ------------------------------------------------------------------------------------------------ shared pieces
    def rotation_table(self, rotation) -> torch.Tensor:
        if rotation not in self._tables:
            # one row more than a slot can hold: the position of an idle slot may sit behind its last token
            self._tables[rotation] = rotation.table(self.max_context + 1, self.device)
        return self._tables[rotation]

    def shared_workspace(self, heads: int, rank: int, splits: int):
        key = (heads, rank, splits)
        if key not in self._workspaces:
            self._workspaces[key] = hops.latent_decode_workspace(self.batch, heads, rank, splits, self.device)
        return self._workspaces[key]

    def zero_scratch(self, used: int, pad: int):
        """[batch, used + pad] activations of a decode step whose last `pad` columns nobody writes: they stay zero."""
        if (used, pad) not in self._scratch:
            self._scratch[used, pad] = torch.zeros(self.batch, used + pad, dtype=self.dtype, device=self.device)
        return self._scratch[used, pad]

    def linear(self, x, weight):
        return F.linear(x, weight)

    def streams_weight(self, weight, swiglu: bool = False) -> bool:
        """Whether a decode-step projection by this weight runs on the package's weight-streaming kernel."""
        n = weight.shape[0] // 2 if swiglu else weight.shape[0]
        return (self.dtype == torch.bfloat16 and weight.shape[1] <= ops.SKINNY_GEMM_PAIR_MAX_K
                and ops.skinny_gemm_supports(self.batch, n, weight.shape[1], swiglu))

    def then(self, own_next: bool) -> int:
        """Overlap flags of a decode-step kernel whose successor is (not) one of this package's."""
        return ops.OVERLAP_START | ops.OVERLAP_TRIGGER if own_next else ops.OVERLAP_START

    def fork(self):
        """A second stream that has waited for the current one (`join` waits for it in turn)."""
        if self._side is None:
            self._side = torch.cuda.Stream(device=self.device)
        self._side.wait_stream(torch.cuda.current_stream(self.device))
        return self._side

    def join(self) -> None:
        torch.cuda.current_stream(self.device).wait_stream(self._side)

    def proj(self, x, weight, own_next: bool):
        """Decode-step projection: the weight-streaming kernel where it takes the shape, cuBLAS otherwise."""
        if self.streams_weight(weight):
            return ops.skinny_gemm(x, weight, overlap=self.then(own_next))
        return F.linear(x, weight)

    def fuses_head(self) -> bool:
        """Whether LM head and greedy choice run as one launch on the decode batch."""
        head = self.w.head
        return (self.dtype == torch.bfloat16 and self.w.vocab_p == self.cfg.vocab and head.shape[1] <= ops.SKINNY_GEMM_MAX_K
                and ops.skinny_gemm_supports(self.batch, head.shape[0], head.shape[1]))

    def logits(self, h, cap: bool = True) -> torch.Tensor:
        """fp32 logits [rows, padded vocab] of normed final rows; padding columns are -inf.  cap=False leaves a soft cap out: it
        does not change the order (a choice needs it not, and cannot be misled by values that saturate)."""
        head = self.w.head
        if self.dtype == torch.float32:
            out = F.linear(h, head)
        else:
            out = torch.mm(h, head.t(), out_dtype=torch.float32)
        if cap and self.cfg.softcap is not None:
            return hops.softcap(out, self.cfg.vocab, self.cfg.softcap)
        if self.w.vocab_p != self.cfg.vocab:
            out[:, self.cfg.vocab:] = float("-inf")
        return out

    def _joint(self, k: int, streams, y=None, ids=None, overlap: int = 0):
        return hops.hyper_connect(streams, self.w.joints[k], self.cfg.width, self.cfg.eps, self.dtype, y=y, ids=ids,
                                  table=self.w.embed if ids is not None else None, overlap=overlap, gains=self.w.gains[k])

    def _traced(self, streams) -> None:
        if self.trace is not None:
            self.trace.append(streams.sum(1)[:, : self.cfg.width].clone())

    # ------------------------------------------------------------------------------------------------------ prefill
    def _forward(self, batch: PackedBatch) -> torch.Tensor:
        """The stack over a packed batch: the final normed hidden rows."""
        streams = torch.empty(batch.tokens, self.cfg.streams, self.w.width_p, dtype=torch.float32, device=self.device)
        h = self._joint(0, streams, ids=batch.ids)
        units = self.w.units
        for k, unit in enumerate(units, start=1):
            h = self._joint(k, streams, y=unit.prefill(h, batch, self, self.states))
            if k == len(units) or units[k].layer != unit.layer:
                self._traced(streams)
        return h

    def _set_pos(self, slots, ends) -> None:
        at = torch.tensor([slots, ends], dtype=torch.int64, device=self.device)
        self.pos.index_copy_(0, at[0], at[1])

    @torch.no_grad()
    def extend(self, slots: list[int], starts: list[int], portions: list[list[int]], want=None) -> torch.Tensor:
        """Run the next tokens of some sequences from the caches and states that earlier calls left.  starts: tokens each
        slot already holds (0: the sequence begins here).  want: per sequence the places among its tokens whose logits are
        returned (default: the last), fp32 [wanted, vocab] in order.  With on-demand pages the pool is grown as needed."""
        assert len(slots) == len(starts) == len(portions) and len(set(slots)) == len(slots)
        assert all(0 <= s < self.batch for s in slots) and all(len(p) > 0 for p in portions)
        ends = [s + len(p) for s, p in zip(starts, portions)]
        assert max(ends) <= self.max_context, f"{max(ends)} tokens, room for {self.max_context}"
        if want is None:
            want = [[len(p) - 1] for p in portions]
        if self.pages is not None:
            for slot, end in zip(slots, ends):
                self.pages.ensure(slot, end)
        if self.active is not None and all(len(p) == 1 for p in portions) and all(s > 0 for s in starts):
            return self._extend_by_one(slots, starts, portions, want)
        batch = PackedBatch(slots, starts, portions, self.device)
        h = self._forward(batch)
        self._set_pos(slots, ends)
        rows, first = [], 0
        for p, w in zip(portions, want):
            rows += [first + i for i in w]
            first += len(p)
        if not rows:
            return torch.empty(0, self.cfg.vocab, device=self.device)
        return self.logits(h.index_select(0, torch.tensor(rows, device=self.device)))[:, : self.cfg.vocab]

    def _extend_by_one(self, slots, starts, portions, want) -> torch.Tensor:
        """One token for some slots through the decode step; the other slots are masked out."""
        others = self.active.clone()
        self.set_active([b in slots for b in range(self.batch)])
        at = torch.tensor([slots, starts, [p[0] for p in portions]], dtype=torch.int64, device=self.device)
        self.pos.index_copy_(0, at[0], at[1])
        tok = self.tok.index_copy(0, at[0], at[2])
        h = self._decode_hidden(tok, False)
        self._move_on()
        self.active.copy_(others)
        rows = [s for s, w in zip(slots, want) for _ in w]
        if not rows:
            return torch.empty(0, self.cfg.vocab, device=self.device)
        return self.logits(h.index_select(0, torch.tensor(rows, device=self.device)))[:, : self.cfg.vocab]

    def _prefill(self, prompts, slots):
        slots = list(range(self.batch)) if slots is None else slots
        assert all(0 < len(p) <= self.max_context for p in prompts)
        cut = self.prefill_chunk or max(len(p) for p in prompts)
        first = torch.zeros(len(prompts), dtype=torch.int64, device=self.device)
        for start in range(0, max(len(p) for p in prompts), cut):
            live = [i for i, p in enumerate(prompts) if len(p) > start]
            portions = [prompts[i][start: start + cut] for i in live]
            batch = PackedBatch([slots[i] for i in live], [start] * len(live), portions, self.device)
            h = self._forward(batch)
            done = [k for k, i in enumerate(live) if len(prompts[i]) <= start + cut]
            if done:
                rows = batch.cu[1:].long()[torch.tensor(done, device=self.device)] - 1
                ids = ops.argmax_rows(self.logits(h.index_select(0, rows), cap=False), self.argmax_ws)
                first[torch.tensor([live[k] for k in done], device=self.device)] = ids
        self._set_pos(slots, [len(p) for p in prompts])
        self.tok.index_copy_(0, torch.tensor(slots, dtype=torch.int64, device=self.device), first)
        return first.clone()

    # ------------------------------------------------------------------------------------------------------- decode
    def _decode_hidden(self, tok, own_head: bool) -> torch.Tensor:
        """The stack over one token per slot; idle slots ride along and touch nothing.  Every kernel of this package that
        follows another one starts early; what the next sublayer's first projection runs on decides a joint's flags."""
        units = self.w.units

        def first_own(k: int) -> bool:               # does a kernel of ours read the output of joint k?
            return own_head if k == len(units) else units[k].starts_own(self)

        streams, untraced = self.streams, self.trace is None
        h = self._joint(0, streams, ids=tok, overlap=self.then(first_own(0)))
        for k, unit in enumerate(units, start=1):
            h = self._joint(k, streams, y=unit.decode(h, self, self.states, True), overlap=self.then(first_own(k) and untraced))
            if k == len(units) or units[k].layer != unit.layer:          # the layer ends here
                self._traced(streams)
        return h

    def _move_on(self) -> None:
        self.pos.add_(1 if self.active is None else self.active)

    @torch.no_grad()
    def _decode(self, tok):
        own_head = self.fuses_head()
        h = self._decode_hidden(tok, own_head)
        if own_head:
            in_place = tok.data_ptr() == self.tok.data_ptr()
            nxt = ops.lm_head_argmax(h, self.w.head, self.argmax_ws, out=tok if in_place else None, overlap=ops.OVERLAP_START)
        else:
            nxt = ops.argmax_rows(self.logits(h, cap=False), self.argmax_ws)
        self._move_on()
        return nxt
