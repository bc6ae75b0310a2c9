"""Torch-facing wrappers of the kernels of hybrid stacks (include/b200_attn.h, last section): hyper-connected residual
streams, minGRU, HGRN2 and latent attention.  The element type of activations and weights (bf16 or fp32) is taken from
the tensors; shapes follow the padded layout the weight loader makes (`hybrid.py`)."""
from __future__ import annotations

import torch

from . import _lib
from .ops import PAGE_SIZE, _ptr, _require_cuda, _stream

LATENT_MAX_SPLITS = 64


def _f32(t) -> int:
    assert t.dtype in (torch.bfloat16, torch.float32)
    return int(t.dtype == torch.float32)


def hyper_connect(streams, weights, true_width: int, eps: float, dtype, y=None, ids=None, table=None, overlap: int = 0, gains=None):
    """One step between two sublayers (b200_hyper_connect): mixes `y` into `streams` [rows, S, width] (in place), or sets
    them from `table[ids]`; returns the next sublayer's normed input [rows, width].  gains: fp32 [width] norm weights on top
    of the single gain."""
    assert streams.dtype == weights.dtype == torch.float32 and streams.is_contiguous() and weights.is_contiguous()
    rows, s, width = streams.shape
    assert weights.numel() == s * s + 2 * s + 1
    assert gains is None or (gains.dtype == torch.float32 and gains.numel() == width and gains.is_contiguous())
    h = torch.empty((rows, width), dtype=dtype, device=streams.device)
    parts = 1
    if y is not None:                       # [rows, width], or [parts, rows, width] to be summed
        parts = y.shape[0] if y.ndim == 3 else 1
        assert y.shape[-2:] == (rows, width) and y.is_contiguous() and y.dtype == dtype
    if ids is not None:
        assert ids.numel() == rows and ids.is_contiguous() and ids.dtype in (torch.int32, torch.int64)
        assert table.dtype == dtype and table.shape[1] == width and table.is_contiguous()
    _require_cuda(streams, weights)
    _lib.call("b200_hyper_connect", _ptr(ids), int(ids is not None and ids.dtype == torch.int64), _ptr(table), _ptr(streams),
              _ptr(y), parts, _ptr(weights), _ptr(gains), _ptr(h), rows, s, width, true_width, float(eps), _f32(h), int(overlap),
              _stream())
    return h


def swiglu_f32(gate_up, intermediate: int):
    assert gate_up.dtype == torch.float32 and gate_up.stride(1) == 1 and gate_up.shape[1] >= 2 * intermediate
    _require_cuda(gate_up)
    out = torch.empty((gate_up.shape[0], intermediate), dtype=torch.float32, device=gate_up.device)
    _lib.call("b200_swiglu_f32", _ptr(gate_up), gate_up.stride(0), _ptr(out), gate_up.shape[0], intermediate, _stream())
    return out


# ------------------------------------------------------------------------------------------------------------- minGRU
MINGRU_BLOCK, MINGRU_COLS = 64, 64


def sm_count(device) -> int:
    key = torch.device(device).index or 0
    if key not in _sm_counts:
        _sm_counts[key] = torch.cuda.get_device_properties(device).multi_processor_count
    return _sm_counts[key]


_sm_counts: dict = {}


def mingru_segments(max_len: int, groups: int, sm_count: int) -> tuple[int, int]:
    """(segment length, segments of the longest sequence).  `groups` CTAs walk whole sequences in blocks of 64 tokens; when
    they do not fill the device (three per SM), sequences are cut into runs of whole blocks, at the price of a second pass."""
    blocks = -(-max_len // MINGRU_BLOCK)
    parts = min(-(-3 * sm_count // groups), blocks, 64)
    if parts < 2:
        return max_len, 1
    per = -(-blocks // parts)
    return per * MINGRU_BLOCK, -(-blocks // per)


def mingru_prefill(zxg, bias, state, batch, segments=None):
    """zxg [tokens, 3*width] projections of a packed batch (`batch`: PackedBatch); state [slots, width] fp32, in place.
    segments: (length, count) to pin how sequences are cut."""
    width = state.shape[1]
    assert zxg.shape[1] == 3 * width and zxg.stride(1) == 1 and bias.numel() == 2 * width
    assert state.dtype == bias.dtype == torch.float32 and state.is_contiguous() and bias.is_contiguous()
    _require_cuda(zxg, bias, state)
    n = batch.count
    segment, count = segments or mingru_segments(batch.max_len, n * -(-width // MINGRU_COLS), sm_count(zxg.device))
    ws = None
    if count > 1:
        ws = torch.empty(_lib.load().b200_mingru_workspace_bytes(n, count, width), dtype=torch.uint8, device=zxg.device)
    out = torch.empty((zxg.shape[0], width), dtype=zxg.dtype, device=zxg.device)
    _lib.call("b200_mingru_prefill", _ptr(zxg), zxg.stride(0), _ptr(bias), _ptr(state), _ptr(batch.cu), _ptr(batch.slots),
              _ptr(batch.start), _ptr(ws), _ptr(out), n, segment, count, width, _f32(zxg), _stream())
    return out


def mingru_decode(zxg, bias, state, pos, active, overlap: int = 0):
    rows, width = state.shape
    assert zxg.shape == (rows, 3 * width) and zxg.stride(1) == 1 and pos.dtype == torch.int64
    _require_cuda(zxg, bias, state, pos)
    out = torch.empty((rows, width), dtype=zxg.dtype, device=zxg.device)
    _lib.call("b200_mingru_decode", _ptr(zxg), zxg.stride(0), _ptr(bias), _ptr(state), _ptr(pos), _ptr(active), _ptr(out), rows,
              width, _f32(zxg), int(overlap), _stream())
    return out


# -------------------------------------------------------------------------------------------------------------- HGRN2
def _check_hgrn2(qfv, lower, bias, norm, state):
    _, heads, dim, vdim = state.shape
    assert qfv.shape[1] == 2 * heads * dim + heads * vdim and qfv.stride(1) == 1
    assert lower.numel() == bias.numel() == heads * dim and norm.numel() == vdim
    for t in (lower, bias, norm, state):
        assert t.dtype == torch.float32 and t.is_contiguous()
    _require_cuda(qfv, lower, bias, norm, state)
    return heads, dim, vdim


def hgrn2_segments(max_len: int, groups: int, sm_count: int) -> tuple[int, int]:
    """(segment length, segments of the longest sequence).  `groups` CTAs work on whole sequences; when they leave half of
    the slots (two per SM) empty, sequences are cut into segments of at least 128 tokens that run side by side, at the
    price of a second pass over the rows."""
    parts = min(2 * sm_count // groups, max_len // 128)
    if parts < 3:
        return max_len, 1
    segment = -(-max_len // parts // 16) * 16 + (0 if max_len % parts == 0 and (max_len // parts) % 16 == 0 else 16)
    return segment, -(-max_len // segment)


def hgrn2_prefill(qfv, lower, bias, norm, state, batch, true_vdim: int, eps: float, serial: bool = False, segments=None):
    """qfv [tokens, 2*heads*dim + heads*vdim]; state [slots, heads, dim, vdim] fp32, in place.  segments: (length, count) to
    pin how sequences are cut."""
    heads, dim, vdim = _check_hgrn2(qfv, lower, bias, norm, state)
    tokens = qfv.shape[0]
    chunked = qfv.dtype == torch.bfloat16 and dim <= 128 and not serial
    segment, count = (batch.max_len, 1) if not chunked else segments or hgrn2_segments(
        batch.max_len, batch.count * heads * -(-vdim // 128), sm_count(qfv.device))
    ws = None
    if count > 1:
        nbytes = _lib.load().b200_hgrn2_workspace_bytes(batch.count, count, heads, dim, vdim)
        ws = torch.empty(nbytes // 4, dtype=torch.float32, device=qfv.device)
    scratch = None if chunked and vdim <= 128 else torch.empty((tokens, heads * vdim), dtype=torch.float32, device=qfv.device)
    out = torch.empty((tokens, heads * vdim), dtype=qfv.dtype, device=qfv.device)
    _lib.call("b200_hgrn2_prefill", _ptr(qfv), qfv.stride(0), _ptr(lower), _ptr(bias), _ptr(norm), _ptr(state), _ptr(batch.cu),
              _ptr(batch.slots), _ptr(batch.start), _ptr(scratch), _ptr(out), batch.count, tokens, heads, dim, vdim, true_vdim,
              float(eps), _f32(qfv), int(serial), segment, count, _ptr(ws), _stream())
    return out


def hgrn2_decode(qfv, lower, bias, norm, state, pos, active, true_vdim: int, eps: float, overlap: int = 0):
    heads, dim, vdim = _check_hgrn2(qfv, lower, bias, norm, state)
    rows = state.shape[0]
    assert qfv.shape[0] == rows
    out = torch.empty((rows, heads * vdim), dtype=qfv.dtype, device=qfv.device)
    _lib.call("b200_hgrn2_decode", _ptr(qfv), qfv.stride(0), _ptr(lower), _ptr(bias), _ptr(norm), _ptr(state), _ptr(pos),
              _ptr(active), _ptr(out), rows, heads, dim, vdim, true_vdim, float(eps), _f32(qfv), int(overlap), _stream())
    return out


# --------------------------------------------------------------------------------------------------- latent attention
def allocate_latent_cache(num_pages: int, row: int, dtype, *, device="cuda"):
    """Zero-filled pages of [latent | rotated key part] rows (the padding columns stay zero)."""
    return torch.zeros((num_pages, PAGE_SIZE, row), dtype=dtype, device=device)


def latent_prep(fused, q_weight, kv_weight, pos, slot, active, block_table, angles, cache, true_q_rank: int, rank: int,
                true_rank: int, eps: float, overlap: int = 0):
    """Query-latent norm, and (cache given) latent norm + key rotation + paged write.  Returns cq [rows, q_rank]."""
    q_rank, rows = q_weight.numel(), fused.shape[0]
    rot = 0
    if cache is not None:
        rot = cache.shape[2] - rank
        assert fused.shape[1] == q_rank + rank + rot and kv_weight.numel() == rank and cache.dtype == fused.dtype
    assert fused.stride(1) == 1 and angles.dtype == torch.float32 and angles.is_contiguous()
    assert pos.dtype in (torch.int32, torch.int64)
    _require_cuda(fused, q_weight, pos, block_table, angles)
    cq = torch.empty((rows, q_rank), dtype=fused.dtype, device=fused.device)
    _lib.call("b200_latent_prep", _ptr(fused), fused.stride(0), _ptr(q_weight), _ptr(kv_weight), _ptr(pos),
              int(pos.dtype == torch.int64), _ptr(slot), _ptr(active), _ptr(block_table), block_table.stride(0), _ptr(angles),
              _ptr(cache), _ptr(cq), rows, q_rank, true_q_rank, rank, true_rank, rot,
              angles.shape[1] if cache is not None else 0, float(eps), _f32(fused), int(overlap), _stream())
    return cq


def rope_interleaved(x, offset: int, pos, angles) -> None:
    """Rotates pairs (offset + 2i, offset + 2i + 1) of x [rows, heads, D] in place; pos int32 [rows]."""
    assert x.ndim == 3 and x.is_contiguous() and pos.dtype == torch.int32 and angles.is_contiguous()
    _require_cuda(x, pos, angles)
    _lib.call("b200_rope_interleaved", _ptr(x), x.stride(0), x.stride(1), offset, x.shape[1], angles.shape[1], _ptr(pos),
              _ptr(angles), x.shape[0], _f32(x), _stream())


def latent_gather(cache, block_table, slots, cu_k, k_pos0, keys: int, max_keys: int):
    """Cache rows of a run of positions per sequence, packed: [keys, row]."""
    out = torch.empty((keys, cache.shape[2]), dtype=cache.dtype, device=cache.device)
    _require_cuda(cache, block_table, slots, cu_k, k_pos0)
    _lib.call("b200_latent_gather", _ptr(cache), _ptr(out), _ptr(block_table), block_table.stride(0), _ptr(slots), _ptr(cu_k),
              _ptr(k_pos0), slots.numel(), max_keys, 1, cache.shape[2] * cache.element_size(), _stream())
    return out


def latent_prefill(q, kv, ctx, cu_q, cu_k, q_pos0, k_pos0, max_q: int, true_dim: int, true_rot: int, vdim: int, rank: int,
                   window: int, scale: float, simple: bool = False):
    """Windowed causal attention of packed queries q [tokens, heads, dim + rot] over expanded keys and values
    kv [keys, heads*dim | heads*vdim] and the shared rotated parts in ctx [keys, rank + rot] -> [tokens, heads*vdim].
    bf16 heads of up to 256 + 256 dimensions run on the tensor-core kernel; simple=True keeps them off it."""
    tokens, heads, width = q.shape
    rot = ctx.shape[1] - rank
    dim = width - rot
    assert kv.shape == (ctx.shape[0], heads * (dim + vdim)) and q.is_contiguous() and kv.is_contiguous() and ctx.is_contiguous()
    _require_cuda(q, kv, ctx)
    out = torch.empty((tokens, heads * vdim), dtype=q.dtype, device=q.device)
    if q.dtype == torch.bfloat16 and width <= 256 and vdim <= 256 and not simple:
        _lib.call("b200_latent_prefill", _ptr(q), _ptr(kv), _ptr(ctx), _ptr(out), _ptr(cu_q), _ptr(cu_k), _ptr(q_pos0),
                  _ptr(k_pos0), cu_q.numel() - 1, max_q, tokens, ctx.shape[0], heads, dim, true_dim, rot, true_rot, vdim, rank,
                  min(window, 1 << 30), float(scale), _stream())
        return out
    _lib.call("b200_latent_prefill_simple", _ptr(q), _ptr(kv), _ptr(ctx), _ptr(out), _ptr(cu_q), _ptr(cu_k), _ptr(q_pos0),
              _ptr(k_pos0), cu_q.numel() - 1, max_q, heads, dim, rot, vdim, rank, min(window, 1 << 30), float(scale), _f32(q),
              _stream())
    return out


def latent_absorb(q, w_uk, pos, angles, overlap: int = 0):
    """q [B, heads, dim + rot], w_uk [heads, dim, rank] -> [B, heads, rank + rot] with the rotated part rotated."""
    batch, heads, width = q.shape
    _, dim, rank = w_uk.shape
    rot = width - dim
    assert q.is_contiguous() and w_uk.is_contiguous() and w_uk.shape[0] == heads and pos.dtype == torch.int64
    _require_cuda(q, w_uk, pos, angles)
    out = torch.empty((batch, heads, rank + rot), dtype=q.dtype, device=q.device)
    _lib.call("b200_latent_absorb", _ptr(q), _ptr(w_uk), _ptr(pos), _ptr(angles), _ptr(out), batch, heads, dim, rot,
              angles.shape[1], rank, _f32(q), int(overlap), _stream())
    return out


def latent_decode_workspace(batch: int, heads: int, rank: int, splits: int, device) -> tuple[torch.Tensor, torch.Tensor]:
    return (torch.empty((batch, heads, splits, 2), dtype=torch.float32, device=device),
            torch.empty((batch, heads, splits, rank), dtype=torch.float32, device=device))


LATENT_DECODE_MAX_ROW = 1344     # widest cache row two stages of the tensor-core kernel's ring hold


def latent_decode_splits(batch: int, heads: int, span: int, sm_count: int) -> int:
    """Key ranges per slot: the count whose launch ends first with two CTAs per SM, at ~100 tokens of fixed cost per CTA and
    a merge that grows with the number of ranges."""
    groups = batch * -(-heads // 16)
    most = max(1, min(LATENT_MAX_SPLITS, span // (2 * PAGE_SIZE)))
    return min(range(1, most + 1), key=lambda s: (-(-groups * s // (2 * sm_count)) * (span / s + 100) + 4 * s, s))


def latent_decode(q, cache, block_table, pos, active, workspace, window: int, scale: float, overlap: int = 0,
                  simple: bool = False) -> None:
    """Decode attention of q [B, heads, rank + rot] over the paged rows; leaves the split results in `workspace`.
    bf16 rows run on the tensor-core kernel where they fit; simple=True keeps them off it."""
    ml, o = workspace
    batch, heads, splits, rank = o.shape
    assert q.shape == (batch, heads, cache.shape[2]) and q.is_contiguous() and pos.dtype == torch.int64
    _require_cuda(q, cache, block_table, pos, ml, o)
    if q.dtype == torch.bfloat16 and rank <= 1024 and cache.shape[2] <= LATENT_DECODE_MAX_ROW and not simple:
        _lib.call("b200_latent_decode", _ptr(q), _ptr(cache), cache.shape[0], _ptr(block_table), block_table.stride(0),
                  _ptr(pos), _ptr(active), _ptr(ml), _ptr(o), batch, heads, rank, cache.shape[2] - rank, min(window, 1 << 30),
                  splits, float(scale), int(overlap), _stream())
        return
    _lib.call("b200_latent_decode_simple", _ptr(q), _ptr(cache), _ptr(block_table), block_table.stride(0), _ptr(pos),
              _ptr(active), _ptr(ml), _ptr(o), batch, heads, rank, cache.shape[2] - rank, min(window, 1 << 30), splits,
              float(scale), _f32(q), int(overlap), _stream())


def latent_value(workspace, w_uv, dtype, overlap: int = 0):
    """Merges the splits and applies w_uv [heads, vdim, rank] -> [B, heads*vdim]."""
    ml, o = workspace
    batch, heads, splits, rank = o.shape
    vdim = w_uv.shape[1]
    assert w_uv.shape == (heads, vdim, rank) and w_uv.is_contiguous() and w_uv.dtype == dtype
    out = torch.empty((batch, heads * vdim), dtype=dtype, device=o.device)
    merged = torch.empty((batch, heads, rank), dtype=dtype, device=o.device)
    _lib.call("b200_latent_value", _ptr(ml), _ptr(o), _ptr(w_uv), _ptr(merged), _ptr(out), batch, heads, rank, vdim, splits, _f32(w_uv),
              int(overlap), _stream())
    return out


# ------------------------------------------------------------------------------------- gated activations and soft cap
ACT_SILU, ACT_GELU_TANH = 0, 1


def _rows(t) -> bool:
    """A matrix whose rows may be further apart than they are long."""
    return t.ndim == 2 and t.stride(1) == 1


def gated_act(gate_up, width: int, out, act: int, overlap: int = 0):
    """out = act(gate_up[:, :width]) * gate_up[:, width: 2*width]; both may be column ranges of wider matrices."""
    assert _rows(gate_up) and gate_up.shape[1] >= 2 * width and _rows(out) and out.shape == (gate_up.shape[0], width)
    assert out.dtype == gate_up.dtype
    _require_cuda(gate_up, out)
    _lib.call("b200_gated_act", _ptr(gate_up), gate_up.stride(0), width, _ptr(out), out.stride(0), out.shape[0], width, act,
              _f32(gate_up), int(overlap), _stream())
    return out


def softcap(logits, vocab: int, cap: float):
    """logits <- cap * tanh(logits / cap) in place; columns from `vocab` on become -inf."""
    assert logits.dtype == torch.float32 and _rows(logits)
    _require_cuda(logits)
    _lib.call("b200_softcap", _ptr(logits), logits.stride(0), logits.shape[0], vocab, logits.shape[1], float(cap), _stream())
    return logits


# ------------------------------------------------------------------------------------------------- windowed attention
def allocate_window_cache(num_pages: int, kv_heads: int, pitch: int, dtype, *, device="cuda"):
    """Zero-filled pages of [key | value] rows, one per key/value head and token."""
    return torch.zeros((num_pages, kv_heads, PAGE_SIZE, pitch), dtype=dtype, device=device)


def window_prep(x, bias, pos, slot, active, block_table, angles, cache, heads: int, dim: int, vdim: int, ctx=None, ctx_row=None,
                overlap: int = 0) -> None:
    """Biases and rotation on the rows x = [q | k | v | ...] of projections: q in place, [k | v] to the pages and to `ctx`."""
    _, kv_heads, _, pitch = cache.shape
    assert _rows(x) and x.shape[1] >= (heads + kv_heads) * dim + kv_heads * vdim and x.dtype == cache.dtype
    assert bias.dtype == torch.float32 and bias.numel() == (heads + kv_heads) * dim + kv_heads * vdim
    assert angles.dtype == torch.float32 and angles.is_contiguous() and cache.is_contiguous() and pos.dtype in (torch.int32, torch.int64)
    if ctx is not None:
        assert ctx.shape[1:] == (kv_heads, pitch) and ctx.dtype == x.dtype and ctx.is_contiguous() and ctx_row.dtype == torch.int32
    _require_cuda(x, bias, pos, block_table, angles, cache)
    _lib.call("b200_window_prep", _ptr(x), x.stride(0), _ptr(bias), _ptr(pos), int(pos.dtype == torch.int64), _ptr(slot),
              _ptr(active), _ptr(block_table), block_table.stride(0), _ptr(angles), _ptr(cache), _ptr(ctx), _ptr(ctx_row), x.shape[0],
              heads, kv_heads, dim, angles.shape[1], vdim, pitch, _f32(x), int(overlap), _stream())


def window_gather(cache, ctx, block_table, slots, cu_k, k_pos0, max_keys: int) -> None:
    """The first max_keys keys (rounded up to 16) of every sequence, from the pages to ctx [keys, kv_heads, pitch]."""
    _, kv_heads, _, pitch = cache.shape
    _require_cuda(cache, ctx, block_table, slots, cu_k, k_pos0)
    _lib.call("b200_latent_gather", _ptr(cache), _ptr(ctx), _ptr(block_table), block_table.stride(0), _ptr(slots), _ptr(cu_k),
              _ptr(k_pos0), slots.numel(), max_keys, kv_heads, pitch * cache.element_size(), _stream())


def window_prefill(q, ctx, gate, out, cu_q, cu_k, q_pos0, k_pos0, max_q: int, heads: int, dim: int, true_dim: int, vdim: int,
                   window: int, scale: float, out_scale: float = 1.0, simple: bool = False):
    """Windowed causal attention of the packed queries in the first heads*dim columns of q over ctx [keys, kv_heads, pitch];
    out [tokens, heads*vdim] = o * sigmoid(gate) * out_scale.  bf16 heads of up to 256 + 256 dimensions run on the
    tensor-core kernel; simple=True keeps them off it."""
    keys, kv_heads, pitch = ctx.shape
    assert _rows(q) and _rows(gate) and _rows(out) and out.shape == gate.shape == (q.shape[0], heads * vdim) and ctx.is_contiguous()
    assert q.dtype == ctx.dtype == gate.dtype == out.dtype and q.shape[1] >= heads * dim
    _require_cuda(q, ctx, gate, out)
    simple = simple or dim > 256 or vdim > 256
    _lib.call("b200_window_prefill", _ptr(q), q.stride(0), _ptr(ctx), _ptr(gate), gate.stride(0), _ptr(out), out.stride(0),
              _ptr(cu_q), _ptr(cu_k), _ptr(q_pos0), _ptr(k_pos0), cu_q.numel() - 1, max_q, q.shape[0], keys, heads, kv_heads, dim,
              true_dim, vdim, pitch, min(window, 1 << 30), float(scale), float(out_scale), int(simple), _f32(q), _stream())
    return out


def window_decode_splits(batch: int, heads: int, kv_heads: int, span: int, sm_count: int) -> int:
    """Key ranges per slot (as for latent attention: a CTA takes up to 16 query heads of one key/value head)."""
    return latent_decode_splits(batch * kv_heads, heads // kv_heads, span, sm_count)


def window_decode(q, cache, block_table, pos, active, workspace, dim: int, window: int, scale: float, overlap: int = 0,
                  simple: bool = False) -> None:
    """One token per slot: the heads in the first heads*dim columns of q (rotated) over the pages; leaves the split results in
    `workspace`."""
    ml, o = workspace
    batch, heads, splits, vdim = o.shape
    _, kv_heads, _, pitch = cache.shape
    assert _rows(q) and q.shape[0] == batch and q.shape[1] >= heads * dim and pos.dtype == torch.int64 and q.dtype == cache.dtype
    _require_cuda(q, cache, block_table, pos, ml, o)
    simple = simple or vdim > 1024 or pitch > LATENT_DECODE_MAX_ROW
    _lib.call("b200_window_decode", _ptr(q), q.stride(0), _ptr(cache), cache.shape[0], _ptr(block_table), block_table.stride(0),
              _ptr(pos), _ptr(active), _ptr(ml), _ptr(o), batch, heads, kv_heads, dim, vdim, pitch, min(window, 1 << 30), splits,
              float(scale), int(simple), _f32(q), int(overlap), _stream())


def window_merge(workspace, gate, out, out_scale: float = 1.0, overlap: int = 0):
    """Merges the splits: out [B, heads*vdim] = o * sigmoid(gate) * out_scale."""
    ml, o = workspace
    batch, heads, splits, vdim = o.shape
    assert _rows(gate) and _rows(out) and out.shape == gate.shape == (batch, heads * vdim) and out.dtype == gate.dtype
    _require_cuda(ml, o, gate, out)
    _lib.call("b200_window_merge", _ptr(ml), _ptr(o), _ptr(gate), gate.stride(0), _ptr(out), out.stride(0), batch, heads, vdim,
              splits, float(out_scale), _f32(out), int(overlap), _stream())
    return out


# --------------------------------------------------------------------------------------------------------- state space
def conv_taps(taps: int) -> int:
    """Taps of the kernels' convolution that hold `taps` of a model's."""
    assert 1 <= taps <= 16, f"convolutions of 1 to 16 taps (got {taps})"
    return 4 if taps <= 4 else 8 if taps <= 8 else 16


def conv_prefill(x, weight, bias, ring, batch):
    """Causal convolution with silu over a packed batch; x [tokens, channels] (a column range), weight fp32 [taps, channels] with
    the current token's row first, ring fp32 [slots, taps, channels] in place."""
    slots, taps, channels = ring.shape
    assert _rows(x) and x.shape[1] == channels and weight.shape == (taps, channels) and bias.numel() == channels
    for t in (weight, bias, ring):
        assert t.dtype == torch.float32 and t.is_contiguous()
    _require_cuda(x, weight, bias, ring)
    out = torch.empty((x.shape[0], channels), dtype=x.dtype, device=x.device)
    _lib.call("b200_conv_prefill", _ptr(x), x.stride(0), _ptr(weight), _ptr(bias), _ptr(ring), _ptr(batch.cu), _ptr(batch.slots),
              _ptr(batch.start), _ptr(out), out.stride(0), batch.count, batch.max_len, channels, taps, _f32(x), _stream())
    return out


def ssd_segments(max_len: int, groups: int, sm_count: int) -> tuple[int, int]:
    """(segment length, segments of the longest sequence) of the chunked state-space prefill, as `hgrn2_segments`."""
    parts = min(2 * sm_count // groups, max_len // 128)
    if parts < 3:
        return max_len, 1
    segment = -(-max_len // (parts * 32)) * 32
    return segment, -(-max_len // segment)


def ssd_prefill(xbc, dt, dt_bias, a_log, skip, state, groups: int, batch, serial: bool = False, segments=None):
    """State-space recurrence of a packed batch: xbc [tokens, x | B | C] after the convolution, dt [tokens, heads] (a column
    range), state fp32 [slots, heads, dim, vdim] in place -> y [tokens, heads*vdim] (bf16 from the chunked kernel, else
    fp32).  segments: (length, count) to pin how sequences are cut."""
    _, heads, dim, vdim = state.shape
    assert _rows(xbc) and xbc.shape[1] == heads * vdim + 2 * groups * dim and _rows(dt) and dt.shape[1] >= heads and dt.dtype == xbc.dtype
    for t in (dt_bias, a_log, skip, state):
        assert t.dtype == torch.float32 and t.is_contiguous()
    _require_cuda(xbc, dt, dt_bias, a_log, skip, state)
    tokens = xbc.shape[0]
    chunked = xbc.dtype == torch.bfloat16 and not serial and bool(_lib.load().b200_ssd_chunked(dim, vdim))
    segment, count = (batch.max_len, 1) if not chunked else segments or ssd_segments(
        batch.max_len, batch.count * max(1, heads * vdim // 128), sm_count(xbc.device))
    ws = None
    if count > 1:
        ws = torch.empty(_lib.load().b200_hgrn2_workspace_bytes(batch.count, count, heads, dim, vdim) // 4, dtype=torch.float32,
                         device=xbc.device)
    y = torch.empty((tokens, heads * vdim), dtype=torch.bfloat16 if chunked else torch.float32, device=xbc.device)
    _lib.call("b200_ssd_prefill", _ptr(xbc), xbc.stride(0), _ptr(dt), dt.stride(0), _ptr(dt_bias), _ptr(a_log), _ptr(skip), _ptr(state),
              _ptr(batch.cu), _ptr(batch.slots), _ptr(batch.start), _ptr(y), batch.count, heads, groups, dim, vdim, _f32(xbc),
              int(not chunked), segment, count, _ptr(ws), _stream())
    return y


def ssd_decode(xbc, dt, dt_bias, a_log, skip, weight, bias, ring, state, groups: int, pos, active, overlap: int = 0):
    """One token per slot: convolution (ring) and recurrence (state) -> y fp32 [B, heads*vdim]; xbc rows are raw projections."""
    rows, heads, dim, vdim = state.shape
    assert _rows(xbc) and xbc.shape == (rows, heads * vdim + 2 * groups * dim) and _rows(dt) and pos.dtype == torch.int64
    assert ring.shape[::2] == xbc.shape and weight.shape == ring.shape[1:]
    _require_cuda(xbc, dt, state, ring, pos)
    y = torch.empty((rows, heads * vdim), dtype=torch.float32, device=xbc.device)
    _lib.call("b200_ssd_decode", _ptr(xbc), xbc.stride(0), _ptr(dt), dt.stride(0), _ptr(dt_bias), _ptr(a_log), _ptr(skip), _ptr(weight),
              _ptr(bias), _ptr(ring), ring.shape[1], _ptr(state), _ptr(pos), _ptr(active), _ptr(y), rows, heads, groups, dim, vdim,
              _f32(xbc), int(overlap), _stream())
    return y


def gated_group_norm(y, z, weight, out, heads: int, true_vdim: int, groups: int, eps: float, overlap: int = 0):
    """out = f / rms(f) * weight with f = y * silu(z), the root mean square over each of `groups` equal parts of the channels;
    heads of weight.numel() / heads columns, the first true_vdim of each in use."""
    assert _rows(y) and _rows(z) and _rows(out) and y.shape == z.shape == out.shape and weight.numel() == y.shape[1]
    assert z.dtype == out.dtype and weight.dtype == torch.float32
    _require_cuda(y, z, weight, out)
    _lib.call("b200_gated_group_norm", _ptr(y), y.stride(0), _ptr(z), z.stride(0), _ptr(weight), _ptr(out), out.stride(0), y.shape[0],
              heads, y.shape[1] // heads, true_vdim, groups, float(eps), _f32(y), _f32(z), int(overlap), _stream())
    return out


# ----------------------------------------------------------------------------------------------- gated linear attention
def _check_gla(qkv, gate, out, norm, bias, state):
    _, heads, dim, vdim = state.shape
    assert _rows(qkv) and qkv.shape[1] >= heads * (2 * dim + vdim) and norm.numel() == vdim and bias.numel() == heads * dim
    assert _rows(gate) and _rows(out) and gate.shape == out.shape == (qkv.shape[0], heads * vdim)
    for t in (norm, bias, state):
        assert t.dtype == torch.float32 and t.is_contiguous()
    _require_cuda(qkv, gate, out, norm, bias, state)
    return heads, dim, vdim


def gla_prefill(qkv, z, bias, norm, gate, state, out, batch, true_vdim: int, q_scale: float, tau: float, eps: float,
                serial: bool = False, segments=None):
    """Gated linear attention of a packed batch: qkv rows [q | k | v | ...], z fp32 [tokens, heads*dim]; state in place."""
    heads, dim, vdim = _check_gla(qkv, gate, out, norm, bias, state)
    tokens = qkv.shape[0]
    assert z.dtype == torch.float32 and _rows(z) and z.shape == (tokens, heads * dim)
    chunked = qkv.dtype == torch.bfloat16 and dim <= 128 and not serial
    segment, count = (batch.max_len, 1) if not chunked else segments or hgrn2_segments(
        batch.max_len, batch.count * heads * -(-vdim // 128), sm_count(qkv.device))
    ws = None
    if count > 1:
        ws = torch.empty(_lib.load().b200_hgrn2_workspace_bytes(batch.count, count, heads, dim, vdim) // 4, dtype=torch.float32,
                         device=qkv.device)
    scratch = None if chunked and vdim <= 128 else torch.empty((tokens, heads * vdim), dtype=torch.float32, device=qkv.device)
    _lib.call("b200_gla_prefill", _ptr(qkv), qkv.stride(0), _ptr(z), z.stride(0), _ptr(bias), _ptr(norm), _ptr(gate), gate.stride(0),
              _ptr(state), _ptr(batch.cu), _ptr(batch.slots), _ptr(batch.start), _ptr(scratch), _ptr(out), out.stride(0), batch.count,
              tokens, heads, dim, vdim, true_vdim, float(q_scale), 1.0 / float(tau), float(eps), _f32(qkv), int(serial), segment, count,
              _ptr(ws), _stream())
    return out


def gla_decode(qkv, low, w_low, bias, norm, gate, state, out, pos, active, true_vdim: int, q_scale: float, tau: float, eps: float,
               overlap: int = 0):
    """One token per slot; low [B, rank] (columns of the same matrix as qkv), w_low [heads*dim, rank]."""
    heads, dim, vdim = _check_gla(qkv, gate, out, norm, bias, state)
    assert low.stride(0) == qkv.stride(0) and w_low.shape == (heads * dim, low.shape[1]) and w_low.is_contiguous()
    _lib.call("b200_gla_decode", _ptr(qkv), qkv.stride(0), _ptr(low), _ptr(w_low), low.shape[1], _ptr(bias), _ptr(norm), _ptr(gate),
              gate.stride(0), _ptr(state), _ptr(pos), _ptr(active), _ptr(out), out.stride(0), qkv.shape[0], heads, dim, vdim, true_vdim,
              float(q_scale), 1.0 / float(tau), float(eps), _f32(qkv), int(overlap), _stream())
    return out
