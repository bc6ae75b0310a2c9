"""Small hybrid-stack configurations and random checkpoints for the tests (weights scaled so that every mechanism moves the
logits: projections N(0, 1/fan-in), biases and norm weights away from 0 and 1, streams mixed by a full matrix)."""
from __future__ import annotations

import torch
from torch.utils._python_dispatch import TorchDispatchMode

from oracle import hybrid_reference as R


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, window, scale=None, base=1000.0, scaling=None, kv_from=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = scaling
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
             "mask": {"size": window}, "rot": rot, "scale": scale or (dim + rot_dim) ** -0.5}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer}


def hgrn2(heads, dim, vdim):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def mingru(width):
    return {"type": "mingru", "mixer": {"width": width}}


def stack(width, vocab, streams, layers, eps=1e-5):
    return {"architecture": "Tofilorn", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "layers": [{**layer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for layer, ff in layers]}


def window(heads, kv_heads, dim, vdim, size, dims=None, base=1000.0, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
            "rot": {"base": base, "dims": dim if dims is None else dims}, "scale": scale or dim ** -0.5}


def state_space(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def parallel(left, right, left_scale=1.0, right_scale=1.0):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def gla(heads, dim, vdim, tau):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def dugilorn(width, vocab, cap, layers, eps=1e-5):
    return {"architecture": "Dugilorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap,
            "layers": [{**layer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for layer, ff in layers]}


YARN = {"factor": 8.0, "original": 64, "fast": 16.0, "slow": 0.5}

CONFIGS = {
    # every size odd in its own way, a shared latent with another window and other heads, three streams
    "ragged": stack(136, 331, 3, [
        (hgrn2(3, 24, 40), 200),
        (latent(5, 40, 24, 56, 72, 88, 37, scaling=YARN), None),
        (mingru(100), None),
        (latent(3, 24, 24, 72, 72, 56, 70, scaling=YARN, kv_from=1), 136),
        (latent(2, 16, 8, 24, 40, 24, 1, base=50.0), 72),
        (mingru(52), 40)]),
    # one stream, one head, no feed-forward, window of two; values that often coincide
    "single": stack(64, 64, 1, [(latent(1, 64, 64, 64, 64, 64, 2), None), (hgrn2(1, 8, 4), None), (mingru(64), 64)]),
    # the sizes of a real layer, few of them
    "large": stack(256, 512, 2, [
        (latent(16, 128, 64, 128, 512, 384, 150, scaling=YARN), 512),
        (hgrn2(4, 128, 128), None),
        (mingru(512), None),
        (latent(16, 128, 64, 128, 512, 384, 150, scaling=YARN, kv_from=0), 512)], eps=1e-6),
    # more heads than one tile, wide latents and heads, wide recurrences, five streams
    "wide": stack(192, 260, 5, [
        (latent(17, 192, 64, 256, 640, 192, 45), None),
        (hgrn2(2, 200, 72), 192),
        (latent(40, 16, 16, 16, 128, 64, 300, kv_from=None), 64)]),
    # Dugilorn.  Sizes odd in their own way: partly rotated heads, norm parts that cut through heads, one to five taps, a
    # window of one, layers without a feed-forward
    "odd": dugilorn(136, 331, 12.0, [
        (parallel(window(6, 3, 20, 24, 37, dims=12), state_space(6, 20, 24, 3, 3, 5), 0.7, 1.3), 200),
        (gla(3, 24, 40, 8.0), None),
        (parallel(window(5, 1, 40, 72, 1, base=50.0), state_space(4, 16, 16, 4, 1, 1), -0.9, 0.8), None),
        (gla(2, 8, 12, 1.0), 40),
        (parallel(window(4, 4, 16, 8, 70, scale=0.4), state_space(2, 136, 40, 1, 5, 2), 1.0, 0.5), 72)], eps=1e-4),
    # values that often coincide
    "plain": dugilorn(64, 64, 30.0, [(parallel(window(1, 1, 64, 64, 2), state_space(1, 64, 64, 1, 4, 1)), 64),
                                     (gla(1, 64, 64, 16.0), 64)]),
    # the sizes of a real layer, few of them
    "real": dugilorn(512, 512, 50.0, [
        (parallel(window(8, 2, 128, 128, 150, base=1e5), state_space(8, 64, 128, 2, 4, 2), 0.8, 0.6), 1024),
        (gla(4, 128, 128, 16.0), 512),
        (parallel(window(8, 4, 64, 192, 129, dims=32), state_space(8, 32, 64, 1, 4, 8), 0.5, 1.2), None)], eps=1e-6),
    # more heads than a tile, keys, values, states and recurrent heads beyond the tensor-core forms
    "broad": dugilorn(192, 260, 20.0, [
        (parallel(window(34, 2, 72, 136, 45), state_space(3, 144, 200, 1, 9, 3), 0.9, 0.9), 64),
        (gla(2, 200, 136, 4.0), None),
        (parallel(window(2, 1, 264, 320, 300), state_space(4, 8, 8, 2, 2, 2), 1.1, 0.7), 64)]),
}


def shapes(config):
    from b200attn.hybrid import HybridConfig, HybridWeights
    return HybridWeights(HybridConfig.from_config(config)).shapes()


def checkpoint(config, seed=0):
    """name -> bf16 tensor"""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(config).items():
        leaf = name.rsplit(".", 1)[-1]
        x = torch.randn(shape, generator=gen)
        if name == "embed":
            pass
        elif leaf.startswith("norm"):
            x = 1.0 + 0.3 * x
        elif leaf == "lower":
            x = torch.rand(shape, generator=gen) * 0.95
        elif leaf == "b":
            x = x * 1.5
        elif leaf == "mix":
            x = 0.6 * torch.eye(shape[0]) + 0.3 * x
        elif leaf == "dt_bias":
            x = 1.2 * x - 1.5
        elif leaf == "D":
            x = 1.0 + 0.3 * x
        elif leaf == "conv":
            x = 0.6 * x
        elif leaf == "in" and len(shape) == 1:
            x = (1.0 + 0.5 * x) / shape[0] ** 0.5
        elif leaf == "out":
            x = 1.0 + 0.3 * x
        elif len(shape) == 2:
            x = x / shape[1] ** 0.5
            if leaf in ("uq", "q"):
                x = x * 1.7                       # attention that is not flat
        out[name] = x.to(torch.bfloat16)
    return out


def oracle_weights(tensors):
    return {k: v.double() for k, v in tensors.items()}


def tokens(config, n, seed):
    return torch.randint(0, config["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def logit_errors(got, want):
    """rms difference of every row over the vocabulary, mean removed, in units of the logits' spread."""
    d = got.double().cpu() - want.double().cpu()
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.double().std()


class Rounded(TorchDispatchMode):
    """Rounds operands and results of the matrix products inside to bf16: the restatement run under it shows how large an
    error rounding alone makes on a model."""

    def __torch_dispatch__(self, func, types, args=(), kwargs=None):
        if func is torch.ops.aten.mm.default:
            args = [a.to(torch.bfloat16).to(a.dtype) for a in args]
            out = func(*args, **(kwargs or {}))
            return out.to(torch.bfloat16).to(out.dtype)
        return func(*args, **(kwargs or {}))


def rounding_errors(config, weights, toks, want):
    with Rounded():
        got, layers = R.forward(config, weights, toks)
    return logit_errors(got, want), layers


def check_logits(got, want, dt, rounding=None, what="", limit=2e-5):
    """fp32: every row within `limit` of the restatement.  bf16: the typical and the largest error stay within a small
    multiple of what rounding the products' operands and results does to the restatement itself (`rounding`: its
    rows' errors); a wrong key, window or state moves a row by about the logits' spread."""
    assert got.shape == want.shape and torch.isfinite(got).all(), what
    e = logit_errors(got, want)
    if dt == "f32":
        assert float(e.max()) < limit, f"{what}: {float(e.max()):.2e} at row {int(e.argmax())}"
    else:
        mid, top = float(rounding.median()), float(rounding.max())
        assert float(e.median()) < (2 * mid if len(e) > 20 else 2.5 * top) and float(e.max()) < 2.5 * top, (
            f"{what}: median {float(e.median()):.3f} (rounding {mid:.3f}), largest {float(e.max()):.3f} at row "
            f"{int(e.argmax())} (rounding {top:.3f})")
