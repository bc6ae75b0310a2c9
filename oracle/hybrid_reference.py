"""Plain, slow restatement of the hybrid decoder stacks in eager PyTorch on the CPU, written from the equations of the
designs: one function per mechanism, whole sequences only, no cache, no chunks.  Tofilorn: latent attention / HGRN2 /
minGRU mixers, hyper-connected residual streams, scalar-gain RMS norms.  Dugilorn: windowed attention beside a state-space
mixer, gated linear attention, mixer and feed-forward reading one norm.  Tests compare the CUDA path with it; the
product never imports it.

Everything is computed in the dtype of the weights handed in (tests use float64).  `weights` maps tensor names
("l0.mix.dq", ...) to tensors; `config` is the parsed config.json dictionary.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------------------------------------- small mechanisms
def rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rotary_frequencies(rot):
    """(frequencies [dims/2] in float64, amplitude of cos and sin) of a rotation, with the YaRN ramp when scaled."""
    dims, base = rot["dims"], float(rot["base"])
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    scaling = rot.get("scaling")
    if not scaling:
        return torch.tensor(freqs, dtype=torch.float64), 1.0

    def turn(t):
        return dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    low = max(math.floor(turn(scaling["fast"])), 0)
    high = min(math.ceil(turn(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(max((i - low) / max(high - low, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, rot, positions):
    """Interleaved rotation of the first rot.dims entries of the last axis; x [T, ..., D], positions [T]."""
    freqs, amplitude = rotary_frequencies(rot)
    angle = positions.double()[:, None] * freqs[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (freqs.numel(),)
    cos = (torch.cos(angle) * amplitude).view(shape).to(x.dtype)
    sin = (torch.sin(angle) * amplitude).view(shape).to(x.dtype)
    out = x.clone()
    u, v = x[..., 0: rot["dims"]: 2], x[..., 1: rot["dims"]: 2]
    out[..., 0: rot["dims"]: 2] = u * cos - v * sin
    out[..., 1: rot["dims"]: 2] = v * cos + u * sin
    return out


def window_attention(q, k, v, scale, window):
    """q, k [T, H, D], v [T, H, Dv]; query i sees keys j with 0 <= i - j < window; ordinary softmax."""
    T = q.shape[0]
    scores = torch.einsum("ihd,jhd->hij", q, k) * scale
    gap = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    scores = scores.masked_fill(~((gap >= 0) & (gap < window))[None], float("-inf"))
    return torch.einsum("hij,jhd->ihd", torch.softmax(scores, dim=-1), v)


def gated_sum(gate, candidate):
    """S_t = (1 - gate_t) S_(t-1) + gate_t candidate_t from S = 0, element by element; [T, width]."""
    state, out = torch.zeros_like(candidate[0]), []
    for g, c in zip(gate, candidate):
        state = (1.0 - g) * state + g * c
        out.append(state)
    return torch.stack(out)


def forget_outer_recurrence(q, f, v):
    """S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T, o_t = S_t^T q_t per head; q, f [T, H, D], v [T, H, Dv]."""
    T, heads, dim = q.shape
    state, out = torch.zeros(heads, dim, v.shape[-1], dtype=q.dtype), []
    for t in range(T):
        state = f[t][:, :, None] * state + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", state, q[t]))
    return torch.stack(out)


# ------------------------------------------------------------------------------------------------------------ mixers
def latent(h, w, pre, mixer, eps):
    """(latent c [T, kv_rank], rotated shared key part [T, rot_dim]) of a layer that has its own down-projection."""
    down = h @ w[pre + "dkv"].T
    rank = mixer["kv_rank"]
    c = rms(down[:, :rank], eps) * w[pre + "dkv.norm"]
    return c, rotate(down[:, rank:], mixer["rot"], torch.arange(h.shape[0]))


def latent_attention(h, w, pre, mixer, eps, kept):
    T, heads, dim, rot_dim = h.shape[0], mixer["heads"], mixer["dim"], mixer["rot_dim"]
    c_q = rms(h @ w[pre + "dq"].T, eps) * w[pre + "dq.norm"]
    q = (c_q @ w[pre + "uq"].T).view(T, heads, dim + rot_dim)
    q_rot = rotate(q[..., dim:], mixer["rot"], torch.arange(T))
    c, k_rot = kept
    k = (c @ w[pre + "uk"].T).view(T, heads, dim)
    v = (c @ w[pre + "uv"].T).view(T, heads, mixer["vdim"])
    q_all = torch.cat((q[..., :dim], q_rot), dim=-1)
    k_all = torch.cat((k, k_rot[:, None, :].expand(T, heads, rot_dim)), dim=-1)
    o = window_attention(q_all, k_all, v, mixer["scale"], mixer["mask"]["size"])
    return o.reshape(T, -1) @ w[pre + "o"].T


def mingru(h, w, pre, mixer, eps):
    z = sigmoid(h @ w[pre + "z"].T + w[pre + "z.b"])
    u = h @ w[pre + "x"].T + w[pre + "x.b"]
    candidate = torch.where(u >= 0, u + 0.5, sigmoid(u))
    state = gated_sum(z, candidate)
    return (state * silu(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def hgrn2(h, w, pre, mixer, eps):
    T, heads, dim, vdim = h.shape[0], mixer["heads"], mixer["dim"], mixer["vdim"]
    q = silu(h @ w[pre + "q"].T).view(T, heads, dim)
    v = (h @ w[pre + "v"].T).view(T, heads, vdim)
    low = w[pre + "lower"]
    f = (low + (1.0 - low) * sigmoid(h @ w[pre + "f"].T + w[pre + "f.b"])).view(T, heads, dim)
    o = rms(forget_outer_recurrence(q, f, v), eps) * w[pre + "norm"]
    return o.reshape(T, -1) @ w[pre + "o"].T


def swiglu_mlp(h, w, pre):
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


# ------------------------------------------------------------------------------- windowed attention, state space, gla
def rotate_halves(x, rot, positions):
    """Rotation of the first rot.dims entries of the last axis, entry i paired with entry i + dims/2."""
    n = rot["dims"] // 2
    freqs, _ = rotary_frequencies(rot)
    angle = positions.double()[:, None] * freqs[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (n,)
    cos, sin = torch.cos(angle).view(shape).to(x.dtype), torch.sin(angle).view(shape).to(x.dtype)
    u, v = x[..., :n], x[..., n: 2 * n]
    return torch.cat((u * cos - v * sin, v * cos + u * sin, x[..., 2 * n:]), dim=-1)


def biased(h, w, name):
    return h @ w[name].T + w[name + ".b"]


def gated_window_attention(h, w, pre, m):
    """Grouped query heads over a sliding window, the heads' outputs times sigmoid of a gate, W_o."""
    T, heads, kv = h.shape[0], m["heads"], m["kv_heads"]
    at = torch.arange(T)
    q = rotate_halves(biased(h, w, pre + "q").view(T, heads, m["dim"]), m["rot"], at)
    k = rotate_halves(biased(h, w, pre + "k").view(T, kv, m["dim"]), m["rot"], at)
    v = biased(h, w, pre + "v").view(T, kv, m["vdim"])
    owner = torch.tensor([i // (heads // kv) for i in range(heads)])
    o = window_attention(q, k[:, owner], v[:, owner], m["scale"], m["mask"]["size"]).reshape(T, -1)
    return (o * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def causal_conv(x, taps, bias):
    """out[t] = sum_j taps[:, K-1-j] x[t-j] + bias with zeros before the start; x [T, channels], taps [channels, K]."""
    out = torch.zeros_like(x)
    for j in range(taps.shape[1]):
        moved = torch.zeros_like(x)
        moved[j:] = x[: max(x.shape[0] - j, 0)]
        out = out + moved * taps[:, taps.shape[1] - 1 - j]
    return out + bias


def softplus(u):
    return torch.clamp(u, min=0) + torch.log1p(torch.exp(-u.abs()))


def state_space_recurrence(x, B, C, dt, A_log, D):
    """S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T, y_t = S_t^T C_t + D x_t; x [T, H, P], B, C [T, H, N], dt [T, H]."""
    T, heads, vdim = x.shape
    S, out = torch.zeros(heads, B.shape[-1], vdim, dtype=x.dtype), []
    for t in range(T):
        keep = torch.exp(-torch.exp(A_log) * dt[t])
        S = keep[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, C[t]) + D[:, None] * x[t])
    return torch.stack(out)


def grouped_rms(x, groups, eps):
    return rms(x.view(*x.shape[:-1], groups, -1), eps).reshape(x.shape)


def state_space(h, w, pre, m, eps):
    T, heads, vdim, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = heads * vdim
    z, xbc, dt = (h @ w[pre + "in"].T).split([inner, inner + 2 * G * N, heads], dim=-1)
    xbc = silu(causal_conv(xbc, w[pre + "conv"], w[pre + "conv.b"]))
    x, B, C = xbc.split([inner, G * N, G * N], dim=-1)
    owner = torch.tensor([i // (heads // G) for i in range(heads)])
    y = state_space_recurrence(x.view(T, heads, vdim), B.view(T, G, N)[:, owner], C.view(T, G, N)[:, owner],
                               softplus(dt + w[pre + "dt_bias"]), w[pre + "A_log"], w[pre + "D"]).reshape(T, inner)
    y = grouped_rms(y * silu(z), m["norm_groups"], eps) * w[pre + "norm"]
    return y @ w[pre + "o"].T


def decayed_outer_recurrence(q, k, v, keep):
    """S_t = diag(keep_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t; q, k, keep [T, H, D], v [T, H, Dv]."""
    S, out = torch.zeros(q.shape[1], q.shape[2], v.shape[-1], dtype=q.dtype), []
    for t in range(q.shape[0]):
        S = keep[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def gated_linear_attention(h, w, pre, m, eps):
    T, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).view(T, heads, dim) * dim ** -0.5
    k = (h @ w[pre + "k"].T).view(T, heads, dim)
    v = (h @ w[pre + "v"].T).view(T, heads, vdim)
    z = (h @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "a2.b"]
    keep = torch.exp(-softplus(-z) / m["tau"]).view(T, heads, dim)          # sigmoid(z) ** (1 / tau)
    o = rms(decayed_outer_recurrence(q, k, v, keep), eps) * w[pre + "norm"]
    return (o.reshape(T, -1) * silu(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def side_by_side(h, w, pre, m, eps):
    return (m["left_scale"] * gated_window_attention(h, w, pre + "left.", m["left"])
            + m["right_scale"] * state_space(h, w, pre + "right.", m["right"], eps))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def geglu_mlp(h, w, pre):
    return (gelu_tanh(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def forward_dugilorn(config, w, tokens):
    """(logits [T, vocab], residual stream after every layer) of a stack whose layers add mixer(h) + ff(h), h = norm(x)."""
    eps = config["norm"]["eps"]
    x, trail = w["embed"][torch.tensor(tokens)], []
    for i, layer in enumerate(config["layers"]):
        pre = f"l{i}."
        h = rms(x, eps) * w[pre + "norm1"]
        y = {"parallel": side_by_side, "gla": gated_linear_attention}[layer["type"]](h, w, pre + "mix.", layer["mixer"], eps)
        if layer["mlp"] is not None:
            y = y + geglu_mlp(h, w, pre + "mlp.")
        x = x + y
        trail.append(x)
    logits = (rms(x, eps) * w["final.norm"]) @ w["head"].T
    cap = config["logit_softcap"]
    return cap * torch.tanh(logits / cap), torch.stack(trail)


# ------------------------------------------------------------------------------------------------------------- stack
def hyper_connect(streams, w, pre, sublayer):
    """u = sum_s in[s] x_s; y = sublayer(u); x_t <- sum_s mix[s, t] x_s + out[t] y.  streams [S, T, width]."""
    u = torch.einsum("s,stw->tw", w[pre + "in"], streams)
    y = sublayer(u)
    return torch.einsum("st,snw->tnw", w[pre + "mix"], streams) + w[pre + "out"][:, None, None] * y[None]


def forward(config, w, tokens):
    """(logits [T, vocab], residual stream after every layer [layers, T, width]) of one sequence."""
    if config["architecture"] == "Dugilorn":
        return forward_dugilorn(config, w, tokens)
    eps = config["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)]
    streams = x[None].repeat(config["streams"], 1, 1)
    kept, trail = {}, []
    for i, layer in enumerate(config["layers"]):
        pre, mixer = f"l{i}.", layer["mixer"]

        def mix(u, i=i, pre=pre, mixer=mixer, kind=layer["type"]):
            h = rms(u, eps) * w[pre + "norm1"]
            if kind == "latent_attention":
                source = mixer.get("kv_from")
                if source is None:
                    kept[i] = latent(h, w, pre + "mix.", mixer, eps)
                return latent_attention(h, w, pre + "mix.", mixer, eps, kept[i if source is None else source])
            return {"mingru": mingru, "hgrn2": hgrn2}[kind](h, w, pre + "mix.", mixer, eps)

        streams = hyper_connect(streams, w, pre + "hc1.", mix)
        if layer["mlp"] is not None:
            streams = hyper_connect(streams, w, pre + "hc2.",
                                    lambda u, pre=pre: swiglu_mlp(rms(u, eps) * w[pre + "norm2"], w, pre + "mlp."))
        trail.append(streams.sum(0))
    x = streams.sum(0)
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T, torch.stack(trail)
