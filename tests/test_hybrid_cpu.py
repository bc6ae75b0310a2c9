"""Host side of the hybrid stacks, without a GPU: configuration and registry, checkpoint files, padded layout, rotation
tables, chunking and key-range arithmetic, and the plain restatement against hand-written special cases."""
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import hybrid_helpers as H
from oracle import hybrid_reference as R

ROOT = Path(__file__).resolve().parent.parent


def test_registry_chooses_by_architecture():
    from b200attn import models

    assert {"Tofilorn", "Dugilorn", "Qwen3.5"} <= set(models.families())
    for name, config in (("Tofilorn", "ragged"), ("Dugilorn", "odd")):
        fam = models.family(H.CONFIGS[config])
        assert fam.name == name and torch.float32 in fam.dtypes and fam.part == "hybrid"
    assert models.family({"architecture": "Qwen3.5"}).config({"architecture": "Qwen3.5", "hidden": 512}).hidden == 512
    with pytest.raises(ValueError, match="unknown architecture"):
        models.family({"architecture": "nobody"})


def test_configuration_errors_are_named():
    from b200attn.hybrid import HybridConfig, HybridWeights

    def weights(layers):
        return HybridWeights(HybridConfig.from_config(H.stack(64, 64, 2, layers)))

    own, other = H.latent(2, 16, 8, 16, 32, 32, 8), H.latent(2, 16, 8, 16, 48, 32, 8, kv_from=0)
    with pytest.raises(AssertionError, match="latent shape or rotation"):
        weights([(own, None), (other, None)])
    with pytest.raises(AssertionError, match="earlier layer"):
        weights([(H.latent(2, 16, 8, 16, 32, 32, 8, kv_from=1), None), (own, None)])
    with pytest.raises(AssertionError, match="keeps no latent"):
        weights([(H.mingru(32), None), (H.latent(2, 16, 8, 16, 32, 32, 8, kv_from=0), None)])
    with pytest.raises(ValueError, match="unknown mixer"):
        weights([({"type": "strange", "mixer": {}}, None)])
    config = H.CONFIGS["single"]
    tensors = H.checkpoint(config)
    w = HybridWeights(HybridConfig.from_config(config))
    with pytest.raises(KeyError, match="final.norm"):
        w.load({k: v for k, v in tensors.items() if k != "final.norm"}, torch.float32, "cpu")
    with pytest.raises(ValueError, match="head has shape"):
        w.load({**tensors, "head": tensors["head"][:-1]}, torch.float32, "cpu")


def test_safetensors_round_trip(tmp_path):
    from b200attn import checkpoint

    tensors = {"a": torch.randn(3, 5).to(torch.bfloat16), "scalar": torch.tensor(2.5), "ids": torch.arange(7, dtype=torch.int32),
               "odd": torch.tensor([1, 2, 3], dtype=torch.uint8), "after": torch.randn(2, 2)}
    checkpoint.write_safetensors(tmp_path / "m.safetensors", tensors)
    back = checkpoint.read_safetensors(tmp_path / "m.safetensors")
    assert set(back) == set(tensors)
    for k, v in tensors.items():
        assert back[k].dtype == v.dtype and torch.equal(back[k], v), k
    raw = (tmp_path / "m.safetensors").read_bytes()
    n = int.from_bytes(raw[:8], "little")
    assert json.loads(raw[8: 8 + n])["a"]["dtype"] == "BF16"


@pytest.mark.parametrize("scaling", [None, H.YARN, {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0},
                                     {"factor": 2.0, "original": 16, "fast": 4.0, "slow": 4.0}])
@pytest.mark.parametrize("dims", [2, 8, 24, 64])
def test_rotation_table(scaling, dims):
    from b200attn.mixers import Rotation

    rot = {"base": 5000.0, "dims": dims, **({"scaling": scaling} if scaling else {})}
    table = Rotation.from_config(rot).table(300, "cpu")
    x = torch.randn(300, dims, dtype=torch.float64)
    want = R.rotate(x, rot, torch.arange(300))
    cos, sin = table[..., 0].double(), table[..., 1].double()
    got = torch.stack((x[:, 0::2] * cos - x[:, 1::2] * sin, x[:, 1::2] * cos + x[:, 0::2] * sin), dim=-1).flatten(1)
    assert (got - want).abs().max() < 1e-6
    if scaling:   # the slowest pair turns `factor` times slower when its period is past the original context
        f = Rotation.from_config(rot).frequencies()
        plain = Rotation(dims, 5000.0).frequencies()
        assert torch.all(f <= plain * (1 + 1e-12)) and torch.all(f >= plain / scaling["factor"] * (1 - 1e-12))


def test_padding_keeps_heads_apart():
    from b200attn.hybrid import HybridConfig, HybridWeights

    config = H.CONFIGS["ragged"]
    tensors = H.checkpoint(config)
    w = HybridWeights(HybridConfig.from_config(config)).load(tensors, torch.float32, "cpu")
    m = w.mixers[1]
    uq = m.uq.view(m.heads, m.dim_p + m.rot_p, m.q_rank_p)
    raw = tensors["l1.mix.uq"].float().view(m.heads, m.dim + m.rot_dim, m.q_rank)
    assert torch.equal(uq[:, : m.dim, : m.q_rank], raw[:, : m.dim])
    assert torch.equal(uq[:, m.dim_p: m.dim_p + m.rot_dim, : m.q_rank], raw[:, m.dim:])
    assert not uq[:, m.dim: m.dim_p].any() and not uq[..., m.q_rank:].any()
    assert torch.equal(m.uv[:, : m.vdim, : m.rank], tensors["l1.mix.uv"].float().view(m.heads, m.vdim, m.rank))
    shared = w.mixers[3]
    assert shared.source == 1 and shared.kv_norm is None and shared.down.shape[0] == shared.q_rank_p
    assert w.embed.shape == (331, 192) and not w.embed[:, 136:].any() and w.head.shape[0] == 336
    assert len(w.joints) == len(list(w.sublayers())) + 1
    s = config["streams"]
    assert torch.equal(w.joints[1][: s * s].view(s, s), tensors["l0.hc1.mix"].float())     # [from, to]


def _core_weights(config, seed=0, rank=None):
    from b200attn.hybrid import HybridConfig, HybridWeights
    tensors = H.checkpoint(config, seed)
    if rank is not None:
        for name in [n for n in tensors if n.endswith(".a1")]:
            tensors[name] = torch.randn(rank, config["width"]).to(torch.bfloat16)
            tensors[name[:-1] + "2"] = torch.randn(tensors[name[:-1] + "2"].shape[0], rank).to(torch.bfloat16)
    return tensors, HybridWeights(HybridConfig.from_config(config)).load(tensors, torch.float32, "cpu")


def _unit_restated(unit, core_index, h):
    """What a core's columns of the input product hold."""
    x = h @ unit.w_in.T
    return x.split(unit.ins, dim=1)[core_index]


def test_cores_share_products_without_mixing():
    """Columns of the stacked products against the restatement's own projections, head by head; padding is zero."""
    config = H.CONFIGS["odd"]
    tensors, w = _core_weights(config)
    t = {k: v.float() for k, v in tensors.items()}
    h = torch.zeros(3, w.width_p)
    h[:, :136] = torch.randn(3, 136, generator=torch.Generator().manual_seed(1))
    unit = w.units[0]
    attn, ssm, mlp = (core for _, core in unit.parts)
    x = _unit_restated(unit, 0, h)
    q, k, v, g = x.split([6 * attn.dim_p, 3 * attn.dim_p, 3 * attn.vdim_p, 6 * attn.vdim_p], dim=1)
    for cols, name, heads, size in ((q, "q", 6, 20), (k, "k", 3, 20), (v, "v", 3, 24), (g, "g", 6, 24)):
        cols = cols.reshape(3, heads, -1)
        want = (h[:, :136] @ t[f"l0.mix.left.{name}"].T).view(3, heads, size)
        assert torch.allclose(cols[..., :size], want, atol=1e-4) and not cols[..., size:].any()
    x = _unit_restated(unit, 1, h)
    raw = h[:, :136] @ t["l0.mix.right.in"].T
    z, xs, b, c, dt = raw.split([120, 120, 72, 72, 6], dim=1)
    zp, xp, bp, cp, dp = x.split([6 * 32, 6 * 32, 3 * 32, 3 * 32, 8], dim=1)
    for got, want, heads, size in ((zp, z, 6, 20), (xp, xs, 6, 20), (bp, b, 3, 24), (cp, c, 3, 24)):
        got = got.reshape(3, heads, -1)
        assert torch.allclose(got[..., :size], want.reshape(3, heads, size), atol=1e-4) and not got[..., size:].any()
    assert torch.allclose(dp[:, :6], dt, atol=1e-4) and not dp[:, 6:].any()
    assert ssm.conv.shape == (4, ssm.channels) and not ssm.conv[3].any()             # three taps, the current token's first
    assert torch.equal(ssm.conv[0, :20], t["l0.mix.right.conv"][:20, 2]) and torch.equal(ssm.conv[2, 32:52], t["l0.mix.right.conv"][20:40, 0])
    assert torch.allclose(ssm.norm.view(6, 32)[:, :20].reshape(-1), 1.3 * t["l0.mix.right.norm"]) and not ssm.norm.view(6, 32)[:, 20:].any()
    assert attn.scale == 0.7 and mlp.out_size == 256
    # the product out: the parts' columns side by side, the rest zero
    a, s, m, rest = unit.w_out.split([*unit.outs, unit.pad], dim=1)
    assert torch.equal(a[:136].reshape(136, 6, 64)[..., :24].reshape(136, -1), t["l0.mix.left.o"])
    assert torch.equal(s[:136].reshape(136, 6, 32)[..., :20].reshape(136, -1), t["l0.mix.right.o"])
    assert torch.equal(m[:136, :200], t["l0.mlp.down"]) and not rest.any() and not unit.w_out[136:].any()
    assert all(torch.equal(p, unit.w_out[:, n * unit.part: (n + 1) * unit.part]) for n, p in enumerate(unit.w_parts))
    # norms: one weight vector per joint
    assert len(w.joints) == len(w.gains) == len(w.units) + 1 == 6 and torch.equal(w.gains[1][:136], t["l1.norm1"])
    assert torch.equal(w.gains[5][:136], t["final.norm"]) and not w.gains[5][136:].any()
    assert [u.layer for u in w.units] == [0, 1, 2, 3, 4] and [len(u.parts) for u in w.units] == [3, 1, 2, 2, 3]


@pytest.mark.parametrize("rank", [5, 16, 32])
def test_decay_rank_comes_from_the_checkpoint(rank):
    tensors, w = _core_weights(H.CONFIGS["odd"], rank=rank)
    core = w.units[1].parts[0][1]
    assert core.rank == rank and core.w_low.shape == (3 * core.dim_p, -(-rank // 8) * 8)
    assert torch.equal(core.w_low.view(3, core.dim_p, -1)[:, :24, :rank].reshape(72, rank), tensors["l1.mix.a2"].float())
    assert w.units[1].w_in.shape[0] == core.in_size == core.low_at + core.rank_p


def test_product_out_is_split_into_parts_the_kernel_takes():
    from b200attn import ops
    config = H.dugilorn(256, 64, 30.0, [(H.parallel(H.window(16, 4, 64, 128, 64), H.state_space(32, 64, 16, 1, 4, 1)), 1500), (H.gla(2, 16, 16, 4.0), None)])
    _, w = _core_weights(config)
    unit = w.units[0]
    assert sum(unit.outs) == 2048 + 2048 + 1536 and len(unit.w_parts) == 2 and unit.part <= ops.SKINNY_GEMM_PAIR_MAX_K
    assert ops.skinny_gemm_supports(32, 256, unit.part) and len(w.units[1].w_parts) == 1
    with pytest.raises(ValueError, match="cannot share its norm"):
        from b200attn.hybrid import HybridConfig, HybridWeights
        HybridWeights(HybridConfig.from_config(H.dugilorn(64, 64, 1.0, [(H.mingru(32), 64)])))


def test_chunking_and_splits():
    from b200attn import hybrid_ops as hops

    for n in (1, 2, 63, 64, 65, 2048, 4096, 4097, 100000):
        for groups in (1, 32, 1000):
            seg, segs = hops.mingru_segments(n, groups, 148)
            assert segs <= 64 and (segs - 1) * seg < n <= segs * seg and (segs == 1 or seg % hops.MINGRU_BLOCK == 0)
        for groups in (1, 16, 32, 500):
            seg, segs = hops.hgrn2_segments(n, groups, 148)
            assert (segs - 1) * seg < n <= segs * seg and (segs == 1 or (seg % 16 == 0 and seg >= 128))
            assert segs == 1 or segs * groups <= 2 * 148
            seg, segs = hops.ssd_segments(n, groups, 148)
            assert (segs - 1) * seg < n <= segs * seg and (segs == 1 or (seg % 32 == 0 and segs * groups <= 2 * 148))
    assert [hops.conv_taps(n) for n in (1, 4, 5, 8, 9, 16)] == [4, 4, 8, 8, 16, 16]
    for batch, heads, kv, span in [(1, 1, 1, 16), (1, 32, 2, 4096), (32, 16, 4, 2048), (256, 64, 8, 512)]:
        s = hops.window_decode_splits(batch, heads, kv, span, 148)
        assert 1 <= s <= hops.LATENT_MAX_SPLITS and (s == 1 or span // s >= 16)
    for batch, heads, span in [(1, 1, 16), (1, 16, 4096), (32, 16, 4096), (256, 128, 512), (1, 1, 1)]:
        s = hops.latent_decode_splits(batch, heads, span, 148)
        assert 1 <= s <= hops.LATENT_MAX_SPLITS and (s == 1 or span // s >= 16)


def test_packed_batch_rows():
    from b200attn.hybrid import PackedBatch

    b = PackedBatch([4, 1], [10, 0], [[7, 8, 9], [5]], "cpu")
    assert b.ids.tolist() == [7, 8, 9, 5] and b.pos.tolist() == [10, 11, 12, 0] and b.slot_of.tolist() == [4, 4, 4, 1]
    assert b.cu.tolist() == [0, 3, 4] and b.slots.tolist() == [4, 1] and b.start.tolist() == [10, 0]
    span = b.context(4)       # query 10 sees 7..10
    assert span.first.tolist() == [7, 0] and span.cu.tolist() == [0, 6, 7] and (span.keys, span.max_keys) == (7, 6)
    assert span.rows.tolist() == [3, 4, 5, 6] and span.max_old == 3      # behind the three keys of earlier passes
    b = PackedBatch([0, 1, 2], [0, 5, 2], [[1, 2], [3], [4, 5, 6]], "cpu")
    span = b.context(3)
    assert span.first.tolist() == [0, 3, 0] and span.cu.tolist() == [0, 2, 5, 10] and span.rows.tolist() == [0, 1, 4, 7, 8, 9]
    assert span.max_old == 2 and b.context(1).max_old == 0


def test_oracle_special_cases():
    """The restatement against closed forms: a window of one returns the value itself, gates pinned open or shut turn the
    recurrences into the input or a constant, a stack of one stream with unit joints is an ordinary residual."""
    g = torch.Generator().manual_seed(3)
    q, k, v = (torch.randn(6, 2, 4, generator=g, dtype=torch.float64) for _ in range(3))
    assert torch.allclose(R.window_attention(q, k, v, 0.7, 1), v)
    full = R.window_attention(q, k, v, 0.7, 99)
    p = torch.softmax(torch.tensor([[float(q[2, 1] @ k[j, 1]) * 0.7 for j in range(3)]], dtype=torch.float64), -1)
    assert torch.allclose(full[2, 1], (p @ v[:3, 1])[0])
    one = torch.ones(5, 3, dtype=torch.float64)
    c = torch.randn(5, 3, generator=g, dtype=torch.float64)
    assert torch.allclose(R.gated_sum(one, c), c) and not R.gated_sum(0 * one, c).any()
    f = torch.zeros(4, 1, 3, dtype=torch.float64)
    qq, vv = torch.randn(4, 1, 3, generator=g, dtype=torch.float64), torch.randn(4, 1, 2, generator=g, dtype=torch.float64)
    assert torch.allclose(R.forget_outer_recurrence(qq, f, vv), qq.sum(-1, keepdim=True) * vv)
    x = torch.randn(1, 5, 4, generator=g, dtype=torch.float64)
    w = {"in": torch.ones(1).double(), "out": torch.ones(1).double(), "mix": torch.ones(1, 1).double()}
    assert torch.allclose(R.hyper_connect(x, w, "", lambda u: 2 * u), 3 * x)
    x = torch.randn(6, 3, generator=g, dtype=torch.float64)
    assert torch.allclose(R.causal_conv(x, torch.tensor([[2.0]] * 3).double(), torch.zeros(3).double()), 2 * x)
    shift = R.causal_conv(x, torch.tensor([[1.0, 0.0]] * 3).double(), torch.ones(3).double())
    assert torch.allclose(shift[1:], x[:-1] + 1) and torch.allclose(shift[0], torch.ones(3).double())
    B, C, xs = (torch.randn(5, 2, n, generator=g, dtype=torch.float64) for n in (3, 3, 4))
    dt, D = torch.rand(5, 2, generator=g).double(), torch.tensor([0.5, -1.0]).double()
    gone = R.state_space_recurrence(xs, B, C, dt, torch.full((2,), 40.0).double(), D)            # every step forgets all
    assert torch.allclose(gone, (dt * (B * C).sum(-1))[..., None] * xs + D[:, None] * xs)
    kept = R.state_space_recurrence(xs, B, C, dt, torch.full((2,), -60.0).double(), 0 * D)       # nothing is forgotten
    assert torch.allclose(kept[4, 0], sum(dt[s, 0] * (B[s, 0] @ C[4, 0]) * xs[s, 0] for s in range(5)))
    keep = torch.zeros(5, 2, 3).double()
    assert torch.allclose(R.decayed_outer_recurrence(C, B, xs, keep), (B * C).sum(-1, keepdim=True) * xs)
    assert torch.allclose(R.decayed_outer_recurrence(C, B, xs, keep + 1)[4, 1], sum((B[s, 1] @ C[4, 1]) * xs[s, 1] for s in range(5)))
    y = torch.randn(2, 12, generator=g, dtype=torch.float64)
    assert torch.allclose(R.grouped_rms(y, 3, 0.0)[:, 4:8], R.rms(y[:, 4:8], 0.0)) and torch.allclose(R.gelu_tanh(torch.tensor(0.0)), torch.tensor(0.0))
    z = torch.randn(7, 2, 8, generator=g, dtype=torch.float64)
    rot = R.rotate_halves(z, {"base": 100.0, "dims": 6}, torch.arange(7))
    assert torch.equal(rot[0], z[0]) and torch.equal(rot[..., 6:], z[..., 6:]) and torch.allclose(rot.norm(dim=-1), z.norm(dim=-1))
    assert torch.allclose(rot[2, 0, 0], z[2, 0, 0] * math.cos(2.0) - z[2, 0, 3] * math.sin(2.0))
    assert math.isclose(float(R.silu(torch.tensor(1.0))), 1 / (1 + math.exp(-1)), rel_tol=1e-6)


def test_trace_command_checks_the_model_first(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Qwen3.5"}))
    res = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                          str(tmp_path), "--max-tokens", "8"], capture_output=True, text=True, stdin=subprocess.DEVNULL)
    assert res.returncode == 3, res.stderr


def test_library_part_has_what_the_family_needs():
    """The sources named for the part link on their own (the linker flags nothing undefined of ours)."""
    import importlib.util

    spec = importlib.util.spec_from_file_location("b200_build_parts", ROOT / "qwen3_5-triton-inference-engine_b200" / "build.py")
    build = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(build)
    for lib, names in build.PARTS.values():
        for n in names:
            assert (build.CSRC / f"{n}.cu").exists(), n
