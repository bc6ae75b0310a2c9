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

    assert {"Tofilorn", "Qwen3.5"} <= set(models.families())
    fam = models.family(H.CONFIGS["ragged"])
    assert fam.name == "Tofilorn" and torch.float32 in fam.dtypes and fam.part == "hybrid"
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
