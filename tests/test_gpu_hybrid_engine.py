"""Whole hybrid stacks through the engine, the batcher and the command line against the plain restatement: whole prompts,
token-by-token decoding, portions down to two tokens, unequal batches against each request alone, slots and pages used
again, long decoding, graph replay, greedy generation.  fp32 engines are held to fp32 rounding, bf16 ones to bf16's."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import hybrid_helpers as H
from oracle import hybrid_reference as R

pytestmark = pytest.mark.gpu
DEV = "cuda"
ROOT = Path(__file__).resolve().parent.parent
DTYPES = {"f32": torch.float32, "bf16": torch.bfloat16}
_models, _wanted = {}, {}


def model(name, dt):
    from b200attn import models
    if (name, dt) not in _models:
        config = H.CONFIGS[name]
        fam = models.family(config)
        cfg = fam.config(config)
        weights = fam.load(cfg, H.checkpoint(config), DTYPES[dt], DEV)
        _models[name, dt] = models.Model(fam, cfg, weights)
    return _models[name, dt]


def wanted(name, n, seed):
    """(tokens, logits [n, vocab], residuals) of the restatement; longer ones are cut from the longest asked for so far."""
    key = (name, n, seed)
    if key not in _wanted:
        config = H.CONFIGS[name]
        toks = H.tokens(config, n, seed)
        _wanted[key] = (toks, *R.forward(config, H.oracle_weights(H.checkpoint(config)), toks))
    return _wanted[key]


def rounding(name):
    """What bf16 rounding alone does to this model's rows (one long request)."""
    key = (name, "rounding")
    if key not in _wanted:
        config = H.CONFIGS[name]
        toks, want, layers = wanted(name, 170, 1)
        rows, rounded = H.rounding_errors(config, H.oracle_weights(H.checkpoint(config)), toks, want)
        _wanted[key] = rows, [float((a - b).abs().max() / b.abs().max()) for a, b in zip(rounded, layers)]
    return _wanted[key]


def check(name, got, want, dt, what="", limit=2e-5):
    H.check_logits(got, want, dt, rounding(name)[0] if dt == "bf16" else None, what, limit)


def engine(name, dt, batch=3, context=256, **kw):
    kw.setdefault("on_demand_pages", True)
    return model(name, dt).engine(batch, context, DEV, **kw)


def run_portions(eng, slot, toks, sizes):
    """All logits of one request fed in portions of the given sizes (the last size repeats)."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(k, len(sizes) - 1)], len(toks) - at)
        out.append(eng.extend([slot], [at], [toks[at: at + n]], [list(range(n))]))
        at, k = at + n, k + 1
    return torch.cat(out)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("name", H.CONFIGS)
def test_whole_prompt_layer_by_layer(name, dt):
    toks, want, layers = wanted(name, 170, 1)
    eng = engine(name, dt)
    eng.trace = []
    got = eng.extend([1], [0], [toks], [list(range(len(toks)))])
    for i, (a, b) in enumerate(zip(eng.trace, layers)):
        err = float((a.double().cpu() - b).abs().max() / b.abs().max())
        assert err < (2e-5 if dt == "f32" else 3 * rounding(name)[1][i]), f"layer {i}: {err:.2e}"
    check(name, got, want, dt)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("name", H.CONFIGS)
def test_token_by_token_from_the_first(name, dt):
    toks, want, _ = wanted(name, 170, 1)
    n = 60 if name in ("wide", "broad") else 100
    got = run_portions(engine(name, dt), 2, toks[:n], [1])
    check(name, got, want[:n], dt)


@pytest.mark.parametrize("sizes", [[2], [3, 2], [16], [17, 1, 30], [64, 2, 63, 1], [150, 1]])
@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("name", ["ragged", "large", "odd", "real"])
def test_portions(name, dt, sizes):
    toks, want, _ = wanted(name, 170, 1)
    got = run_portions(engine(name, dt), 0, toks, sizes)
    check(name, got, want, dt)


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("name", H.CONFIGS)
def test_unequal_batch_and_used_slots(name, dt):
    """Requests of unequal lengths and portions in one pass, in slots and pages other requests have just left."""
    eng = engine(name, dt, batch=4, context=208, num_pages=30)
    junk = H.tokens(H.CONFIGS[name], 200, 99)
    for slot in (3, 0):
        eng.extend([slot], [0], [junk])
        eng.extend([slot], [200], [junk[:1]])
        eng.pages.release(slot)
    lengths = {0: 1, 1: 33, 3: 170}
    reqs = {s: wanted(name, n, 1 if n == 170 else 10 + s) for s, n in lengths.items()}
    cuts = [{1: 2, 3: 40}, {0: 1, 1: 17, 3: 3}, {3: 90}, {1: 13, 3: 2}, {1: 1, 3: 35}]
    at = {s: 0 for s in lengths}
    got = {s: [] for s in lengths}
    for cut in cuts:
        slots = list(cut)
        portions = [reqs[s][0][at[s]: at[s] + n] for s, n in cut.items()]
        assert all(len(p) == n for p, n in zip(portions, cut.values()))
        logits = eng.extend(slots, [at[s] for s in slots], portions, [list(range(len(p))) for p in portions])
        for s, part in zip(slots, logits.split([len(p) for p in portions])):
            got[s].append(part)
            at[s] += part.shape[0]
        eng.pages.check()
    assert at == lengths
    for s in lengths:
        check(name, torch.cat(got[s]), reqs[s][1], dt, f"slot {s}")


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("name", ["ragged", "odd"])
def test_decoding_some_slots_leaves_the_others_alone(name, dt):
    toks, want, _ = wanted(name, 170, 1)
    other, other_want, _ = wanted(name, 60, 5)
    eng = engine(name, dt)
    a = [eng.extend([0], [0], [toks[:30]], [[29]])]
    b = [eng.extend([2], [0], [other[:20]], [[19]])]
    for i in range(30, 60):                                # slot 2 pauses every other step, in between both decode
        if i % 2:
            a.append(eng.extend([0], [i], [[toks[i]]], [[0]]))
        else:
            j = 20 + (i - 30) // 2
            both = eng.extend([2, 0], [j, i], [[other[j]], [toks[i]]], [[0], [0]])
            b.append(both[:1])
            a.append(both[1:])
    check(name, torch.cat(a), want[29:60], dt)
    check(name, torch.cat(b), other_want[19:35], dt)


@pytest.mark.parametrize("name", ["ragged", "odd"])
def test_long_decoding_stays_exact(name):
    """Several windows' worth of decoded tokens: windows slide over decoded keys, pages fill, states run on."""
    toks, want, _ = wanted(name, 400, 3)
    eng = engine(name, "f32", context=400)
    got = torch.cat((eng.extend([0], [0], [toks[:20]], [list(range(20))]), run_from(eng, 0, toks, 20)))
    check(name, got, want, "f32", limit=3e-5)


def run_from(eng, slot, toks, at):
    return torch.cat([eng.extend([slot], [i], [[toks[i]]], [[0]]) for i in range(at, len(toks))])


@pytest.mark.parametrize("dt", DTYPES)
@pytest.mark.parametrize("chunk", [None, 7, 64])
@pytest.mark.parametrize("name", ["ragged", "odd"])
def test_prefill_in_chunks_and_graph_decode(name, dt, chunk):
    """`prefill` (whole or cut) + `step`, eager and as a graph replay, teacher-forced on the restatement's greedy choice:
    where its margin is beyond rounding the engine's token is the same."""
    config = H.CONFIGS[name]
    w = H.oracle_weights(H.checkpoint(config))
    prompts = [H.tokens(config, n, 40 + n) for n in (3, 50, 130)]
    refs = []
    for p in prompts:
        seq = list(p)
        for _ in range(9):
            seq.append(int(R.forward(config, w, seq)[0][-1].argmax()))
        logits = R.forward(config, w, seq)[0]
        refs.append((seq, logits))
    runs = []
    for graph in (False, True):
        eng = engine(name, dt, on_demand_pages=False, page_seed=3, prefill_chunk=chunk)
        ids = [eng.prefill(prompts).tolist()]
        for k in range(8):
            eng.tok.copy_(torch.tensor([refs[b][0][len(prompts[b]) + k] for b in range(3)]))
            ids.append(eng.step().tolist())
            if graph and k == 1:
                eng.capture()
        assert eng.pos.tolist() == [len(p) + 8 for p in prompts]
        runs.append(ids)
    for b, (seq, logits) in enumerate(refs):
        for k in range(9):
            row = logits[len(prompts[b]) - 1 + k]
            for ids in runs:
                gap = float(row.max() - row[ids[k][b]]) / float(row.std())
                assert gap < (1e-4 if dt == "f32" else 0.15), (b, k, gap)


@pytest.mark.parametrize("graph", [False, True])
@pytest.mark.parametrize("name", ["ragged", "odd"])
def test_continuous_batching(name, graph):
    """Requests of different lengths through few slots and a pool too small for all: every page comes back, and each
    request's greedy tokens are the restatement's (fp32; a near-tie may fall either way, checked by its margin)."""
    from b200attn.serving import ContinuousBatcher
    config = H.CONFIGS[name]
    w = H.oracle_weights(H.checkpoint(config))
    eng = engine(name, "f32", batch=3, context=96, num_pages=12, prefill_chunk=20)
    cb = ContinuousBatcher(eng, check_invariants=True)
    prompts = [H.tokens(config, n, 70 + n) for n in (5, 40, 17, 48, 33, 9)]
    budgets = [12, 20, 30, 8, 25, 28]
    rids = []
    for i, (p, n) in enumerate(zip(prompts, budgets)):
        rids.append(cb.submit(p, n))
        if i in (1, 3):
            cb.step()
            cb.step()
            if graph and eng.graph is None:
                eng.capture()
    out = cb.run(max_steps=500)
    assert eng.pages.num_free == 11 and (eng.block_table == eng.pages.spare).all()
    for rid, prompt, n in zip(rids, prompts, budgets):
        got = out[rid]
        assert len(got) == n
        logits = R.forward(config, w, prompt + got)[0][len(prompt) - 1: -1]
        margin = (logits.max(-1).values - logits.gather(1, torch.tensor(got)[:, None])[:, 0]) / logits.std()
        assert float(margin.max()) < 1e-4


@pytest.mark.parametrize("dt", DTYPES)
def test_shared_latent_reads_the_rows_of_its_source(dt):
    """Changing the sharing layer's own weights leaves the cache alone; changing the source's changes both layers."""
    eng = engine("large", dt)
    toks = wanted("large", 170, 1)[0][:40]
    eng.extend([0], [0], [toks])
    assert "cache" in eng.states[0] and "cache" not in eng.states[3]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["ragged", "odd"])
def test_command_line(tmp_path, name, dtype):
    """generate and trace on a model folder: the trace of a prompt plus what was generated gives the same tokens."""
    from b200attn import checkpoint
    config = H.CONFIGS[name]
    (tmp_path / "config.json").write_text(json.dumps(config))
    checkpoint.write_safetensors(tmp_path / "model.safetensors", H.checkpoint(config))
    prompts = [H.tokens(config, n, 5 + n) for n in (4, 60)]
    res = subprocess.run([sys.executable, str(ROOT / "bin" / "generate"), "--model", str(tmp_path), "--dtype", dtype,
                          "--max-new-tokens", "6"], input="\n".join(json.dumps(p) for p in prompts), capture_output=True, text=True)
    assert res.returncode == 0, res.stderr
    made = [json.loads(line) for line in res.stdout.splitlines()]
    steps, w = [], H.oracle_weights(H.checkpoint(config))
    for i, (p, g) in enumerate(zip(prompts, made)):
        assert len(g) == 6
        steps.append({"step": 2 * i, "entries": [{"id": f"q{i}", "tokens": p, "want": [len(p) - 1]}], "end": []})
        steps.append({"step": 2 * i + 1, "entries": [{"id": f"q{i}", "tokens": g[:1], "want": [0]}], "end": [f"q{i}"]})
    res = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out",
                          str(tmp_path), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                         capture_output=True, text=True)
    assert res.returncode == 0, res.stderr
    assert [line for line in res.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(4)]
    for i, (p, g) in enumerate(zip(prompts, made)):
        want = R.forward(config, w, p + g[:1])[0][-2:]
        got = torch.stack([torch.frombuffer(bytearray((tmp_path / f"{2 * i + k}.f32").read_bytes()), dtype=torch.float32)
                           for k in range(2)])
        assert got.shape == (2, config["vocab"])
        check(name, got, want, "f32" if dtype == "float32" else "bf16")
