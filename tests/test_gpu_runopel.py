"""The Runopel decoder through the framework's own entry points against the plain forward pass: prompts, portions,
token-by-token decoding, slots, long decoding, generation, the command line and the trace runner."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from hf2q_b200 import registry, safetensors
from hf2q_b200.engine import Engine, Entry
from hf2q_b200.runopel import RunopelConfig, RunopelDecoder
from hf2q_b200.ops import Hf2qError
from oracle import runopel_forward as F
from tests import runopel_util as U

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
TOL = {torch.float32: 1e-4}
LEN = {"a": 190, "b": 120, "c": 330}


def config_of(name, dtype):
    """In bf16 every expert is taken: two scores that nearly tie would let the rounded rows choose the other one."""
    return U.CONFIGS[name] if dtype == torch.float32 else U.all_experts(U.CONFIGS[name])


def load(ctx, name, dtype, seed=0, **kw):
    cfg = config_of(name, dtype)
    w = U.weights(cfg, seed)
    kw.setdefault("max_seq", 1024)
    return RunopelDecoder(ctx, RunopelConfig(cfg), w.__getitem__, dtype=dtype, **kw), cfg, w


_want = {}


def want_of(name, n, seed=1, dtype=torch.float32):
    if (name, n, seed, dtype) not in _want:
        cfg = config_of(name, dtype)
        ids = U.tokens(cfg, n, seed)
        _want[name, n, seed, dtype] = ids, U.oracle_logits(cfg, U.weights(cfg), ids)
    return _want[name, n, seed, dtype]


def run(m, ids, cuts):
    slot, out, at = m.open_slot(), [], 0
    for c in cuts:
        out.append(m.extend(slot, torch.tensor(ids[at:at + c], dtype=torch.int32), range(c)))
        at += c
    m.close_slot(slot)
    m.ctx.check_status()
    return torch.cat(out)


def cuts_of(n, pattern):
    out = []
    while sum(out) < n:
        out.append(min(pattern[len(out) % len(pattern)], n - sum(out)))
    return out


@pytest.mark.parametrize("name", ["a", "b", "c"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_prompt_portions_and_single_tokens(gpu_ctx, name, dtype):
    m, cfg, _ = load(gpu_ctx, name, dtype)
    ids, want = want_of(name, LEN[name], dtype=dtype)
    n = len(ids)
    for cuts in ([n], [1] * n, cuts_of(n, [3, 64, 2, 2, 7, 1]), cuts_of(n, [2]), [n - 5] + [1] * 5):
        assert U.close(run(m, ids, cuts), want, dtype), cuts[:6]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_every_layer_run(gpu_ctx, dtype):
    m, cfg, w = load(gpu_ctx, "a", dtype)
    ids, _ = want_of("a", 60)
    got, want = [], []
    m.on_layer = lambda r, x: got.append(x.clone())
    slot = m.open_slot()
    m.extend(slot, torch.tensor(ids, dtype=torch.int32), [])
    F.forward(cfg, U.as_f64(w), ids, want)
    assert len(got) == len(want) == len(m.layers)
    for r, (a, b) in enumerate(zip(got, want)):
        e = U.errors(a, b)
        assert e.max() < 1e-4 if dtype == torch.float32 else np.median(e) < 5e-2 and e.max() < 0.3, (r, np.median(e), e.max())


def test_internal_chunks_do_not_show(gpu_ctx):
    ids, want = want_of("a", LEN["a"])
    for chunk in (16, 50):
        m, _, _ = load(gpu_ctx, "a", torch.float32, prefill_chunk=chunk)
        assert U.error(run(m, ids, [len(ids)]), want) < TOL[torch.float32]
        assert U.error(run(m, ids, [100, 90]), want) < TOL[torch.float32]


def test_a_sequence_no_longer_than_the_window(gpu_ctx):
    """max_seq below the window: the ring is cut to what can be filled."""
    m, _, _ = load(gpu_ctx, "c", torch.float32, max_seq=100)
    ids, want = want_of("c", 100)
    assert U.error(run(m, ids, [70] + [1] * 30), want) < TOL[torch.float32]
    slot = m.open_slot()
    with pytest.raises(Hf2qError):
        m.extend(slot, torch.zeros(101, dtype=torch.int32), [])


def test_the_first_token_is_still_seen_far_away(gpu_ctx):
    """Two prompts that differ in their first token: the logits' difference at the end, beyond every window, must be the
    plain forward's (it travels through the recurrent states alone)."""
    cfg, w = U.CFG_A, U.weights(U.CFG_A)
    for name in w:                                               # weak decays keep the states
        if name.endswith(".A_log"):
            w[name] = w[name] - 5.0
    m = RunopelDecoder(gpu_ctx, RunopelConfig(cfg), w.__getitem__, dtype=torch.float32, max_seq=256)
    ids = U.tokens(cfg, 160)
    other = [(ids[0] + 5) % cfg["vocab"]] + ids[1:]
    want = U.oracle_logits(cfg, w, other)[-1] - U.oracle_logits(cfg, w, ids)[-1]
    assert np.abs(want).max() > 1e-3
    for cuts in ([160], [100] + [1] * 60, cuts_of(160, [2, 31])):
        got = (run(m, other, cuts)[-1] - run(m, ids, cuts)[-1]).double().cpu().numpy()
        assert np.linalg.norm(got - want) / np.linalg.norm(want) < 2e-2, cuts[:4]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_interleaved_sequences_and_reused_slots(gpu_ctx, dtype):
    m, cfg, w = load(gpu_ctx, "a", dtype, n_slots=2)
    e = Engine(m)
    seqs = {i: want_of("a", n, seed, dtype) for i, (n, seed) in {"p": (70, 1), "q": (41, 2), "r": (90, 3), "s": (23, 4)}.items()}
    at, rows = {i: 0 for i in seqs}, {i: [] for i in seqs}
    rng = np.random.default_rng(0)
    live, waiting = ["p", "q"], ["r", "s"]
    while live:
        entries, end = [], []
        for i in list(live):
            ids = seqs[i][0]
            c = min(int(rng.choice([1, 2, 3, 17])), len(ids) - at[i])
            entries.append(Entry(i, ids[at[i]:at[i] + c], list(range(c))[::-1]))       # wanted places in any order
            at[i] += c
            if at[i] == len(ids):
                end.append(i)
        got, k = e.step(entries, end), 0
        for en in entries:
            rows[en.id].append(got[k:k + len(en.tokens)].flip(0))
            k += len(en.tokens)
        for i in end:
            live.remove(i)
            if waiting:
                live.append(waiting.pop(0))
    for i, (_, want) in seqs.items():
        assert U.close(torch.cat(rows[i]), want, dtype), i
    # in a reused slot a sequence gives the very bits it gives alone
    fresh, _, _ = load(gpu_ctx, "a", dtype)
    ids = seqs["s"][0]
    assert torch.equal(run(m, ids, [20, 1, 1, 1]), run(fresh, ids, [20, 1, 1, 1]))


def greedy(cfg, w, prompt, n):
    ids, w64 = list(prompt), U.as_f64(w)
    gaps = []
    for _ in range(n):
        lg = F.forward(cfg, w64, ids)[-1]
        top = np.sort(lg)[-2:]
        gaps.append(top[1] - top[0])
        ids.append(int(lg.argmax()))
    return ids[len(prompt):], min(gaps)


def test_greedy_generation_and_long_decoding(gpu_ctx):
    m, cfg, w = load(gpu_ctx, "a", torch.float32, n_slots=2)
    prompts = [U.tokens(cfg, n, 9 + n) for n in (5, 1, 12)]
    got = Engine(m).generate(prompts, 12)
    for p, g in zip(prompts, got):
        want, gap = greedy(cfg, w, p, 12)
        assert gap > 1e-4 and g == want
    assert m.pool.n_free == 2
    # 250 decoded tokens, past every window, then the logits of one more token
    slot = m.open_slot()
    m.extend(slot, torch.tensor(prompts[0], dtype=torch.int32), [])
    m.bind(slot)
    first = int(m.tok[0])
    ids = prompts[0] + [first] + m.generate(250).tolist()
    lg = m.extend(slot, torch.tensor(ids[-1:], dtype=torch.int32), [0])
    assert U.error(lg, F.forward(cfg, U.as_f64(w), ids)[-1:]) < TOL[torch.float32]
    # the captured loop and the eager one agree
    m.close_slot(slot)
    for use_graph in (True, False):
        slot = m.open_slot()
        m.extend(slot, torch.tensor(prompts[2], dtype=torch.int32), [])
        m.bind(slot)
        assert m.generate(11, use_graph=use_graph).tolist() == got[2][1:]
        m.close_slot(slot)


def write_model(d, cfg):
    (d / "config.json").write_text(json.dumps(cfg))
    safetensors.save(d / "model.safetensors", U.weights(cfg))
    return d


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    return write_model(tmp_path_factory.mktemp("model"), U.CFG_B)


def test_registry_loads_the_folder_and_checks_shapes(gpu_ctx, folder, tmp_path):
    m = registry.load_model(gpu_ctx, folder, dtype=torch.float32, max_seq=256)
    ids, want = want_of("b", LEN["b"])
    assert U.error(run(m, ids, [len(ids)]), want) < TOL[torch.float32]
    assert m.decode_bytes_per_token() > 0
    w = U.weights(U.CFG_B)
    w["l1.mix.q"] = w["l1.mix.q"][:-1]
    safetensors.save(tmp_path / "model.safetensors", w)
    (tmp_path / "config.json").write_text(json.dumps(U.CFG_B))
    with pytest.raises(Hf2qError, match="l1.mix.q"):
        registry.load_model(gpu_ctx, tmp_path)


def test_command_line_generates(folder):
    prompt = U.tokens(U.CFG_B, 6, 5)
    r = subprocess.run([sys.executable, "-m", "hf2q_b200", "generate", "--model", str(folder), "--dtype", "float32", "--new", "8", "--max-seq", "64",
                        "--prompt", ",".join(map(str, prompt)), "--prompt", "3"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = [json.loads(x) for x in r.stdout.splitlines()]
    assert got[0] == greedy(U.CFG_B, U.weights(U.CFG_B), prompt, 8)[0] and got[1] == greedy(U.CFG_B, U.weights(U.CFG_B), [3], 8)[0]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_replays_portions(tmp_path, tmp_path_factory, dtype):
    folder = write_model(tmp_path_factory.mktemp("model"), config_of("b", getattr(torch, dtype)))
    ids, want = want_of("b", LEN["b"], dtype=getattr(torch, dtype))
    steps, at = [], 0
    for c in (50, 2, 1, 3, 1, len(ids) - 57):
        steps.append({"step": len(steps), "entries": [{"id": "x", "tokens": ids[at:at + c], "want": list(range(c)) if c != 3 else []}], "end": []})
        at += c
    steps[-1]["end"] = ["x"]
    steps.append({"step": len(steps), "entries": [{"id": "y", "tokens": ids[:9], "want": [8]}], "end": ["y"]})
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "128"],
                       input="".join(json.dumps(s) + "\n" for s in steps), cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {s['step']}" for s in steps]
    assert not (tmp_path / "3.f32").exists()
    at = 0
    for s in steps[:-1]:
        c = len(s["entries"][0]["tokens"])
        if s["entries"][0]["want"]:
            got = np.fromfile(tmp_path / f"{s['step']}.f32", "<f4").reshape(c, -1)
            assert U.close(got.astype(np.float64), want[at:at + c], getattr(torch, dtype))
        at += c
    got = np.fromfile(tmp_path / f"{len(steps) - 1}.f32", "<f4")[None]
    assert U.close(got.astype(np.float64), want[8:9], getattr(torch, dtype))
