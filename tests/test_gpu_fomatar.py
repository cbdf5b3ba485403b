"""The Fomatar decoder through the framework's own entry points against the plain forward pass: prompts, portions,
token-by-token decoding, slots, long decoding, generation, the command line and the trace runner."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import hf2q_b200 as hq
from hf2q_b200 import registry, safetensors
from hf2q_b200.engine import Engine, Entry
from hf2q_b200.fomatar import FomatarConfig, FomatarDecoder
from hf2q_b200.ops import Hf2qError
from oracle import fomatar_forward as F
from tests import fomatar_util as U

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
TOL = {torch.float32: 1e-4}
LEN = {"a": 190, "b": 120, "c": 330}


def load(ctx, name, dtype, seed=0, **kw):
    cfg, w = U.CONFIGS[name], U.weights(U.CONFIGS[name], seed)
    kw.setdefault("max_seq", 1024)
    return FomatarDecoder(ctx, FomatarConfig(cfg), w.__getitem__, dtype=dtype, **kw), cfg, w


_want = {}


def want_of(name, n, seed=1):
    if (name, n, seed) not in _want:
        cfg = U.CONFIGS[name]
        ids = U.tokens(cfg, n, seed)
        _want[name, n, seed] = ids, U.oracle_logits(cfg, U.weights(cfg), ids)
    return _want[name, n, seed]


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
    ids, want = want_of(name, LEN[name])
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
    assert len(got) == len(want) == len(m.runs)
    for r, (a, b) in enumerate(zip(got, want)):
        assert U.close(a, b, dtype), r


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
    for name in w:                                               # keep the memories: weak decay, open forget gates
        if name.endswith(".A_log"):
            w[name] = w[name] - 6.0
        if name.endswith("right.f.b"):
            w[name] = w[name] + 6.0
        if name.endswith("right.i.b"):
            w[name] = w[name] - 2.0
    m = FomatarDecoder(gpu_ctx, FomatarConfig(cfg), w.__getitem__, dtype=torch.float32, max_seq=256)
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
    seqs = {i: want_of("a", n, seed) for i, (n, seed) in {"p": (70, 1), "q": (41, 2), "r": (90, 3), "s": (23, 4)}.items()}
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


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    d = tmp_path_factory.mktemp("model")
    (d / "config.json").write_text(json.dumps(U.CFG_B))
    safetensors.save(d / "model.safetensors", U.weights(U.CFG_B))
    return d


def test_registry_loads_the_folder_and_checks_shapes(gpu_ctx, folder, tmp_path):
    m = registry.load_model(gpu_ctx, folder, dtype=torch.float32, max_seq=256)
    ids, want = want_of("b", LEN["b"])
    assert U.error(run(m, ids, [len(ids)]), want) < TOL[torch.float32]
    assert m.decode_bytes_per_token() > 0
    w = U.weights(U.CFG_B)
    w["l0.mix.left.q"] = w["l0.mix.left.q"][:-1]
    safetensors.save(tmp_path / "model.safetensors", w)
    (tmp_path / "config.json").write_text(json.dumps(U.CFG_B))
    with pytest.raises(Hf2qError, match="left.q"):
        registry.load_model(gpu_ctx, tmp_path)


def test_command_line_generates(folder):
    prompt = U.tokens(U.CFG_B, 6, 5)
    r = subprocess.run([sys.executable, "-m", "hf2q_b200", "generate", "--model", str(folder), "--dtype", "float32", "--new", "8", "--max-seq", "64",
                        "--prompt", ",".join(map(str, prompt)), "--prompt", "3"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    got = [json.loads(x) for x in r.stdout.splitlines()]
    assert got[0] == greedy(U.CFG_B, U.weights(U.CFG_B), prompt, 8)[0] and got[1] == greedy(U.CFG_B, U.weights(U.CFG_B), [3], 8)[0]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_replays_portions(folder, tmp_path, dtype):
    ids, want = want_of("b", LEN["b"])
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


def test_llama_through_the_same_registry_and_engine(gpu_ctx, tmp_path):
    """A GGUF file of the quantized decoder loads by its architecture key and runs in portions through the engine."""
    import oracle
    from hf2q_b200 import gguf
    from tests.util import make_quant_weight
    hidden, n_q, n_kv, hd, ffn, vocab = 2048, 16, 4, 128, 6144, 512
    g = gguf.GgufWriter()
    g.add_kv("general.architecture", gguf.T_STRING, "llama")
    for k, v in {"block_count": 1, "embedding_length": hidden, "attention.head_count": n_q, "attention.head_count_kv": n_kv, "feed_forward_length": ffn}.items():
        g.add_kv("llama." + k, gguf.T_U32, v)
    g.add_kv("llama.attention.layer_norm_rms_epsilon", gguf.T_F32, 1e-5)
    g.add_kv("llama.rope.freq_base", gguf.T_F32, 10000.0)
    rng = np.random.default_rng(0)

    def q(name, n, k, t=12):
        g.add_tensor(name, (n, k), t, make_quant_weight(t, n, k, seed=len(name) + n))
    q("token_embd.weight", vocab, hidden)
    q("output.weight", vocab, hidden, 14)
    for name, n, k, t in (("attn_q", n_q * hd, hidden, 12), ("attn_k", n_kv * hd, hidden, 12), ("attn_v", n_kv * hd, hidden, 14), ("attn_output", hidden, n_q * hd, 12),
                          ("ffn_gate", ffn, hidden, 12), ("ffn_up", ffn, hidden, 12), ("ffn_down", hidden, ffn, 14)):
        q(f"blk.0.{name}.weight", n, k, t)
    for name in ("blk.0.attn_norm.weight", "blk.0.ffn_norm.weight", "output_norm.weight"):
        g.add_tensor(name, (hidden,), 0, (1 + 0.1 * rng.standard_normal(hidden)).astype(np.float32))
    g.write(tmp_path / "m.gguf")
    m = registry.load_model(gpu_ctx, tmp_path / "m.gguf", max_seq=256)
    ids = rng.integers(0, vocab, 80).tolist()
    whole = Engine(m).step([Entry("a", ids, [10, 39, 79])], end=["a"])
    e = Engine(m)
    parts = [e.step([Entry("b", ids[:40], [10, 39])]), e.step([Entry("b", ids[40:], [39])], end=["b"])]
    assert U.error(torch.cat(parts), whole.double().cpu().numpy()) < 2e-2
    first = int(whole[2].argmax())
    got = Engine(m).generate([ids], 4)[0]
    assert got[0] == first and len(got) == 4
    with pytest.raises(Hf2qError):
        registry.load_model(gpu_ctx, tmp_path / "m.gguf", dtype=torch.float32)
