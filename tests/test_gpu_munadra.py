"""The Munadra model on the GPU through the framework's own parts -- registry, cache manager, Engine, command line --
against the plain restatement: whole prompts, portions, decoding, batches, slots and pages that are used again."""
import io
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from latent_helpers import as_dtype, dense, latent, moe, quiet_experts, random_model, rglru, rms, small_config
from oracle import munadra as plain

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent


@pytest.fixture(scope="module")
def case():
    raw = small_config()
    return raw, quiet_experts(random_model(raw, 7))


def _tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed))


def _model(case, device, dtype):
    from kinetics_b200 import Munadra
    raw, W = case
    return Munadra(Munadra.from_config(raw), W, device, dtype)


def _engine(model, slots=4, max_len=256, num_pages=None, page_size=16, **kw):
    from kinetics_b200 import Engine
    kv = model.new_cache(slots, max_len, num_pages, page_size)
    return Engine(model, kv, max_len, model.device, temperature=0.0, eos=[], repeat_check=False, **kw)


def _run(engine, slot, tokens, sizes):
    engine.open_slot(slot)
    out, at = [], 0
    for n in sizes:
        out.append(engine.extend(slot, tokens[at:at + n].tolist(), list(range(n))).cpu())
        at += n
    assert at == tokens.numel()
    engine.kv.check_status()
    engine.model.check_status()
    return torch.cat(out)


def _agree(got, want, dtype, median=3e-2):
    err = (got.double() - want.double()).pow(2).mean(-1).sqrt() / rms(want)
    if dtype == torch.float32:
        assert err.max() < 2e-4, float(err.max())
    else:
        # a router decision may fall either way where two logits are close: rare rows, not all
        assert err.median() < median and (err > 0.15).double().mean() < 0.1, (float(err.median()), float(err.max()))


DTYPES = [torch.float32, torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
def test_prompt_portions_and_decoding_match_the_restatement(cuda_device, case, dtype):
    raw, W = case
    tokens = _tokens(150, raw["vocab"], 1)
    want = plain.forward(tokens, as_dtype(W, torch.float64), raw)
    model = _model(case, cuda_device, dtype)
    for page_size in (16, 64):
        engine = _engine(model, page_size=page_size)
        for sizes in ([150], [1] * 150, [2] * 75, [16, 64, 2, 1, 3, 63, 1], [100] + [1] * 50, [129, 2, 2, 17]):
            _agree(_run(engine, 2, tokens, sizes), want, dtype)
            engine.clear_request(2)
        assert engine.kv.pool.free_pages == engine.kv._num_pool_pages


@pytest.mark.parametrize("dtype", DTYPES)
def test_stream_behind_every_layer(cuda_device, case, dtype):
    raw, W = case
    tokens = _tokens(33, raw["vocab"], 2)
    want, got = [], []
    plain.forward(tokens, as_dtype(W, torch.float64), raw, streams=want)
    model = _model(case, cuda_device, dtype)
    kv = model.new_cache(1, 64)
    kv.admit(0, 33, 64)
    model._hidden(tokens[None].to(cuda_device), torch.tensor([0], device=cuda_device), kv, streams=got)
    for a, b in zip(got, want):
        _agree(a.cpu(), b, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_one_token_alone(cuda_device, case, dtype):
    raw, W = case
    want = plain.forward(torch.tensor([5]), as_dtype(W, torch.float64), raw)
    model = _model(case, cuda_device, dtype)
    _agree(_run(_engine(model), 0, torch.tensor([5]), [1]), want, dtype)


def test_other_sizes(cuda_device):
    # sizes that small_config has equal or round: one head, many heads, a rank wider than the stream, single experts, top =
    # all, one tap, one block, a width that is no multiple of 8, unrotated parts of one column
    raw = small_config([
        rglru(33, 3, 1, dense(9)),
        latent(1, 1, 2, 3, 260, moe(1, 1, 8), scale=1.0, base=7.0),
        latent(70, 8, 4, 5, 24, dense(40), factor=1.25, original=9, fast=3.0, slow=0.2),
        latent(6, 128, 64, 128, 512, moe(9, 9, 72, limit=0.25), kv_from=None, factor=40.0, original=30, fast=32.0, slow=1.0),
        rglru(200, 5, 6, None),
        latent(4, 16, 4, 130, 24, moe(33, 2, 31), kv_from=2, factor=1.25, original=9, fast=3.0, slow=0.2),
        rglru(16, 2, 4, moe(4, 3, 16)),
    ], vocab=333, width=203, eps=1e-3, embed_scale=0.5, logit_scale=1.0, softcap=30.0)
    tokens = _tokens(90, 333, 3)
    for dtype in DTYPES:
        W = quiet_experts(random_model(raw, 4, boost=1.5)) if dtype == torch.bfloat16 else random_model(raw, 4)
        want = plain.forward(tokens, as_dtype(W, torch.float64), raw)
        engine = _engine(_model((raw, W), cuda_device, dtype), page_size=32)
        for sizes in ([90], [40, 2, 30] + [1] * 18, [65, 25]):
            _agree(_run(engine, 0, tokens, sizes), want, dtype, median=5e-2)      # seven layers
            engine.clear_request(0)


def test_layers_of_one_kind_only(cuda_device):
    # no pages at all, and nothing but pages
    for layers in ([rglru(40, 2, 4, dense(32)), rglru(24, 1, 3, None)], [latent(2, 8, 8, 8, 16, dense(24), factor=2.0)]):
        raw = small_config(layers, vocab=50, width=40)
        W = random_model(raw, 5)
        tokens = _tokens(60, 50, 6)
        want = plain.forward(tokens, as_dtype(W, torch.float64), raw)
        for dtype in DTYPES:
            engine = _engine(_model((raw, W), cuda_device, dtype))
            _agree(_run(engine, 1, tokens, [30, 2] + [1] * 28), want, dtype)


def test_greedy_generation_through_the_engine(cuda_device, case):
    # fp32: the tokens of the restatement, for unequal requests that share slots and a pool too small for all
    raw, W = case
    W64 = as_dtype(W, torch.float64)
    prompts = [_tokens(n, raw["vocab"], 20 + n).tolist() for n in (40, 9, 77, 3, 1, 64, 23)]
    new = 12
    want = {}
    for i, p in enumerate(prompts):
        hist = plain.History(len(raw["layers"]))
        logits, out = plain.forward(torch.tensor(p), W64, raw, hist), []
        for _ in range(new):
            out.append(int(logits[-1].argmax()))
            logits = plain.forward(torch.tensor(out[-1:]), W64, raw, hist)
        want[i] = out
    model = _model(case, cuda_device, torch.float32)
    for kw in (dict(), dict(prefill_chunk=16), dict(slots=2, num_pages=8)):
        engine = _engine(model, **{**dict(slots=3, max_len=128), **kw})
        done = engine.offline_exec([{"id": i, "input_ids": p} for i, p in enumerate(prompts)], max_new_tokens=new)
        got = {r["id"]: r["output_tokens"] for r in done}
        # a sequence's last sampled token is not part of its output
        assert got == {i: w[:new - 1] for i, w in want.items()}
        assert engine.kv.pool.free_pages == engine.kv._num_pool_pages
        engine.kv.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_decoding_equals_each_request_alone(cuda_device, case, dtype):
    raw, _ = case
    model = _model(case, cuda_device, dtype)
    lens = (70, 3, 1, 129, 64)
    engine = _engine(model, slots=5, max_len=200)
    alone = _engine(model, slots=1, max_len=200)
    steps = 20
    for slot, n in enumerate(lens):
        engine.prefill(slot, _tokens(n, raw["vocab"], slot)[None], steps + 1)
    for _ in range(steps):
        engine.decode([4, 0, 2, 1, 3])
    for slot, n in enumerate(lens):
        seq = engine.slots_tokens[slot, :n + steps + 1].cpu()
        logits = _run(alone, 0, seq[:-1], [n + steps])     # the sequence that was generated, as one prompt
        alone.clear_request(0)
        best, pick = logits.max(-1).values, logits[torch.arange(n + steps), seq[1:]]
        # every generated token is the best one up to rounding
        gap = (best - pick)[n - 1:] / rms(logits)
        assert gap.max() < (1e-3 if dtype == torch.float32 else 0.5)
        assert (gap < 0.05).double().mean() > 0.85


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_and_pages_are_used_again(cuda_device, case, dtype):
    # a pool of ten pages serves sequence after sequence; neighbours keep running meanwhile
    raw, W = case
    W64 = as_dtype(W, torch.float64)
    model = _model(case, cuda_device, dtype)
    engine = _engine(model, slots=3, max_len=120, num_pages=10)
    long = _tokens(60, raw["vocab"], 50)
    engine.open_slot(1)
    outs, at = [], 0
    for round_ in range(4):
        outs.append(engine.extend(1, long[at:at + 15].tolist(), list(range(15))).cpu())
        at += 15
        slot = (0, 2)[round_ % 2]
        tokens = _tokens(50 + round_, raw["vocab"], 60 + round_)
        got = _run(engine, slot, tokens, [20, 2, 28 + round_])
        _agree(got, plain.forward(tokens, W64, raw), dtype)
        engine.clear_request(slot)
    _agree(torch.cat(outs), plain.forward(long, W64, raw), dtype)
    engine.clear_request(1)
    assert engine.kv.pool.free_pages == 10


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(cuda_device, case, dtype):
    raw, W = case
    tokens = _tokens(400, raw["vocab"], 70)
    want = plain.forward(tokens, as_dtype(W, torch.float64), raw)
    engine = _engine(_model(case, cuda_device, dtype), max_len=512, page_size=64)
    _agree(_run(engine, 3, tokens, [37] + [1] * 363), want, dtype)


def test_graphed_decode_equals_the_eager_step(cuda_device, case):
    raw, _ = case
    model = _model(case, cuda_device, torch.bfloat16)
    lens = (150, 37, 3, 96)

    def make():
        e = _engine(model, slots=4, max_len=256)
        for slot, n in enumerate(lens):
            e.prefill(slot, _tokens(n, raw["vocab"], slot)[None], 40)
        return e

    eager, graphed = make(), make()
    for step in range(24):
        eager.decode([0, 1, 2, 3])
        graphed.decode_graphed([0, 1, 2, 3])
        torch.cuda.synchronize()
        assert torch.equal(eager.slots_tokens, graphed.slots_tokens), step
    graphed.kv.check_status()
    assert graphed.kv.pool.free_pages == eager.kv.pool.free_pages


def _folder(tmp_path, case):
    from kinetics_b200.checkpoint import save
    raw, W = case
    (tmp_path / "m").mkdir()
    (tmp_path / "m" / "config.json").write_text(json.dumps(raw))
    save(tmp_path / "m" / "model.safetensors", W)
    return tmp_path / "m"


def test_generate_command(cuda_device, case, tmp_path):
    from kinetics_b200 import cli
    raw, W = case
    path = _folder(tmp_path, case)
    args = cli._parse(["generate", "--model", str(path), "--dtype", "float32", "--prompt", "5,17,3", "--prompt", "8",
                       "--max-new-tokens", "6"])
    out = io.StringIO()
    assert cli.generate(args, out) == 0
    lines = [json.loads(x) for x in out.getvalue().splitlines()]
    assert [x["id"] for x in lines] == [0, 1]
    hist = plain.History(len(raw["layers"]))
    W64 = as_dtype(W, torch.float64)
    logits = plain.forward(torch.tensor([5, 17, 3]), W64, raw, hist)
    for t in lines[0]["output_tokens"]:
        assert t == int(logits[-1].argmax())
        logits = plain.forward(torch.tensor([t]), W64, raw, hist)
    args = cli._parse(["generate", "--model", str(path), "--prompt", "1,2", "--temperature", "0.8", "--top-k", "5",
                       "--top-p", "0.9", "--seed", "3", "--max-new-tokens", "4"])
    assert cli.generate(args, io.StringIO()) == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner(cuda_device, case, tmp_path, dtype):
    raw, W = case
    path = _folder(tmp_path, case)
    out = tmp_path / "out"
    out.mkdir()
    a, b = _tokens(60, raw["vocab"], 80), _tokens(9, raw["vocab"], 81)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:41].tolist(), "want": [0, 40]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[41:42].tolist(), "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b.tolist(), "want": [8, 3]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[42:44].tolist(), "want": []}], "end": []},
             {"step": 4, "entries": [{"id": "a", "tokens": a[44:].tolist(), "want": list(range(16))}], "end": ["a"]}]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(path), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "69"], input="\n".join(json.dumps(s) for s in steps) + "\n", text=True,
                       capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    read = lambda i: torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, raw["vocab"]).copy())
    assert not (out / "3.f32").exists()
    W64, dt = as_dtype(W, torch.float64), torch.float32 if dtype == "float32" else torch.bfloat16
    wa, wb = plain.forward(a, W64, raw), plain.forward(b, W64, raw)
    got = torch.cat((read(0), read(1), read(2), read(4)))
    _agree(got, torch.cat((wa[[0, 40, 41]], wb[[8, 3]], wa[44:])), dt)
