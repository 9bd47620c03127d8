"""The Lizazen family through the engine: checkpoints written to disk and loaded by the model directory, schedules replayed
through the scheduler, the pools and the state slots, compared with the plain oracle over whole sequences.  Covers prefill
against token-by-token decoding, portions down to two tokens, unequal batches against each request alone, pages and slots that
are freed and used again, long decoding that carries every window and chunk far from the first tokens, the residual after
every layer, prompt steps large enough for the grouped expert products, loud weights, greedy generation through
LLMEngine.generate, the server and the trace replay program."""
import json
import os
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import lizazen_ref as R
import lizazen_util as U

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, make in U.CONFIGS.items():
        cfg = make()
        W = R.random_model(cfg, seed=ord(name))
        out[name] = (cfg, W, U.save_checkpoint(tmp_path_factory.mktemp("lizazen_" + name), cfg, W))
    return out


_oracle_cache = {}


def _oracle(cfg, W, toks):
    key = (id(W), tuple(toks))
    if key not in _oracle_cache:
        _oracle_cache[key] = W, U.oracle_logits(cfg, W, toks)      # W stays alive: its id names the entry
    return _oracle_cache[key][1]


def _check(got, cfg, W, reqs, dtype, what=""):
    for rid, toks in reqs.items():
        err = U.rel_err(got[rid], _oracle(cfg, W, toks), dtype)
        assert err <= U.TOL[dtype], f"{what} request {rid}: error {err:.3e} above {U.TOL[dtype]:.1e} ({dtype})"


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompt_and_token_by_token(cuda, models, name, dtype):
    cfg, W, path = models[name]
    eng = U.make_engine(path, dtype)
    reqs = {"p": U.tokens(70, cfg["vocab"], 1), "q": U.tokens(1, cfg["vocab"], 2)}
    whole = U.replay(eng, reqs, [[("p", 70)], [("q", 1)]])
    _check(whole, cfg, W, reqs, dtype, "whole")
    single = U.replay(eng, {"p": reqs["p"]}, [[("p", 1)] for _ in range(70)])          # every token a step of its own
    _check(single, cfg, W, {"p": reqs["p"]}, dtype, "token by token")
    assert U.rel_err(single["p"], whole["p"], dtype) <= U.TOL[dtype]
    eng.close()


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_residual_after_every_layer(cuda, models, name):
    cfg, W, path = models[name]
    eng = U.make_engine(path, "float32", eager=True)
    toks = U.tokens(29, cfg["vocab"], 3)
    eng.model.capture = []
    eng.replay_step([("r", toks, [])], ["r"])
    trail = []
    R.forward(cfg, W, toks, trail)
    assert len(eng.model.capture) == len(cfg["layers"])
    for i, x in enumerate(eng.model.capture):
        assert x.dtype == torch.float32
        err = float((x.double().cpu() - trail[i]).abs().max() / trail[i].abs().max())
        assert err <= 2e-5, f"layer {i}: {err:.3e}"
    eng.close()


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
def test_portions_of_many_sizes(cuda, models, name):
    """Cuts inside pages (16) and inside and at the edges of the windows, portions of 2 and 3."""
    cfg, W, path = models[name]
    eng = U.make_engine(path, "float32")
    toks = U.tokens(131, cfg["vocab"], 7)
    for cuts in ([2, 3, 11, 17, 31, 2, 33, 30, 2], [64, 2, 2, 63], [15, 1, 1, 16, 32, 1, 65], [6, 1, 13, 43, 1, 67]):
        assert sum(cuts) == 131
        got = U.replay(eng, {"r": toks}, [[("r", n)] for n in cuts])
        _check(got, cfg, W, {"r": toks}, "float32", f"cuts {cuts}")
    eng.close()


@pytest.mark.parametrize("name", sorted(U.CONFIGS))
@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batches_with_reuse_of_pages_and_slots(cuda, models, name, dtype):
    """Up to four live requests, prompt portions beside single tokens; requests leave and new ones take over their pages
    (a pool of 15 pages for ~320 tokens in total).  Every request equals the oracle over its own tokens, and itself alone."""
    cfg, W, path = models[name]
    V = cfg["vocab"]
    reqs = {"a": U.tokens(90, V, 1), "b": U.tokens(33, V, 2), "c": U.tokens(1, V, 3), "d": U.tokens(47, V, 4),
            "e": U.tokens(60, V, 5), "f": U.tokens(52, V, 6), "g": U.tokens(40, V, 7)}
    sched = [[("a", 30), ("b", 31), ("c", 1)],                       # c lives for one step
             [("a", 1), ("b", 1), ("d", 17)],
             [("a", 1), ("b", 1), ("d", 2), ("e", 3)],               # b ends: its pages go back
             [("a", 28), ("d", 1), ("e", 1), ("f", 20)],
             [("a", 1), ("d", 27), ("e", 40), ("f", 1)],             # d ends
             [("a", 29), ("e", 16), ("f", 31), ("g", 2)],            # a, e, f end
             [("g", 1)], [("g", 1)], [("g", 36)]]
    eng = U.make_engine(path, dtype, max_tokens=15 * 16)
    got = U.replay(eng, reqs, sched)
    assert eng.sched.num_free_blocks == eng.num_blocks and eng.sched.num_running == 0
    _check(got, cfg, W, reqs, dtype, "mixed")
    for rid, toks in reqs.items():
        alone = U.replay(eng, {rid: toks}, [[(rid, len(toks))]])
        assert U.rel_err(got[rid], alone[rid], dtype) <= (1e-5 if dtype == "float32" else 2e-2), f"request {rid} against itself alone"
    eng.close()


@pytest.mark.parametrize("name,eager", [("a", False), ("a", True), ("c", False), ("e", False)])
def test_long_decoding_through_graph_and_eager_steps(cuda, models, name, eager):
    """A 20-token prompt then 230 single-token steps (the decode-only step is a CUDA graph unless eager), beside a second
    request that joins late."""
    cfg, W, path = models[name]
    reqs = {"x": U.tokens(250, cfg["vocab"], 21), "y": U.tokens(120, cfg["vocab"], 22)}
    sched = [[("x", 20)]] + [[("x", 1)] for _ in range(110)] + [[("x", 1), ("y", 1)] for _ in range(120)]
    eng = U.make_engine(path, "float32", eager=eager)
    got = U.replay(eng, reqs, sched)
    _check(got, cfg, W, reqs, "float32", "long decode")
    assert eng.stats.decode_steps >= 229 and (eager or len(eng._graphs) >= 2)
    eng.close()


@pytest.mark.parametrize("name", ["e", "f"])
def test_large_prompt_steps(cuda, models, name):
    """bf16 steps with so many (token, choice) pairs that routing and experts run as library products: alone, beside decode rows, and
    behind a context.  The logits equal the oracle's and those of the same requests cut into small portions."""
    from b200attn import ops
    cfg, W, path = models[name]
    V = cfg["vocab"]
    top = max(L["mlp"]["router"]["top"] for L in cfg["layers"] if L["mlp"] and L["mlp"]["kind"] == "moe")
    n = ops.MOE_GROUPED_GEMM_MIN_PAIRS // top + 40
    reqs = {"a": U.tokens(n + 60, V, 41), "b": U.tokens(n + 7, V, 42), "c": U.tokens(30, V, 43)}
    eng = U.make_engine(path, "bfloat16", max_tokens=4 * n)
    got = U.replay(eng, reqs, [[("a", 50), ("c", 20)], [("a", 1), ("b", n), ("c", 1)], [("a", n), ("b", 1), ("c", 9)], [("a", 9), ("b", 6)]])
    small = U.replay(eng, reqs, [[("a", 60)]] + [[("a", min(100, n - i))] for i in range(0, n, 100)]
                     + [[("b", 7)]] + [[("b", min(100, n - i))] for i in range(0, n, 100)] + [[("c", 30)]])
    _check({"c": got["c"]}, cfg, W, {"c": reqs["c"]}, "bfloat16", "large steps")
    for rid in ("a", "b"):
        want = R.forward(cfg, W, reqs[rid][:150])
        assert U.rel_err(got[rid][:150], want, "bfloat16") <= U.TOL["bfloat16"], f"request {rid}"
    for rid in reqs:
        assert U.rel_err(got[rid], small[rid], "bfloat16") <= 3e-2, f"request {rid}: large against small steps"
    eng.close()


LOUD = [("l0.mix.sink", 3.0, 2.0), ("l0.mix.q.norm", 0.0, 3.0), ("l0.mix.k.norm", 0.0, 3.0), ("l0.mix.q.b", 1.0, 2.0), ("l0.mix.k.b", 1.0, 2.0),
        ("l0.mix.o.b", 1.0, 3.0), ("l1.mix.lq1", 0.2, 2.0), ("l1.mix.lk2", 0.2, 2.0), ("l2.mix.left.v.b", 1.0, 3.0), ("l2.mix.left.o.b", 1.0, 3.0),
        ("l2.mix.left.out", 0.0, 3.0), ("l2.mix.right.out", 0.0, 3.0), ("l0.norm1b", 0.0, 3.0), ("l1.norm2b", 0.0, 3.0), ("bigram", 0.0, 3.0),
        ("l0.mlp.router", 0.0, 0.2)]


@pytest.mark.parametrize("name,add,times", LOUD)
def test_every_small_tensor_shows_in_the_logits(cuda, models, tmp_path, name, add, times):
    """Small tensors made loud: the engine follows the oracle there too, and the logits differ from the plain model's."""
    cfg, W, _ = models["e"]
    W2 = dict(W)
    W2[name] = (W[name].float() * times + add).to(torch.bfloat16)
    toks = U.tokens(66, cfg["vocab"], 13)
    eng = U.make_engine(U.save_checkpoint(tmp_path / "m", cfg, W2), "float32")
    got = U.replay(eng, {"r": toks}, [[("r", 60)], [("r", 2)]] + [[("r", 1)]] * 4)
    eng.close()
    _check(got, cfg, W2, {"r": toks}, "float32", name)
    assert U.rel_err(_oracle(cfg, W2, toks), _oracle(cfg, W, toks)) > 20 * U.TOL["float32"]


def test_a_slot_keeps_nothing_of_its_last_sequence(cuda, models):
    """One state slot serves a loud sequence and then another: the second equals itself in a fresh engine to the bit, decoded and
    in portions (the token before, the matrix state, the pages)."""
    cfg, W, path = models["a"]
    V = cfg["vocab"]
    first, second = U.tokens(70, V, 3), U.tokens(60, V, 4)
    cuts = [[("s", 1)], [("s", 30)], [("s", 2)]] + [[("s", 1)]] * 27
    eng = U.make_engine(path, "float32", max_num_seqs=1, max_tokens=80)
    U.replay(eng, {"f": first}, [[("f", 40)]] + [[("f", 1)]] * 30)
    used = U.replay(eng, {"s": second}, cuts)["s"]
    eng.close()
    eng = U.make_engine(path, "float32", max_num_seqs=1, max_tokens=80)
    fresh = U.replay(eng, {"s": second}, cuts)["s"]
    eng.close()
    assert torch.equal(used, fresh)
    _check({"s": used}, cfg, W, {"s": second}, "float32", "used slot")


def test_block_size_and_pool_do_not_change_the_logits(cuda, models):
    cfg, W, path = models["c"]
    toks = U.tokens(77, cfg["vocab"], 9)
    ref = None
    for bs in (8, 16, 32):
        eng = U.make_engine(path, "float32", max_tokens=96, block_size=bs)
        got = U.replay(eng, {"r": toks}, [[("r", 50)], [("r", 2)], [("r", 25)]])["r"]
        _check({"r": got}, cfg, W, {"r": toks}, "float32", f"block size {bs}")
        ref = got if ref is None else ref
        assert U.rel_err(got, ref) <= 1e-5
        eng.close()


@pytest.mark.parametrize("name", ["a", "d"])
def test_greedy_generation_through_the_engine(cuda, models, name):
    """LLMEngine.generate (scheduler policy, chunked prefill, CUDA-graph decode, b2_sample at temperature 0) continues
    three prompts exactly as the oracle's argmax does, with fewer sequence slots than requests."""
    from b200attn.engine import SamplingParams
    cfg, W, path = models[name]
    eng = U.make_engine(path, "float32", max_num_seqs=2)
    prompts = [U.tokens(n, cfg["vocab"], 30 + n) for n in (5, 19, 1)]
    outs = eng.generate(prompts, SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True))
    compared = 0
    for p, out in zip(prompts, outs):
        seq = list(p)
        for k in range(12):
            lg = U.oracle_logits(cfg, W, seq)[-1]
            top2 = torch.topk(lg, 2).values
            if float(top2[0] - top2[1]) < 1e-2 * float(lg.abs().max()):
                break                                               # a near tie for a sampler that reads the logits in 16 bits
            assert out[k] == int(lg.argmax()), f"token {k} of prompt of {len(p)}"
            seq.append(out[k])
            compared += 1
    assert compared >= 6
    eng.close()


def test_random_init_and_checkpoint_shape_check(cuda, tmp_path, models):
    """Without weights in the directory the engine serves seeded random weights of the configuration; a checkpoint
    whose shapes contradict config.json, or that lacks a tensor, is refused."""
    cfg, W, _ = models["b"]
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    eng = U.make_engine(tmp_path, "bfloat16")
    lg = eng.replay_step([("r", U.tokens(9, cfg["vocab"], 1), [8])], ["r"])
    assert lg.shape == (1, cfg["vocab"]) and bool(torch.isfinite(lg).all())
    eng.close()
    bad = dict(W)
    bad["l1.mix.sink"] = torch.zeros(5, dtype=torch.bfloat16)
    U.save_checkpoint(tmp_path / "bad", cfg, bad)
    with pytest.raises(ValueError, match="sink"):
        U.make_engine(tmp_path / "bad", "bfloat16")
    U.save_checkpoint(tmp_path / "less", cfg, {k: v for k, v in W.items() if k != "l0.mix.lq2"})
    with pytest.raises(ValueError, match="lacks"):
        U.make_engine(tmp_path / "less", "bfloat16")


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_program(cuda, models, tmp_path, dtype):
    """bin/trace_run as a subprocess: steps on standard input, one `done` line per step, logits files for the wanted rows."""
    cfg, W, path = models["d"]
    root = Path(__file__).resolve().parent.parent
    a, b = U.tokens(40, cfg["vocab"], 11), U.tokens(9, cfg["vocab"], 12)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:33], "want": [0, 32]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[33:34], "want": [0]}, {"id": "b", "tokens": b, "want": [8]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[34:], "want": []}], "end": ["a"]}]
    out = tmp_path / "out"
    out.mkdir()
    env = {k: v for k, v in os.environ.items() if k != "B200ATTN_LIB"}
    r = subprocess.run([sys.executable, str(root / "bin" / "trace_run"), "--model", str(path), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True,
                       text=True, env=env, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not (out / "2.f32").exists()
    la, lb = U.oracle_logits(cfg, W, a), U.oracle_logits(cfg, W, b)
    got0 = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(2, -1))
    got1 = torch.from_numpy(np.fromfile(out / "1.f32", dtype="<f4").reshape(2, -1))
    tol = U.TOL[dtype] * (1 if dtype == "float32" else 3)
    assert U.rel_err(got0, la[[0, 32]]) <= tol and U.rel_err(got1, torch.stack([la[33], lb[8]])) <= tol


def test_server_serves_a_model_directory(cuda, models):
    """`python -m b200attn.server --model DIR --dtype float32`: the family comes from config.json, completions are the
    oracle's greedy continuation of a token-id prompt."""
    import socket
    import time

    import requests
    cfg, W, path = models["b"]
    sock = socket.socket()
    sock.bind(("127.0.0.1", 0))
    port = sock.getsockname()[1]
    sock.close()
    root = Path(__file__).resolve().parent.parent
    env = dict(os.environ, PYTHONPATH=str(root / "vllm-backend-public_b200"))
    proc = subprocess.Popen([sys.executable, "-m", "b200attn.server", "--model", str(path), "--dtype", "float32", "--port", str(port),
                             "--host", "127.0.0.1", "--max-num-seqs", "4", "--max-model-len", "256",
                             "--num-gpu-blocks-override", "80", "--served-model-name", "lizazen-test"], env=env,
                            stdout=subprocess.PIPE, stderr=subprocess.STDOUT)
    base = f"http://127.0.0.1:{port}"
    try:
        for _ in range(600):
            if proc.poll() is not None:
                raise RuntimeError("server exited: " + proc.stdout.read().decode()[-2000:])
            try:
                if requests.get(base + "/health", timeout=1).status_code == 200:
                    break
            except requests.RequestException:
                pass
            time.sleep(0.2)
        else:
            raise RuntimeError("server did not become healthy")
        body = None
        for seed in range(80, 100):                                 # a prompt whose six greedy steps all have a clear winner
            prompt = U.tokens(11, cfg["vocab"], seed)
            seq, clear = list(prompt), True
            for _ in range(6):
                lg = U.oracle_logits(cfg, W, seq)[-1]
                top2 = torch.topk(lg, 2).values
                clear = clear and float(top2[0] - top2[1]) > 1e-2 * float(lg.abs().max())
                seq.append(int(lg.argmax()))
            if not clear:
                continue
            r = requests.post(base + "/v1/completions", json={"model": "lizazen-test", "prompt": prompt, "max_tokens": 6,
                                                              "temperature": 0.0, "ignore_eos": True}, timeout=60)
            assert r.status_code == 200, r.text
            body = r.json()
            assert body["usage"]["prompt_tokens"] == 11 and body["usage"]["completion_tokens"] == 6
            want = bytes(t % 256 for t in seq[11:]).decode("utf-8", errors="replace")      # the byte tokenizer's text
            assert body["choices"][0]["text"] == want
            break
        assert body is not None
    finally:
        proc.terminate()
        try:
            proc.wait(20)
        except subprocess.TimeoutExpired:
            proc.kill()
