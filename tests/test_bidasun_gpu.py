"""GPU tests of the Bidasun design through the framework's engine, scheduler and command line, against the
plain implementation in oracle/bidasun_ref.py (float64, whole sequences, no cache)."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import bidasun_cases as cases
from oracle import bidasun_ref as ref
from tensorwarp_b200 import _dense, dense, registry
from tensorwarp_b200.engine import DenseEngine
from tensorwarp_b200.models import bidasun
from tensorwarp_b200.scheduler import Scheduler
from tensorwarp_b200.state import StateError

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 2e-5, torch.bfloat16: 4e-2}
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
CASE = pytest.mark.parametrize("case", sorted(cases.CASES))

_oracle_cache = {}


def oracle(case, n, seed):
    """Logits and residual stream after every layer of `n` seeded tokens."""
    key = (case, n, seed)
    if key not in _oracle_cache:
        cfg = cases.CASES[case]
        layers = []
        toks = cases.tokens(cfg, n, seed)
        logits = ref.forward(cfg, cases.as_float64(cases.weights(cfg, 7)), toks, layers)
        _oracle_cache[key] = (toks, logits, layers)
    return _oracle_cache[key]


def engine(case, dtype, **options):
    cfg = cases.CASES[case]
    spec, t = bidasun.parse_config(cfg), cases.weights(cfg, 7)
    return DenseEngine(dense.DenseModel(spec, bidasun.model_tensors(spec, lambda n, s: t[n]), dtype), **options)


def close(got, want, dtype):
    err = cases.error(got.cpu().numpy() if torch.is_tensor(got) else got, want)
    assert err.max() < TOL[dtype], (int(err.argmax()), float(err.max()))
    assert _dense.device_error() == 0


@BOTH
@CASE
def test_whole_prompt_and_every_layer(case, dtype):
    n = 200
    toks, logits, layers = oracle(case, n, 1)
    eng = engine(case, dtype)
    seq, got = eng.open(), []
    out = eng.step(seq, toks, list(range(n)), layer_trace=got)
    close(out, logits, dtype)
    assert len(got) == 1 and got[0].shape == (len(layers), n, cases.CASES[case]["width"])
    for g, want in zip(got[0].cpu().numpy(), layers):
        assert np.sqrt(((g - want) ** 2).mean()) < TOL[dtype] * want.std()


@BOTH
@CASE
def test_token_by_token(case, dtype):
    """Decoding from the first token on: every window's edge, the first kept keys and tile borders pass by."""
    n = 200
    toks, logits, _ = oracle(case, n, 1)
    eng = engine(case, dtype)
    seq = eng.open()
    rows = [eng.step(seq, [t], [0]).clone() for t in toks]
    close(torch.cat(rows), logits, dtype)


@BOTH
@CASE
@pytest.mark.parametrize("portion", [2, 3, 7, 63, 64, 65, 129])
def test_portions(case, dtype, portion):
    n = 200
    toks, logits, _ = oracle(case, n, 1)
    eng = engine(case, dtype)
    seq, rows = eng.open(), []
    for at in range(0, n, portion):
        part = toks[at:at + portion]
        rows.append(eng.step(seq, part, list(range(len(part)))).clone())
    close(torch.cat(rows), logits, dtype)


@BOTH
def test_portions_of_changing_size_with_decoding_between(dtype):
    n = 250
    toks, logits, _ = oracle("tiles", n, 2)
    eng = engine("tiles", dtype)
    seq, at, want = eng.open(), 0, []
    got = []
    for k, size in enumerate([1, 2, 1, 5, 60, 1, 1, 62, 2, 3, 1, 64, 1, 1, 40, 5]):
        pick = [size - 1] if k % 3 else []
        out = eng.step(seq, toks[at:at + size], pick)
        assert (out is None) == (not pick)
        if pick:
            got.append(out.clone())
            want.append(at + size - 1)
        at += size
    assert at == n
    close(torch.cat(got), logits[want], dtype)


@BOTH
def test_more_tokens_and_wanted_rows_than_the_buffers_take(dtype):
    """A step that has to be cut inside the engine, by its tokens and by its wanted rows."""
    n = 200
    toks, logits, _ = oracle("tiles", n, 1)
    eng = engine("tiles", dtype, portion=48)
    assert eng.max_rows == 48
    eng.max_want = 11
    want = [0, 1, 2, 3, 10, 11, 12, 13, 14, 15, 16, 17, 40, 47, 48, 49, 95, 96, 97] + list(range(150, 200))
    out = eng.step(eng.open(), toks, want)
    close(out, logits[want], dtype)


@BOTH
def test_slots_used_again_and_sequences_interleaved(dtype):
    """Several sequences in flight, slots freed and taken by others of other lengths: each as if alone."""
    eng = engine("uneven", dtype, max_live=2)
    plan = [("a", 60, 3), ("b", 200, 1), ("c", 45, 4), ("d", 9, 5), ("e", 130, 6)]
    live, waiting, done = {}, list(plan), set()
    while waiting or live:
        while waiting and len(live) < 2:
            name, n, seed = waiting.pop(0)
            live[name] = [eng.open(), 0, n, oracle("uneven", n, seed)]
        for name in list(live):
            seq, at, n, (toks, logits, _) = live[name]
            size = min([1, 13, 2, 30][(at + len(name) + n) % 4], n - at)
            out = eng.step(seq, toks[at:at + size], [size - 1])
            close(out, logits[at + size - 1:at + size], dtype)
            live[name][1] += size
            if live[name][1] == n:
                eng.close(seq)
                done.add(name)
                del live[name]
    assert done == set("abcde") and eng.state.free_slots == 2
    with pytest.raises(StateError):
        eng.step(0, [1])


@BOTH
def test_long_decoding_far_from_the_first_tokens(dtype):
    n = 500
    toks, logits, _ = oracle("tiles", n, 3)
    eng = engine("tiles", dtype)
    seq = eng.open()
    eng.step(seq, toks[:100])
    rows = [eng.step(seq, [t], [0]).clone() for t in toks[100:]]
    close(torch.cat(rows), logits[100:], dtype)


def test_a_sequence_ends_at_its_slot():
    eng = engine("uneven", torch.float32, max_tokens=50)
    seq = eng.open()
    eng.step(seq, [1] * 50)
    with pytest.raises(StateError):
        eng.step(seq, [1])
    with pytest.raises(ValueError):
        eng.step(eng.open(), [131])
    with pytest.raises(ValueError):
        eng.step(eng.open(), [1, 2], [1, 0])


@BOTH
def test_eager_decoding_equals_the_captured_graph(dtype):
    toks = cases.tokens(cases.TILES, 90, 4)
    rows = []
    for graphs in (True, False):
        eng = engine("tiles", dtype, use_graphs=graphs)
        seq = eng.open()
        eng.step(seq, toks[:70])
        rows.append(torch.cat([eng.step(seq, [t], [0]).clone() for t in toks[70:]]))
    assert torch.equal(rows[0], rows[1])


# --------------------------------------------- single keys that stand out --
def _lone_layer(dtype, heads, kv_heads, dim, vdim, window, keep):
    cfg = cases.config(64, 40, [cases.layer(cases.attention(heads, kv_heads, dim, vdim, window, keep, 1.0), None)], max_positions=700)
    t = cases.weights(cfg, 9)
    spec = bidasun.parse_config(cfg)
    return DenseEngine(dense.DenseModel(spec, bidasun.model_tensors(spec, lambda n, s: t[n]), dtype), portion=512), cases.as_float64(t)


@pytest.mark.parametrize("dtype,kernel", [(torch.float32, 1), (torch.bfloat16, 1), (torch.bfloat16, 2), (torch.bfloat16, 3)])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window,keep", [(4, 2, 64, 64, 100, 3), (3, 1, 128, 128, 64, 64), (2, 2, 32, 144, 65, 130),
                                                                 (8, 2, 80, 48, 1, 1), (2, 1, 64, 128, 300, 0), (2, 2, 128, 64, 600, 5)])
@pytest.mark.parametrize("first,rows", [(0, 330), (70, 5), (191, 130), (320, 64)])
def test_attention_one_key_stands_out(dtype, kernel, heads, kv_heads, dim, vdim, window, keep, first, rows):
    """All scores far below zero but for one key, whose value is its own: a query's output shows whether it sees
    that key, and with what weight, for keys inside and outside the window, among the kept ones and at tile borders."""
    if kernel == 3 and max(dim, vdim) > 128:
        pytest.skip("the tcgen05 attention takes heads of up to 128 columns")
    eng, w = _lone_layer(dtype, heads, kv_heads, dim, vdim, window, keep)
    n = first + rows
    rng = np.random.default_rng(n + window)
    dp, vp = dense.pad16(dim), dense.pad16(vdim)
    q, k = np.zeros((n, heads, dim)), np.zeros((n, kv_heads, dim))
    q[:, :, 0] = 1.0
    k[:, :, 0] = -30.0
    marks = sorted({0, 1, max(keep - 1, 0), keep, keep + 1, n // 3, max(first - 1, 0), first, max(n - 1 - window, 0), max(n - window, 0),
                    63, 64, 65, 127, 128} & set(range(n)))
    v = rng.standard_normal((n, kv_heads, vdim))
    gate = rng.standard_normal((n, heads, vdim))
    as_dtype = lambda a: torch.from_numpy(a).to(dtype).double().numpy()
    q, v, gate = as_dtype(q), as_dtype(v), as_dtype(gate)
    r1, r2, pb = (w["l0.mix." + x] for x in ("r1", "r2", "pb"))
    for mark in marks:
        kk = k.copy()
        kk[mark, :, 0] = 2.0
        want = ref.sigmoid_attention(q, kk, v, 1.0, r1, r2, pb, ref.visible(n, window, keep))[first:] * ref.sigmoid(gate[first:])
        columns = heads * dp + kv_heads * (dp + vp) + heads * vp
        pq = torch.zeros((rows, heads, dp), dtype=dtype, device="cuda")
        pq[:, :, :dim] = torch.from_numpy(q[first:]).to("cuda", dtype)
        pg = torch.zeros((rows, heads, vp), dtype=dtype, device="cuda")
        pg[:, :, :vdim] = torch.from_numpy(gate[first:]).to("cuda", dtype)
        eng._buf["proj"].zero_()
        eng._buf["proj"][:rows, :heads * dp] = pq.reshape(rows, -1)
        eng._buf["proj"][:rows, columns - heads * vp:columns] = pg.reshape(rows, -1)
        ck = torch.zeros((n, kv_heads, dp), dtype=dtype, device="cuda")
        ck[:, :, :dim] = torch.from_numpy(kk).to("cuda", dtype)
        cv = torch.zeros((n, kv_heads, vp), dtype=dtype, device="cuda")
        cv[:, :, :vdim] = torch.from_numpy(v).to("cuda", dtype)
        eng.state.k[0][2].fill_(7.0)
        eng.state.v[0][2].fill_(7.0)
        eng.state.k[0][2, :n] = ck.reshape(n, -1)
        eng.state.v[0][2, :n] = cv.reshape(n, -1)
        torch.cuda.synchronize()
        eng._set_step(first, 2)
        _dense.check(_dense.lib().twm_dense_attention(C.byref(eng._desc), 0, C.byref(eng._b), rows, first, kernel, 0,
                                                      eng.stream.cuda_stream), "attention")
        eng.stream.synchronize()
        got = eng._buf["att"][:rows].double().cpu().numpy().reshape(rows, heads, vp)
        assert np.abs(got[:, :, vdim:]).max(initial=0.0) == 0.0
        err = np.abs(got[:, :, :vdim] - want)
        assert err.max() < (2e-6 if dtype == torch.float32 else 2 ** -8) * max(1.0, np.abs(want).max()), (mark, float(err.max()))
    assert _dense.device_error() == 0


@BOTH
@pytest.mark.parametrize("case", ["tiles", "uneven"])
def test_decoded_keys_at_window_edges_stand_out(case, dtype):
    """A token whose embedding is large makes a key that stands out; the steps at which it leaves each layer's
    window, and after which it must not be seen, are decoded one by one."""
    cfg = json.loads(json.dumps(cases.CASES[case]))
    t = cases.weights(cfg, 7)
    t["embed"] = t["embed"].clone()
    t["embed"][5] *= 20
    rng = np.random.default_rng(0)
    toks = rng.integers(6, cfg["vocab"], 230)
    toks[[3, 70, 128]] = 5
    toks = toks.tolist()
    want = ref.forward(cfg, cases.as_float64(t), toks)
    spec = bidasun.parse_config(cfg)
    eng = DenseEngine(dense.DenseModel(spec, bidasun.model_tensors(spec, lambda n, s: t[n]), dtype))
    seq = eng.open()
    eng.step(seq, toks[:60])
    close(torch.cat([eng.step(seq, [x], [0]).clone() for x in toks[60:]]), want[60:], dtype)


# -------------------------------------------- scheduler and command line --
def _greedy(case, prompt, count):
    cfg = cases.CASES[case]
    w, toks = cases.as_float64(cases.weights(cfg, 7)), list(prompt)
    for _ in range(count):
        toks.append(int(ref.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    """Unequal requests, more than there are slots, in portions and bursts: each as the oracle generates it alone."""
    eng = engine("uneven", torch.float32, max_live=2)
    sch = Scheduler(eng, portion=16, burst=5)
    prompts = [cases.tokens(cases.UNEVEN, n, 20 + n) for n in (1, 40, 17, 2, 33)]
    requests = [sch.submit(p, 4 + 3 * i) for i, p in enumerate(prompts)]
    assert len(list(sch.run())) == 5 and eng.state.free_slots == 2
    for i, (p, r) in enumerate(zip(prompts, requests)):
        assert r.generated == _greedy("uneven", p, 4 + 3 * i), i
    assert _dense.device_error() == 0


def test_greedy_16_bit_agrees_with_stepwise_arg_max():
    eng = engine("tiles", torch.bfloat16)
    prompt = cases.tokens(cases.TILES, 70, 8)
    seq = eng.open()
    generated = eng.greedy(seq, prompt, 40)
    assert eng.length(seq) == 70 + 39
    again = eng.open()
    token = int(eng.step(again, prompt, [69])[0].argmax())
    for got in generated:
        assert got == token
        token = int(eng.step(again, [got], [0])[0].argmax())


def test_command_line(tmp_path):
    cases.save(str(tmp_path), cases.UNEVEN, cases.weights(cases.UNEVEN, 7))
    prompts = [cases.tokens(cases.UNEVEN, n, 40 + n) for n in (12, 3)]
    cmd = [sys.executable, "-m", "tensorwarp_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new-tokens", "6",
           "--max-live", "1"]
    for p in prompts:
        cmd += ["--tokens", ",".join(map(str, p))]
    out = subprocess.run(cmd, capture_output=True, text=True, cwd=ROOT, timeout=300)
    assert out.returncode == 0, out.stderr
    got = {x["request"]: x["generated"] for x in map(json.loads, out.stdout.splitlines())}
    assert got == {i: _greedy("uneven", p, 6) for i, p in enumerate(prompts)}


@BOTH
def test_trace_program(tmp_path, dtype):
    model, out = tmp_path / "model", tmp_path / "out"
    model.mkdir(), out.mkdir()
    cases.save(str(model), cases.TILES, cases.weights(cases.TILES, 7))
    toks, logits, _ = oracle("tiles", 200, 1)
    steps, at = [], 0
    for i, size in enumerate([90, 2, 1, 1, 70, 1, 35]):
        steps.append({"step": i, "entries": [{"id": "q", "tokens": toks[at:at + size], "want": [0, size - 1] if size > 1 else [0]}],
                      "end": ["q"] if at + size == 200 else []})
        at += size
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype",
                          "float32" if dtype == torch.float32 else "bfloat16", "--out", str(out), "--max-tokens", "256"],
                         input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    assert [x for x in run.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(7)]
    at = 0
    for s in steps:
        e = s["entries"][0]
        got = np.fromfile(out / f"{s['step']}.f32", "<f4").reshape(len(e["want"]), 300)
        close(got, logits[[at + p for p in e["want"]]], dtype)
        at += len(e["tokens"])


def test_checkpoint_on_disk_equals_tensors_in_memory(tmp_path):
    cases.save(str(tmp_path), cases.WIDE, cases.weights(cases.WIDE, 7))
    toks, logits, _ = oracle("wide", 60, 2)
    eng = registry.load(str(tmp_path), dtype=torch.float32, max_tokens=64)
    close(eng.step(eng.open(), toks, list(range(60))), logits, torch.float32)
