"""GPU tests of the Zukotar design through the framework's engine, scheduler and command line, and of its mechanisms
alone, against the plain implementation in oracle/zukotar_ref.py (float64, whole sequences, no cache)."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import zukotar_cases as cases
from oracle import zukotar_ref as ref
from tensorwarp_b200 import _dense, dense, registry
from tensorwarp_b200.engine import DenseEngine
from tensorwarp_b200.scheduler import Scheduler
from tensorwarp_b200.state import StateError

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 2e-5, torch.bfloat16: 5e-2}
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
CASE = pytest.mark.parametrize("case", sorted(cases.CASES))

_oracle_cache = {}


def oracle(case, n, seed):
    """Logits and residual stream after every layer run of `n` seeded tokens."""
    key = (case, n, seed)
    if key not in _oracle_cache:
        cfg = cases.CASES[case]
        layers = []
        toks = cases.tokens(cfg, n, seed)
        logits = ref.forward(cfg, cases.as_float64(cases.weights(cfg, 7, cases.RANKS[case])), toks, layers)
        _oracle_cache[key] = (toks, logits, layers)
    return _oracle_cache[key]


def engine(case, dtype, **options):
    cfg, rank = cases.CASES[case], cases.RANKS[case]
    options.setdefault("max_tokens", 640)
    return DenseEngine(cases.model(cfg, cases.weights(cfg, 7, rank), rank, dtype), **options)


def close(got, want, dtype, case="tiles", tol=None):
    """In 16 bits a choice of experts that is nearly a tie may go either way: where the model chooses, most rows are compared.
    Where all experts are used, rounding the norms alone to 16 bits in the oracle moves single rows by 0.06, half of them
    by less than 0.015."""
    err = cases.error(got.cpu().numpy() if torch.is_tensor(got) else got, want)
    if dtype == torch.bfloat16:
        q = 0.9 if case == "tiles" else 0.75
        assert np.quantile(err, q) < TOL[dtype] and np.isfinite(err).all(), float(np.quantile(err, q))
        assert case != "tiles" or err.max() < 0.2, (int(err.argmax()), float(err.max()))
    else:
        assert err.max() < (tol or TOL[dtype]), (int(err.argmax()), float(err.max()))
    assert _dense.device_error() == 0


@BOTH
@CASE
def test_whole_prompt_and_every_layer(case, dtype):
    n = 200
    toks, logits, layers = oracle(case, n, 1)
    eng = engine(case, dtype)
    seq, got = eng.open(), []
    out = eng.step(seq, toks, list(range(n)), layer_trace=got)
    close(out, logits, dtype, case)
    assert len(got) == 1 and got[0].shape == (len(layers), n, cases.CASES[case]["width"])
    for g, want in zip(got[0].cpu().numpy(), layers):
        rows = np.sqrt(((g - want) ** 2).mean(axis=1)) / want.std()
        assert (rows.max() if dtype == torch.float32 else np.quantile(rows, 0.9 if case == "tiles" else 0.75)) < TOL[dtype]


@BOTH
@CASE
def test_token_by_token(case, dtype):
    """Decoding from the first token on: every window's edge and tile borders pass by."""
    n = 200
    toks, logits, _ = oracle(case, n, 1)
    eng = engine(case, dtype)
    seq = eng.open()
    rows = [eng.step(seq, [t], [0]).clone() for t in toks]
    close(torch.cat(rows), logits, dtype, case)


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
    close(torch.cat(rows), logits, dtype, case)


@BOTH
@CASE
def test_portions_of_changing_size_with_decoding_between(case, dtype):
    n = 250
    toks, logits, _ = oracle(case, n, 2)
    eng = engine(case, dtype)
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
    close(torch.cat(got), logits[want], dtype, case)


@BOTH
def test_more_tokens_and_wanted_rows_than_the_buffers_take(dtype):
    """A step that has to be cut inside the engine, by its tokens and by its wanted rows."""
    n = 200
    toks, logits, _ = oracle("tiles", n, 1)
    eng = engine("tiles", dtype, portion=48)
    assert eng.max_rows == 48
    eng.max_want = 11
    want = [0, 1, 2, 3, 10, 11, 12, 13, 14, 15, 16, 17, 40, 47, 48, 49, 95, 96, 97] + list(range(150, 200))
    close(eng.step(eng.open(), toks, want), logits[want], dtype)


@BOTH
@pytest.mark.parametrize("case", ["uneven", "tiles"])
def test_slots_used_again_and_sequences_interleaved(case, dtype):
    """Several sequences in flight, slots freed and taken by others of other lengths: each as if alone."""
    eng = engine(case, dtype, max_live=2)
    plan = [("a", 60, 3), ("b", 200, 1), ("c", 45, 4), ("d", 9, 5), ("e", 130, 6)]
    live, waiting, got, want = {}, list(plan), [], []
    while waiting or live:
        while waiting and len(live) < 2:
            name, n, seed = waiting.pop(0)
            live[name] = [eng.open(), 0, n, oracle(case, n, seed)]
        for name in list(live):
            seq, at, n, (toks, logits, _) = live[name]
            size = min([1, 13, 2, 30][(at + len(name) + n) % 4], n - at)
            got.append(eng.step(seq, toks[at:at + size], [size - 1]).clone())
            want.append(logits[at + size - 1:at + size])
            live[name][1] += size
            if live[name][1] == n:
                eng.close(seq)
                del live[name]
    assert eng.state.free_slots == 2
    close(torch.cat(got), np.concatenate(want), dtype, case)
    with pytest.raises(StateError):
        eng.step(0, [1])


@BOTH
@pytest.mark.parametrize("case", ["uneven", "tiles"])
def test_long_decoding_far_from_the_first_tokens(case, dtype):
    n = 500
    toks, logits, _ = oracle(case, n, 3)
    eng = engine(case, dtype)
    seq = eng.open()
    eng.step(seq, toks[:100])
    rows = [eng.step(seq, [t], [0]).clone() for t in toks[100:]]
    close(torch.cat(rows), logits[100:], dtype, case)


@BOTH
def test_long_prompt(dtype):
    """More tokens than the kernels' grids hold at once; every window has passed many times.  Over thousands of tokens the
    32-bit rounding of slow decays (next to 1) adds up in the state."""
    n = 2200
    toks, logits, _ = oracle("tiles", n, 5)
    eng = engine("tiles", dtype, max_tokens=n, portion=n)
    want = [0, 1, 63, 64, 65, 1023, 1024, 2047, 2048, 2049] + list(range(2150, n))
    for _ in range(3):
        seq = eng.open()
        close(eng.step(seq, toks, want), logits[want], dtype, tol=1e-4)
        eng.close(seq)


@BOTH
@pytest.mark.parametrize("width,ff,top", [(80, 1200, 3), (2400, 40, 3), (1300, 1210, 2), (5000, 16, 2)])
def test_experts_larger_than_one_pass_of_the_decode_products(width, ff, top, dtype):
    cfg = cases.config(width, 61, [cases.layer(cases.linear(2, 16, 16), cases.experts(top, top, ff)),
                                   cases.layer(cases.latent(2, 16, 8, 16, 16, 5), cases.experts(top, top, ff))])
    t = cases.weights(cfg, 3, 4)
    toks = cases.tokens(cfg, 14, 3)
    want = ref.forward(cfg, cases.as_float64(t), toks)
    eng = DenseEngine(cases.model(cfg, t, 4, dtype), max_tokens=32)
    seq = eng.open()
    close(torch.cat([eng.step(seq, [x], [0]).clone() for x in toks]), want, dtype)
    close(eng.step(eng.open(), toks, list(range(14))), want, dtype)


def test_a_sequence_ends_at_its_slot():
    eng = engine("uneven", torch.float32, max_tokens=50)
    seq = eng.open()
    eng.step(seq, [1] * 50)
    with pytest.raises(StateError):
        eng.step(seq, [1])
    with pytest.raises(ValueError):
        eng.step(eng.open(), [131])


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


@BOTH
@CASE
def test_a_key_that_stands_out_passes_every_window(case, dtype):
    """A token whose embedding is large makes a key and a state that stand out; the steps at which it leaves each layer's
    window, and after which it must not be seen, are decoded one by one, and come again in one prompt."""
    cfg, rank = json.loads(json.dumps(cases.CASES[case])), cases.RANKS[case]
    t = cases.weights(cfg, 7, rank)
    t["embed"] = t["embed"].clone()
    t["embed"][5] *= 20
    toks = np.random.default_rng(0).integers(6, cfg["vocab"], 230)
    toks[[3, 70, 128]] = 5
    toks = toks.tolist()
    want = ref.forward(cfg, cases.as_float64(t), toks)
    eng = DenseEngine(cases.model(cfg, t, rank, dtype), max_tokens=256)
    seq = eng.open()
    eng.step(seq, toks[:60])
    close(torch.cat([eng.step(seq, [x], [0]).clone() for x in toks[60:]]), want[60:], dtype, case)
    close(eng.step(eng.open(), toks, list(range(230))), want, dtype, case)


# ----------------------------------------------------- mechanisms alone --
def as_dtype(a, dtype):
    return torch.from_numpy(np.ascontiguousarray(a)).to(dtype).double().numpy()


def put(rows, parts, dtype):
    """[rows, ...] arrays side by side, each head's columns padded to a multiple of 16."""
    out = []
    for a in parts:
        a = a.reshape(rows, -1, a.shape[-1])
        p = torch.zeros((rows, a.shape[1], dense.pad16(a.shape[2])), dtype=dtype)
        p[:, :, :a.shape[2]] = torch.from_numpy(a).to(dtype)
        out.append(p.reshape(rows, -1))
    return torch.cat(out, dim=1).cuda()


@pytest.mark.parametrize("dtype,kernel", [(torch.float32, 1), (torch.bfloat16, 1), (torch.bfloat16, 3)])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank,window", [(3, 64, 16, 64, 48, 100), (2, 128, 64, 128, 96, 64), (2, 40, 32, 80, 20, 65),
                                                            (5, 16, 6, 33, 30, 1), (1, 96, 48, 112, 64, 300), (2, 64, 64, 16, 33, None)])
@pytest.mark.parametrize("first,rows", [(0, 330), (70, 5), (191, 130), (320, 64)])
def test_latent_attention_one_key_stands_out(dtype, kernel, heads, dim, rot, vdim, rank, window, first, rows):
    """Queries along one latent direction, in which all tokens but one lie on the far side: a query's output shows whether it
    sees that token, and with what weight, inside and outside the window and at tile borders."""
    n = first + rows
    cfg = cases.config(64, 40, [cases.layer(cases.latent(heads, dim, rot, vdim, rank, window, 1.0, 300.0), None)])
    t = cases.weights(cfg, 9, 1)
    eng = DenseEngine(cases.model(cfg, t, 1, dtype), max_tokens=512, max_live=4)
    w = cases.as_float64(t)
    rng = np.random.default_rng(n + (window or 0))
    uk, uv = w["l0.mix.uk"].reshape(heads, dim, rank), w["l0.mix.uv"].reshape(heads, vdim, rank)
    first_col = uk[:, :, 0]
    q = np.zeros((n, heads, dim + rot))
    q[:, :, :dim] = first_col / (first_col ** 2).sum(axis=1, keepdims=True)
    q[:, :, dim:] = rng.standard_normal((n, heads, rot)) * 0.3
    q, gate = as_dtype(q, dtype), as_dtype(rng.standard_normal((n, heads)), dtype)
    pos = np.arange(n)
    down0 = rng.standard_normal((n, rank + rot)) * 0.5
    down0[:, 0] = -6.0
    window_of = window if window is not None else n
    marks = sorted({0, 1, n // 3, max(first - 1, 0), first, max(n - 1 - window_of, 0), max(n - window_of, 0), 63, 64, 65, 127, 128} & set(range(n)))
    for mark in marks[::2] if kernel != 3 else marks:
        down = down0.copy()
        down[mark, 0] = 6.0
        down = as_dtype(down, dtype)
        lat = ref.rms_norm(down[:, :rank], w["l0.mix.dkv.norm"], cfg["norm"]["eps"])
        q_rot, k_rot = ref.rotate(q[:, :, dim:], pos, 300.0), ref.rotate(down[:, rank:], pos, 300.0)
        k = np.concatenate([np.einsum("hdr,nr->nhd", uk, lat), np.broadcast_to(k_rot[:, None], (n, heads, rot))], axis=2)
        v = np.einsum("her,nr->nhe", uv, lat)
        want = ref.softmax_attention(np.concatenate([q[:, :, :dim], q_rot], axis=2), k, v, 1.0, ref.visible(n, window))
        want = (want * ref.sigmoid(gate)[:, :, None])[first:]
        proj = put(rows, [np.concatenate([np.pad(q[first:, :, :dim], ((0, 0), (0, 0), (0, dense.pad16(dim) - dim))), q[first:, :, dim:]], axis=2),
                          down[first:, :rank], down[first:, rank:], gate[first:]], dtype)
        eng._buf["proj"].zero_()
        eng._buf["proj"].view(-1)[:proj.numel()] = proj.reshape(-1)
        cache = eng.state.runs[0]["latent_cache"]
        cache[2].fill_(7.0)
        if first:
            cache[2, :first] = put(first, [lat[:first], k_rot[:first]], dtype)
        torch.cuda.synchronize()
        eng._set_step(first, 2)
        _dense.check(_dense.lib().twm_dense_attention(C.byref(eng._desc), 0, C.byref(eng._b), rows, first, kernel, 0,
                                                      eng.stream.cuda_stream), "attention")
        eng.stream.synchronize()
        got = eng._buf["att"].view(-1)[:rows * heads * dense.pad16(vdim)].double().cpu().numpy().reshape(rows, heads, -1)
        assert np.abs(got[:, :, vdim:]).max(initial=0.0) == 0.0
        err = np.abs(got[:, :, :vdim] - want)
        assert err.max() < (1e-5 if dtype == torch.float32 else 4e-2) * max(1.0, np.abs(want).max()), (mark, float(err.max()))
    assert _dense.device_error() == 0


@pytest.mark.parametrize("dtype,kernel", [(torch.float32, 1), (torch.bfloat16, 1), (torch.bfloat16, 2)])
@pytest.mark.parametrize("heads,dim,vdim,rank,tau,bias", [(2, 64, 64, 16, 16.0, (0, 5)), (3, 128, 128, 40, 4.0, (-1, 6)), (2, 20, 36, 5, 1.0, (-3, 3)),
                                                          (1, 48, 112, 16, 2.0, (-30, 5)), (2, 32, 16, 16, 0.5, (-60, -20)),
                                                          (2, 160, 80, 16, 8.0, (0, 9))])
@pytest.mark.parametrize("portions", [(200,), (1, 63, 64, 65, 7), (2, 130)])
def test_linear_attention_alone(dtype, kernel, heads, dim, vdim, rank, tau, bias, portions):
    """State carried over portions of any size, with decays from nearly none to nearly total (far below what a chunk's
    exponents could hold in one factor)."""
    cfg = cases.config(64, 40, [cases.layer(cases.linear(heads, dim, vdim, tau), None)])
    t = cases.weights(cfg, 9, rank)
    rng = np.random.default_rng(dim + rank)
    t["l0.mix.a2.b"] = torch.from_numpy(rng.uniform(*bias, heads * dim)).to(torch.bfloat16)
    eng = DenseEngine(cases.model(cfg, t, rank, dtype), max_tokens=512, max_live=3)
    w = cases.as_float64(t)
    n = sum(portions)
    q, k = (as_dtype(rng.standard_normal((n, heads, dim)), dtype) for _ in range(2))
    v, gate = (as_dtype(rng.standard_normal((n, heads, vdim)), dtype) for _ in range(2))
    low = as_dtype(rng.standard_normal((n, rank)), dtype)
    z = low @ w["l0.mix.a2"].T + w["l0.mix.a2.b"]
    alpha = np.exp(-np.logaddexp(0.0, -z) / tau).reshape(n, heads, dim)
    o, state = ref.recurrence(q * dim ** -0.5, k, v, alpha)
    want = ref.rms_norm(o, w["l0.mix.norm"], cfg["norm"]["eps"]) * ref.silu(gate)
    kept = eng.state.runs[0]["gla_state"]
    kept.fill_(3.0)                                         # another sequence's
    at, got = 0, []
    for rows in portions:
        s = slice(at, at + rows)
        proj = put(rows, [q[s], k[s], v[s], gate[s], low[s]], dtype)
        eng._buf["proj"].view(-1)[:proj.numel()] = proj.reshape(-1)
        torch.cuda.synchronize()
        eng._set_step(at, 1)
        _dense.check(_dense.lib().twm_dense_gla(C.byref(eng._desc), 0, C.byref(eng._b), rows, kernel, 0, eng.stream.cuda_stream), "gla")
        eng.stream.synchronize()
        out = eng._buf["att"].view(-1)[:rows * heads * dense.pad16(vdim)].double().cpu().numpy().reshape(rows, heads, -1)
        assert np.abs(out[:, :, vdim:]).max(initial=0.0) == 0.0
        got.append(out[:, :, :vdim])
        at += rows
    err = np.abs(np.concatenate(got) - want)
    # a norm makes every head's o large: where o is a difference of large terms its error grows with it
    assert err.max() < (2e-4 if dtype == torch.float32 else 3e-2) * max(1.0, np.abs(want).max()), float(err.max())
    assert np.sqrt((err ** 2).mean()) < (1e-5 if dtype == torch.float32 else 4e-3)
    held = kept[1, :, :dim, :vdim].double().cpu().numpy()
    assert np.abs(held - state).max() < (1e-5 if dtype == torch.float32 else 1e-4) * np.abs(state).max()
    assert bool((kept[0] == 3.0).all()) and bool((kept[2] == 3.0).all()) and _dense.device_error() == 0


@pytest.mark.parametrize("n,top,groups,keep", [(12, 3, 2, 1), (10, 4, 5, 3), (64, 6, 1, 1), (256, 8, 8, 4), (1000, 32, 40, 3), (7, 7, 1, 1), (5, 1, 5, 1)])
def test_router(n, top, groups, keep):
    rows = 61
    z = torch.from_numpy(np.random.default_rng(n).standard_normal((rows, n)).astype(np.float32) * 3).cuda()
    ids, weights = torch.zeros((rows, top), dtype=torch.int32, device="cuda"), torch.zeros((rows, top), device="cuda")
    _dense.check(_dense.lib().twm_dense_route(z.data_ptr(), n, top, groups, keep, rows, ids.data_ptr(), weights.data_ptr(), 0,
                                              torch.cuda.current_stream().cuda_stream), "route")
    torch.cuda.synchronize()
    for r in range(rows):
        chosen, s = ref.route(z[r].double().cpu().numpy(), top, {"count": groups, "keep": keep})
        assert ids[r].tolist() == chosen.tolist()
        assert np.abs(weights[r].double().cpu().numpy() - s).max() < 1e-6


@pytest.mark.parametrize("counts,n,k", [((3, 0, 130, 1), 64, 48), ((0, 0, 5), 200, 80), ((128, 128), 130, 256), ((1,) * 40, 48, 16),
                                        ((257, 0, 300, 64, 2, 500), 320, 192), ((7, 900, 0), 1030, 64), ((1500, 0, 900, 3), 2048, 96)])
@pytest.mark.parametrize("dtype,kernel", [(torch.float32, 1), (torch.bfloat16, 1), (torch.bfloat16, 64), (torch.bfloat16, 128), (torch.bfloat16, 256),
                                          (torch.bfloat16, 0)])
@pytest.mark.parametrize("epi", [_dense.EPI_STORE, _dense.EPI_STORE_F32, _dense.EPI_RELU2])
def test_grouped_product(counts, n, k, dtype, kernel, epi):
    gen = torch.Generator(device="cuda").manual_seed(n + k)
    rows = sum(counts)
    a = torch.randn((rows, k), generator=gen, device="cuda").to(dtype)
    w = (torch.randn((len(counts), n, k), generator=gen, device="cuda") / k ** 0.5).to(dtype)
    offsets = torch.tensor(np.concatenate([[0], np.cumsum(counts)]), dtype=torch.int32, device="cuda")
    c = torch.full((rows, n + 3), 7.0, dtype=torch.float32 if epi == _dense.EPI_STORE_F32 else dtype, device="cuda")
    dt = _dense.TWM_DENSE_F32 if dtype == torch.float32 else _dense.TWM_DENSE_BF16
    _dense.check(_dense.lib().twm_dense_grouped_gemm(dt, a.data_ptr(), k, w.data_ptr(), k, c.data_ptr(), n + 3, offsets.data_ptr(), len(counts),
                                                     rows, n, k, epi, kernel, 0, torch.cuda.current_stream().cuda_stream), "grouped_gemm")
    torch.cuda.synchronize()
    assert _dense.device_error() == 0 and bool((c[:, n:] == 7.0).all())
    want, at = [], 0
    for e, m in enumerate(counts):
        want.append(a[at:at + m].double() @ w[e].double().T)
        at += m
    want = torch.cat(want)
    if epi == _dense.EPI_RELU2:
        want = want.clamp(min=0) ** 2
    stored16 = dtype == torch.bfloat16 and epi != _dense.EPI_STORE_F32
    assert bool(((c[:, :n].double() - want).abs() <= want.abs() * (2 ** -8 if stored16 else 2e-5) + 3e-5).all())


# -------------------------------------------- scheduler and command line --
def _greedy(case, prompt, count):
    cfg = cases.CASES[case]
    w, toks = cases.as_float64(cases.weights(cfg, 7, cases.RANKS[case])), list(prompt)
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
    cases.save(str(tmp_path), cases.UNEVEN, cases.weights(cases.UNEVEN, 7, cases.RANKS["uneven"]))
    prompts = [cases.tokens(cases.UNEVEN, n, 40 + n) for n in (12, 3)]
    cmd = [sys.executable, "-m", "tensorwarp_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--max-new-tokens", "6",
           "--max-live", "1", "--max-tokens", "64"]
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
    cases.save(str(model), cases.TILES, cases.weights(cases.TILES, 7, cases.RANKS["tiles"]))
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
    cases.save(str(tmp_path), cases.WIDE, cases.weights(cases.WIDE, 7, cases.RANKS["wide"]))
    toks, logits, _ = oracle("wide", 60, 2)
    eng = registry.load(str(tmp_path), dtype=torch.float32, max_tokens=64)
    close(eng.step(eng.open(), toks, list(range(60))), logits, torch.float32)
