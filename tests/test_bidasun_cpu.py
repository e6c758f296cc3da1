"""CPU tests of the Bidasun design's parts that need no GPU: configuration, checkpoint, weight layout, sequence
slots, scheduler, trace replay; and of the oracle: each mechanism against its closed form, and that a
mechanism that is off by one shows in the logits of the test models."""
import copy
import io
import json
import math

import numpy as np
import pytest
import torch

import bidasun_cases as cases
from oracle import bidasun_ref as ref
from tensorwarp_b200 import checkpoint, dense, registry, trace
from tensorwarp_b200.models import bidasun
from tensorwarp_b200.scheduler import Scheduler
from tensorwarp_b200.state import SequenceState, StateError


# ------------------------------------------------------------------- oracle --
def test_oracle_mechanisms_closed_forms():
    assert np.allclose(ref.rms_norm(np.array([[3.0, 4.0]]), np.array([1.0, 2.0]), 0.0), [[3 / math.sqrt(12.5), 8 / math.sqrt(12.5)]])
    assert ref.rms_norm(np.zeros((1, 4)), np.ones(4), 1e-6).max() == 0.0
    assert abs(ref.gelu_tanh(np.array(1.0)) - 0.841192) < 1e-6
    assert np.allclose(ref.sigmoid(np.array([0.0, 800.0, -800.0])), [0.5, 1.0, 0.0])
    x = np.array([[1.0], [2.0], [4.0]])
    assert np.allclose(ref.token_shift(x, np.array([0.25])), [[0.75], [1.75], [3.5]])
    assert ref.distance_bias(2.0, 0.5, 0) == 0.0 and abs(ref.distance_bias(2.0, 0.5, 2) - 2 * math.log(2)) < 1e-12
    m = ref.visible(6, 2, 1)
    assert m[5].tolist() == [True, False, False, False, True, True] and m[1].tolist() == [True, True, False, False, False, False]
    assert np.array_equal(ref.visible(5, 100, 0), np.tril(np.ones((5, 5), bool)))


def test_oracle_attention_by_hand():
    q = np.array([[[1.0, 0.0]], [[0.0, 2.0]]])
    k = np.array([[[3.0, 1.0]], [[0.5, -1.0]]])
    v = np.array([[[1.0]], [[10.0]]])
    out = ref.sigmoid_attention(q, k, v, 0.5, np.array([0.7]), np.array([0.3]), np.array([-1.0]), ref.visible(2, 5, 0))
    s = lambda z: 1 / (1 + math.exp(-z))
    assert abs(out[0, 0, 0] - s(1.5 - 1)) < 1e-12
    assert abs(out[1, 0, 0] - (s(1.0 - 0.7 * math.log(1.3) - 1) + 10 * s(-1.0 - 1))) < 1e-12


@pytest.mark.parametrize("case", sorted(cases.CASES))
def test_planted_mistakes_show(case):
    """Every mechanism moved by one, dropped or doubled in the oracle changes the logits by far more than the
    tolerances of the GPU tests (2e-5 in 32-bit)."""
    cfg, w = cases.CASES[case], cases.as_float64(cases.weights(cases.CASES[case], 11))
    toks = cases.tokens(cfg, 150, 5)
    base = ref.forward(cfg, w, toks)

    def moved(change_cfg=None, change_w=None):
        c, ww = copy.deepcopy(cfg), dict(w)
        for i, lay in enumerate(c["layers"]):
            if change_cfg:
                change_cfg(lay["mixer"])
            if change_w:
                change_w(ww, f"l{i}.")
        return float(cases.error(ref.forward(c, ww, toks), base).max())

    def mask(key, by):
        def change(m):
            if "mask" in m:
                m["mask"][key] = max(m["mask"][key] + by, 0)
        return change

    def fill(name, value):
        return lambda ww, p: ww.__setitem__(p + name, np.full_like(ww[p + name], value))

    assert moved(mask("size", 1)) > 2e-3
    assert moved(mask("keep_first", 1)) > 2e-3
    assert moved(mask("keep_first", -1)) > 2e-3
    assert moved(lambda m: m.__setitem__("scale", m["scale"] * 1.05)) > 2e-3
    for name, value in (("shift", 0.0), ("mix.r1", 0.0), ("mix.r2", 0.0), ("mix.pb", 0.0), ("mix.g", 0.0), ("mix.q.norm", 1.0),
                        ("mix.k.norm", 1.0), ("norm1", 1.0)):
        assert moved(change_w=fill(name, value)) > 2e-3, name


# ------------------------------------------------------------ configuration --
def test_config_is_read_layer_by_layer():
    spec = bidasun.parse_config(cases.UNEVEN)
    assert (spec.vocab, spec.width, spec.eps, spec.max_positions) == (131, 52, 3e-4, 320)
    assert [x.ff for x in spec.layers] == [72, None, 50, 33]
    assert spec.layers[0].mixer == dense.AttentionSpec(4, 2, 24, 40, 0.3, 9, 3)
    assert spec.layers[3].mixer.window >= 1 << 20 and spec.layers[3].mixer.keep_first == 0
    shapes = bidasun.tensor_shapes(spec)
    assert shapes["l2.mix.o"] == (52, 288) and shapes["l0.mix.k.norm"] == (48,) and shapes["pos"] == (320, 52)
    assert "l1.norm2" not in shapes and "l1.mlp.up" not in shapes and "l1.shift" in shapes


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].__setitem__("type", "other"),
    lambda c: c["layers"][0]["mixer"].__setitem__("heads", 3),
    lambda c: c["layers"][0]["mixer"].__setitem__("unheard_of", 1),
    lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("unheard_of", 1),
    lambda c: c["layers"][0]["mlp"].__setitem__("kind", "other"),
])
def test_what_the_design_does_not_have_is_refused(change):
    cfg = copy.deepcopy(cases.UNEVEN)
    change(cfg)
    with pytest.raises(checkpoint.CheckpointError):
        bidasun.parse_config(cfg)


def test_registry():
    assert {"Bidasun", "TWMarlinQ4"} <= set(registry.architectures())
    with pytest.raises(checkpoint.CheckpointError, match="unknown architecture"):
        registry.builder_for({"architecture": "nobody"})
    assert registry.builder_for(cases.UNEVEN) is bidasun.build


# --------------------------------------------------------------- checkpoints --
def test_checkpoint_round_trip_and_errors(tmp_path):
    t = {"a": torch.randn(3, 5).bfloat16(), "b": torch.arange(6, dtype=torch.int32).reshape(2, 3), "c": torch.randn(4)}
    path = str(tmp_path / "x.safetensors")
    checkpoint.write_safetensors(path, t)
    f = checkpoint.SafetensorsFile(path)
    assert sorted(f.names()) == ["a", "b", "c"]
    for name, want in t.items():
        got = f.get(name, tuple(want.shape))
        assert got.dtype == want.dtype and torch.equal(got, want)
    with pytest.raises(checkpoint.CheckpointError, match="missing"):
        f.get("d", (1,))
    with pytest.raises(checkpoint.CheckpointError, match="shape"):
        f.get("a", (5, 3))
    f.close()
    (tmp_path / "short").write_bytes(b"\0" * 4)
    with pytest.raises(checkpoint.CheckpointError):
        checkpoint.SafetensorsFile(str(tmp_path / "short"))


def test_header_of_any_length(tmp_path):
    """Data that does not start on a 16-byte boundary of the file."""
    t = torch.randn(7, 3).bfloat16()
    raw = t.view(torch.uint8).numpy().tobytes()
    head = json.dumps({"__metadata__": {"x": "y"}, "w": {"dtype": "BF16", "shape": [7, 3], "data_offsets": [0, len(raw)]}}).encode()
    path = tmp_path / "odd.safetensors"
    path.write_bytes(len(head + b" ").to_bytes(8, "little") + head + b" " + raw)
    assert torch.equal(checkpoint.SafetensorsFile(str(path)).get("w", (7, 3)), t)


# ------------------------------------------------------------- weight layout --
@pytest.mark.parametrize("case", sorted(cases.CASES))
def test_padded_fused_weights_compute_the_same(case):
    """The padded, fused tensors of a layer give the projections, norms and outputs of the plain ones, and nothing
    in the padding."""
    cfg = cases.CASES[case]
    spec = bidasun.parse_config(cfg)
    tensors = cases.weights(cfg, 3)
    model = dense.DenseModel(spec, bidasun.model_tensors(spec, lambda n, s: tensors[n]), torch.float32, "cpu")
    plain = {k: v.double() for k, v in tensors.items()}
    x = torch.randn(3, spec.width, dtype=torch.float64)
    xp = torch.zeros(3, model.width_pad, dtype=torch.float64)
    xp[:, :spec.width] = x
    for i, (lay, w) in enumerate(zip(spec.layers, model.layers)):
        m, p = lay.mixer, f"l{i}."
        dp, vp = dense.pad16(m.dim), dense.pad16(m.vdim)
        y = xp @ w["w_in"].double().T
        parts = torch.split(y, [m.heads * dp, m.kv_heads * dp, m.kv_heads * vp, m.heads * vp], dim=1)
        for part, name, n, size in zip(parts, "qkvg", (m.heads, m.kv_heads, m.kv_heads, m.heads), (m.dim, m.dim, m.vdim, m.vdim)):
            part = part.reshape(3, n, -1)
            assert torch.allclose(part[:, :, :size].reshape(3, -1), x @ plain[p + "mix." + name].T, atol=1e-5)
            assert bool((part[:, :, size:] == 0).all())
        assert torch.equal(w["q_norm"].reshape(m.heads, dp)[:, :m.dim].reshape(-1).double(), plain[p + "mix.q.norm"])
        a = torch.randn(3, m.heads, vp, dtype=torch.float64)
        o = a.reshape(3, -1) @ w["w_out"].double().T
        assert torch.allclose(o, a[:, :, :m.vdim].reshape(3, -1) @ plain[p + "mix.o"].T, atol=1e-5)
        if lay.ff is not None:
            fp = dense.pad16(lay.ff)
            gu = xp @ w["w_gate_up"].double().T
            assert torch.allclose(gu[:, :lay.ff], x @ plain[p + "mlp.gate"].T, atol=1e-5) and bool((gu[:, lay.ff:fp] == 0).all())
            assert torch.allclose(gu[:, fp:fp + lay.ff], x @ plain[p + "mlp.up"].T, atol=1e-5) and bool((gu[:, fp + lay.ff:] == 0).all())
        table = w["bias_table"].double().numpy()
        for h in (0, m.heads - 1):
            r1, r2, pb = (float(plain[p + "mix." + n][h]) for n in ("r1", "r2", "pb"))
            want = pb - ref.distance_bias(r1, r2, np.arange(spec.max_positions, dtype=np.float64))
            assert np.abs(table[h] - want).max() < 1e-6 * max(1.0, np.abs(want).max())


# --------------------------------------------------------------------- state --
def _cpu_model():
    spec = bidasun.parse_config(cases.UNEVEN)
    t = cases.weights(cases.UNEVEN, 1)
    return dense.DenseModel(spec, bidasun.model_tensors(spec, lambda n, s: t[n]), torch.bfloat16, "cpu")


def test_slots_are_taken_returned_and_bounded():
    st = SequenceState(_cpu_model(), slots=2, capacity=10)
    a, b = st.open(), st.open()
    assert {a, b} == {0, 1} and st.free_slots == 0
    with pytest.raises(StateError):
        st.open()
    st.advance(a, 7)
    with pytest.raises(StateError):
        st.advance(a, 4)
    assert st.length(a) == 7 and st.length(b) == 0
    st.close(a)
    with pytest.raises(StateError):
        st.length(a)
    with pytest.raises(StateError):
        st.close(a)
    assert st.open() == a and st.length(a) == 0
    assert st.k[2].shape == (2, 10, 2 * 80) and st.v[2].shape == (2, 10, 2 * 144) and st.shift[0].shape == (2, 2, 64)
    assert st.bytes() > 0


# ----------------------------------------------------------------- scheduler --
class CountingEngine:
    """The next token is the sum of all tokens so far modulo the vocabulary: an engine whose answers show
    any token that was lost, doubled or run in another sequence."""
    vocab, capacity = 97, 64

    def __init__(self, max_live=2):
        self.max_live, self.live, self.calls, self.most = max_live, {}, [], 0

    def open(self):
        seq = min(set(range(self.max_live)) - set(self.live))
        self.live[seq] = []
        self.most = max(self.most, len(self.live))
        return seq

    def close(self, seq):
        del self.live[seq]

    def length(self, seq):
        return len(self.live[seq])

    def step(self, seq, tokens, want=()):
        self.calls.append((seq, len(tokens)))
        rows = []
        for i, t in enumerate(tokens):
            self.live[seq].append(t)
            if i in want:
                rows.append(torch.nn.functional.one_hot(torch.tensor(sum(self.live[seq]) % self.vocab), self.vocab).float())
        return torch.stack(rows) if rows else None

    def greedy(self, seq, tokens, count):
        out = []
        for _ in range(count):
            out.append(int(self.step(seq, tokens, [len(tokens) - 1])[0].argmax()))
            tokens = out[-1:]
        return out


def _count(tokens, n):
    tokens, out = list(tokens), []
    for _ in range(n):
        out.append(sum(tokens) % 97)
        tokens.append(out[-1])
    return out


def test_scheduler_serves_more_requests_than_sequences():
    eng = CountingEngine(2)
    sch = Scheduler(eng, portion=5, burst=3)
    prompts = [list(range(1, n + 1)) for n in (1, 17, 4, 6, 11)]
    requests = [sch.submit(p, 3 + i) for i, p in enumerate(prompts)]
    finished = list(sch.run())
    assert sorted(map(id, finished)) == sorted(map(id, requests))
    for i, (p, r) in enumerate(zip(prompts, requests)):
        assert r.done and r.generated == _count(p, 3 + i)
    assert eng.live == {} and eng.most == 2 and max(n for _, n in eng.calls) <= 5


def test_scheduler_stop_token_and_limits():
    eng = CountingEngine(1)
    sch = Scheduler(eng, burst=4)
    want = _count([5, 6], 12)
    r = sch.submit([5, 6], 12, stop_token=want[5])
    list(sch.run())
    assert r.generated == want[:want.index(want[5]) + 1] and eng.live == {}
    for bad in (([], 1), ([1], 0), ([1] * 60, 6), ([97], 1), ([-1], 1)):
        with pytest.raises(ValueError):
            sch.submit(*bad)


# --------------------------------------------------------------------- trace --
def test_trace_replay(tmp_path):
    eng = CountingEngine(2)
    lines = [json.dumps({"step": 0, "entries": [{"id": "x", "tokens": [3, 4, 5], "want": [0, 2]}], "end": []}), "",
             json.dumps({"step": 1, "entries": [{"id": "x", "tokens": [6], "want": []}], "end": ["x"]}),
             json.dumps({"step": 2, "entries": [{"id": "y", "tokens": [9], "want": [0]}], "end": ["y"]})]
    said = []
    trace.replay(eng, io.StringIO("\n".join(lines)), str(tmp_path), said.append)
    assert said == ["done 0", "done 1", "done 2"] and eng.live == {}
    got = np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, 97)
    assert got.argmax(1).tolist() == [3, 12] and not (tmp_path / "1.f32").exists()
    assert np.fromfile(tmp_path / "2.f32", "<f4").argmax() == 9
