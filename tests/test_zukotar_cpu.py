"""CPU tests of the Zukotar design's parts that need no GPU: configuration, weight layout, layer runs and their state; and of
the oracle: each mechanism against its closed form, and that a mechanism that is off by one shows in the logits of the
test models."""
import copy
import math

import numpy as np
import pytest
import torch

import zukotar_cases as cases
from oracle import zukotar_ref as ref
from tensorwarp_b200 import checkpoint, dense, registry
from tensorwarp_b200.models import zukotar
from tensorwarp_b200.state import SequenceState


# ------------------------------------------------------------------- oracle --
def test_oracle_mechanisms_closed_forms():
    assert np.allclose(ref.rms_norm(np.array([[3.0, 4.0]]), np.array([1.0, 2.0]), 0.0), [[3 / math.sqrt(12.5), 8 / math.sqrt(12.5)]])
    assert np.allclose(ref.sigmoid(np.array([0.0, 800.0, -800.0])), [0.5, 1.0, 0.0])
    assert np.allclose(ref.softmax(np.array([1000.0, 1000.0 + math.log(3)])), [0.25, 0.75])
    assert ref.squared_relu(np.array([-2.0, 3.0])).tolist() == [0.0, 9.0]
    assert np.allclose(ref.silu(np.array([0.0, 40.0])), [0.0, 40.0])
    m = ref.visible(6, 2)
    assert m[5].tolist() == [False] * 4 + [True] * 2 and m[0].tolist() == [True] + [False] * 5
    assert np.array_equal(ref.visible(5, None), np.tril(np.ones((5, 5), bool)))
    x = ref.rotate(np.array([[1.0, 0.0, 0.0, 2.0]]), np.array([3.0]), 100.0)
    assert np.allclose(x, [[math.cos(3), math.sin(3), -2 * math.sin(0.3), 2 * math.cos(0.3)]])
    both = ref.rotate(np.random.default_rng(0).standard_normal((2, 8)), np.array([5.0, 9.0]), 50.0)
    far = ref.rotate(np.random.default_rng(0).standard_normal((2, 8)), np.array([105.0, 109.0]), 50.0)
    assert abs(both[0] @ both[1] - far[0] @ far[1]) < 1e-9      # a product of rotated vectors knows the distance only


def test_oracle_decay_and_recurrence_by_hand():
    w = {"x.a1": np.array([[2.0]]), "x.a2": np.array([[1.0], [-3.0]]), "x.a2.b": np.array([0.5, 1.0])}
    a = ref.decays(np.array([[0.25]]), w, "x.", 4.0)
    assert np.allclose(a, [[ref.sigmoid(np.array(1.0)) ** 0.25, ref.sigmoid(np.array(-0.5)) ** 0.25]])
    q = np.array([[[1.0, 1.0]], [[1.0, 2.0]]])
    k = np.array([[[1.0, 0.5]], [[3.0, 0.0]]])
    v = np.array([[[2.0]], [[10.0]]])
    alpha = np.array([[[0.5, 0.5]], [[0.25, 0.5]]])
    o, s = ref.recurrence(q, k, v, alpha)
    assert np.allclose(o[:, 0, 0], [3.0, (0.5 + 30.0) + 2 * 0.5]) and np.allclose(s[0, :, 0], [30.5, 0.5])


def test_oracle_router_by_hand():
    z = np.log(np.array([0.30, 0.02, 0.25, 0.20, 0.05, 0.18]))
    chosen, weight = ref.route(z, 2, {"count": 3, "keep": 1})          # the best group has the best single expert: 0 and 1
    assert chosen.tolist() == [0, 1] and np.allclose(weight, [0.30, 0.02])
    chosen, weight = ref.route(z, 3, {"count": 3, "keep": 2})
    assert chosen.tolist() == [0, 2, 3] and np.allclose(weight, [0.30, 0.25, 0.20])
    assert ref.route(z, 3, None)[0].tolist() == [0, 2, 3]


def test_oracle_layer_runs():
    cfg = {"layers": [0] * 5, "loop": {"start": 1, "stop": 3, "times": 2}}
    assert ref.layer_runs(cfg) == [(0, None), (1, 0), (2, 0), (1, 1), (2, 1), (3, None), (4, None)]


@pytest.mark.parametrize("case", sorted(cases.CASES))
def test_planted_mistakes_show(case, monkeypatch):
    """Every mechanism moved by one, dropped or changed in the oracle moves the logits by far more than the tolerances of
    the GPU tests (2e-5 in 32-bit)."""
    cfg, w = cases.CASES[case], cases.as_float64(cases.weights(cases.CASES[case], 11, cases.RANKS[case]))
    toks = cases.tokens(cfg, 150, 5)
    base = ref.forward(cfg, w, toks)

    def moved(change_cfg=None, change_w=None):
        c, ww = copy.deepcopy(cfg), dict(w)
        if change_cfg:
            change_cfg(c)
        if change_w:
            change_w(ww)
        return float(cases.error(ref.forward(c, ww, toks), base).max())

    def mixers(kind, change):
        def f(c):
            for lay in c["layers"]:
                if lay["type"] == kind:
                    change(lay["mixer"])
        return f

    def fill(suffix, value):
        return lambda ww: ww.update({k: np.full_like(v, value) for k, v in ww.items() if k.endswith(suffix)})

    def window(by):
        def change(m):
            if "mask" in m:
                m["mask"]["size"] += by
        return change

    assert moved(mixers("latent_attention", window(1))) > 2e-3
    assert moved(mixers("latent_attention", window(-1))) > 2e-3
    assert moved(mixers("latent_attention", lambda m: m.__setitem__("scale", m["scale"] * 1.05))) > 2e-3
    assert moved(mixers("latent_attention", lambda m: m["rot"].__setitem__("base", m["rot"]["base"] * 2))) > 2e-3
    assert moved(mixers("gla", lambda m: m.__setitem__("tau", m["tau"] * 1.1))) > 2e-3
    assert moved(lambda c: c["embedding"].__setitem__("scale", c["embedding"]["scale"] * 1.1)) > 2e-3
    assert moved(lambda c: c["loop"].__setitem__("times", c["loop"]["times"] - 1)) > 2e-3
    for name, value in (("mix.g", 0.0), ("dkv.norm", 1.0), ("mix.norm", 1.0), ("a2.b", 2.0), ("norm1", 1.0), ("norm1b", 1.0), ("norm2", 1.0),
                        ("norm2b", 1.0), ("loop.step", 0.0), ("final.norm", 1.0), ("router", 0.0)):
        assert moved(change_w=fill(name, value)) > 2e-3, name
    plain = ref.route
    if case == "uneven":
        monkeypatch.setattr(ref, "route", lambda z, top, groups: plain(z, top, None))
        assert moved() > 2e-3
    monkeypatch.setattr(ref, "route", plain)
    rec = ref.recurrence

    def lost_state(q, k, v, alpha, state=None):
        first, _ = rec(q[:70], k[:70], v[:70], alpha[:70])
        return np.concatenate([first, rec(q[70:], k[70:], v[70:], alpha[70:])[0]]), None

    monkeypatch.setattr(ref, "recurrence", lost_state)
    assert moved() > 2e-3


# ------------------------------------------------------------ configuration --
def test_config_is_read_layer_by_layer():
    s = cases.spec(cases.UNEVEN, 5)
    assert (s.vocab, s.width, s.eps, s.max_positions, s.embed_scale) == (131, 52, 3e-4, None, 3.0)
    assert s.layers[0].mixer == dense.GatedLinearSpec(3, 20, 36, 4.0, 5)
    assert s.layers[1].mixer == dense.LatentAttentionSpec(5, 24, 6, 10000.0, 40, 37, 0.3, 9)
    assert s.layers[3].mixer.window >= 1 << 20 and s.layers[3].mixer.rot_base == 500.0
    assert s.layers[0].ff == dense.RoutedSpec(10, 4, 24, 5, 3) and s.layers[2].ff is None
    assert s.layers[3].ff == dense.RoutedSpec(7, 3, 9, 1, 1)
    assert s.runs() == [(0, 0), (1, None), (0, 1), (1, None), (2, None), (3, None)]
    shapes = zukotar.tensor_shapes(s)
    assert shapes["l0.mix.a2"] == (60, 5) and shapes["l1.mix.dkv"] == (43, 52) and shapes["l1.mix.g"] == (5, 52)
    assert shapes["l3.mlp.e6.down"] == (52, 9) and shapes["loop.step"] == (2, 52) and "head" not in shapes
    assert "l2.norm2" not in shapes and "l2.mlp.router" not in shapes and "l2.norm1b" in shapes
    no_loop = dict(cases.UNEVEN, loop=None)
    assert cases.spec(no_loop, 5).runs() == [(i, None) for i in range(4)] and "loop.step" not in zukotar.tensor_shapes(cases.spec(no_loop, 5))


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].__setitem__("type", "other"),
    lambda c: c["layers"][0]["mixer"].__setitem__("unheard_of", 1),
    lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("unheard_of", 1),
    lambda c: c["layers"][1]["mixer"].__setitem__("rot_dim", 5),
    lambda c: c["layers"][1]["mixer"]["mask"].__setitem__("size", 0),
    lambda c: c["layers"][0]["mlp"].__setitem__("kind", "other"),
    lambda c: c["layers"][0]["mlp"]["router"]["groups"].__setitem__("count", 3),
    lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 7),
    lambda c: c["loop"].__setitem__("stop", 9),
])
def test_what_the_design_does_not_have_is_refused(change):
    cfg = copy.deepcopy(cases.UNEVEN)
    change(cfg)
    with pytest.raises(checkpoint.CheckpointError):
        cases.spec(cfg, 5)


def test_registry_and_rank_from_the_checkpoint(tmp_path):
    assert registry.builder_for(cases.UNEVEN) is zukotar.build
    cases.save(str(tmp_path), cases.UNEVEN, cases.weights(cases.UNEVEN, 1, 5))
    f = checkpoint.SafetensorsFile(str(tmp_path / "model.safetensors"))
    assert zukotar.parse_config(cases.UNEVEN, f.shape).layers[2].mixer.rank == 5
    with pytest.raises(checkpoint.CheckpointError, match="missing"):
        f.shape("nothing")


# ------------------------------------------------------------- weight layout --
@pytest.mark.parametrize("case", sorted(cases.CASES))
def test_padded_fused_weights_compute_the_same(case):
    cfg, rank = cases.CASES[case], cases.RANKS[case]
    tensors = cases.weights(cfg, 3, rank)
    model = cases.model(cfg, tensors, rank, torch.float32, "cpu")
    plain = {k: v.double() for k, v in tensors.items()}
    spec, pad = model.spec, dense.pad16
    x = torch.randn(3, spec.width, dtype=torch.float64)
    xp = torch.zeros(3, model.width_pad, dtype=torch.float64)
    xp[:, :spec.width] = x
    assert model.head is model.embed

    def heads(part, n, want):
        """the part's padded heads hold `want` and zeros"""
        part, want = part.reshape(3, n, -1), want.reshape(3, n, -1)
        assert torch.allclose(part[:, :, :want.shape[2]], want, atol=1e-5) and bool((part[:, :, want.shape[2]:] == 0).all())

    for i, (lay, w) in enumerate(zip(spec.layers, model.layers)):
        m, p = lay.mixer, f"l{i}.mix."
        y = xp @ w["w_in"].double().T
        if isinstance(m, dense.LatentAttentionSpec):
            dp, rp, kp, vp = pad(m.dim), pad(m.rot_dim), pad(m.rank), pad(m.vdim)
            q, c, kr, g = torch.split(y, [m.heads * (dp + rp), kp, rp, pad(m.heads)], dim=1)
            q, want = q.reshape(3, m.heads, -1), (x @ plain[p + "q"].T).reshape(3, m.heads, -1)
            heads(q[:, :, :dp], m.heads, want[:, :, :m.dim])
            heads(q[:, :, dp:], m.heads, want[:, :, m.dim:])
            down = x @ plain[p + "dkv"].T
            heads(c, 1, down[:, :m.rank])
            heads(kr, 1, down[:, m.rank:])
            heads(g, 1, x @ plain[p + "g"].T)
            lat = torch.randn(3, m.rank, dtype=torch.float64)
            kv = torch.nn.functional.pad(lat, (0, kp - m.rank)) @ w["w_expand"].double().T
            heads(kv[:, :m.heads * dp], m.heads, lat @ plain[p + "uk"].T)
            heads(kv[:, m.heads * dp:], m.heads, lat @ plain[p + "uv"].T)
        else:
            dp, vp, lp = pad(m.dim), pad(m.vdim), pad(m.rank)
            parts = torch.split(y, [m.heads * dp, m.heads * dp, m.heads * vp, m.heads * vp, lp], dim=1)
            for part, name in zip(parts[:4], "qkvg"):
                heads(part, m.heads, x @ plain[p + name].T)
            low = x @ plain[p + "a1"].T
            heads(parts[4], 1, low)
            heads(parts[4] @ w["w_decay"].double().T, m.heads, low @ plain[p + "a2"].T)
            heads(w["decay_bias"].double().expand(3, -1), m.heads, plain[p + "a2.b"].expand(3, -1))
        o = torch.randn(3, m.heads, pad(m.vdim), dtype=torch.float64)
        assert torch.allclose(o.reshape(3, -1) @ w["w_out"].double().T, o[:, :, :m.vdim].reshape(3, -1) @ plain[p + "o"].T, atol=1e-5)
        if lay.ff is not None:
            e = lay.ff.experts - 1
            up = xp @ w["w_gate_up"][e].double().T
            heads(up, 1, x @ plain[f"l{i}.mlp.e{e}.up"].T)
            heads(up @ w["w_down"][e].double().T, 1, (x @ plain[f"l{i}.mlp.e{e}.up"].T) @ plain[f"l{i}.mlp.e{e}.down"].T)


def test_rotation_table():
    t = dense.rotation_table(500.0, 6, 40, "cpu").double()
    assert t.shape == (40, 8, 2)
    for p, i in ((0, 0), (7, 1), (39, 2)):
        a = p * 500.0 ** (-2 * i / 6)
        assert abs(float(t[p, i, 0]) - math.cos(a)) < 1e-7 and abs(float(t[p, i, 1]) - math.sin(a)) < 1e-7
    assert bool((t[:, 3:, 0] == 1).all()) and bool((t[:, 3:, 1] == 0).all())


# --------------------------------------------------------------------- state --
def test_every_pass_has_a_state_of_its_own():
    model = cases.model(cases.UNEVEN, cases.weights(cases.UNEVEN, 1, 5), 5, torch.bfloat16, "cpu")
    st = SequenceState(model, slots=2, capacity=10)
    assert [sorted(r) for r in st.runs] == [["gla_state"], ["latent_cache"], ["gla_state"], ["latent_cache"], ["gla_state"], ["latent_cache"]]
    assert st.runs[0]["gla_state"].shape == (2, 3, 32, 48) and st.runs[0]["gla_state"].dtype == torch.float32
    assert st.runs[1]["latent_cache"].shape == (2, 10, 48 + 16) and st.runs[1]["latent_cache"].dtype == torch.bfloat16
    ptrs = [t.data_ptr() for r in st.runs for t in r.values()]
    assert len(set(ptrs)) == len(ptrs) and st.bytes() > 0
    d = model.descriptor(st)
    assert d.n_layers == 6 and d.layers[0].w_in == d.layers[2].w_in and d.layers[0].gla_state != d.layers[2].gla_state
    assert d.layers[0].step and d.layers[2].step and d.layers[0].step != d.layers[2].step and not d.layers[1].step
    assert d.layers[1].rot_table == d.layers[3].rot_table != d.layers[5].rot_table
