"""Host side of the hybrid model: configuration, states, refusals; the plain implementation itself; and that the random
models of the GPU tests would show the faults they look for. No GPU needed."""
import copy
import ctypes as C

import pytest
import torch

import hybrid_cases as cases
from oracle import hybrid_lm as plain


# ---- configuration -------------------------------------------------------------------
def test_configuration_is_read_as_written():
    from llvq_b200.hybrid import DeltaConfig, HybridConfig, ParallelConfig
    c = HybridConfig.parse(cases.UNEVEN)
    assert (c.width, c.vocab, c.eps) == (90, 203, 1e-3) and c.runs == (0, 1, 2, 3, 1, 2, 3, 4)
    p = c.layers[1].mixer
    assert isinstance(p, ParallelConfig) and (p.left_scale, p.right_scale) == (0.7, 1.3)
    assert (p.left.heads, p.left.kv_heads, p.left.dim, p.left.vdim, p.left.scale, p.left.window) == (6, 2, 13, 9, 0.5, 19)
    assert (p.right.width, p.right.blocks, p.right.taps) == (42, 3, 3) and c.layers[1].mlp is None
    d = c.layers[0].mixer
    assert isinstance(d, DeltaConfig) and (d.heads, d.kv_heads, d.dim, d.vdim, d.taps, d.channels) == (3, 1, 11, 7, 2, 43)
    assert (c.layers[0].mlp.ff, c.layers[0].mlp.experts, c.layers[0].mlp.top) == (21, 5, 3) and c.layers[3].mlp.experts == 0
    e = copy.deepcopy(cases.UNEVEN)
    del e["loop"]
    e["layers"][1]["mixer"]["left"]["mask"] = None
    assert HybridConfig.parse(e).runs == (0, 1, 2, 3, 4) and HybridConfig.parse(e).layers[1].mixer.left.window is None


@pytest.mark.parametrize("loop,runs", [(None, (0, 1, 2)), ({"start": 0, "stop": 3, "times": 1}, (0, 1, 2)), ({"start": 0, "stop": 2, "times": 2}, (0, 1, 0, 1, 2)),
                                       ({"start": 1, "stop": 2, "times": 3}, (0, 1, 1, 1, 2)), ({"start": 1, "stop": 3, "times": 2}, (0, 1, 2, 1, 2))])
def test_order_of_layer_runs(loop, runs):
    from llvq_b200.hybrid import HybridConfig
    assert HybridConfig.order(3, loop) == runs
    assert tuple(plain.layer_runs({"layers": [0] * 3, "loop": loop})) == runs


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="shared"), lambda c: c["layers"][0]["mixer"].update(kv_heads=2),
    lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0),
    lambda c: c["layers"][1]["mixer"]["right"].update(blocks=4), lambda c: c["layers"][1]["mixer"]["right"].update(conv=0),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=6), lambda c: c["layers"][0]["mlp"]["router"].update(top=0), lambda c: c["layers"][3]["mlp"].update(ff=0),
    lambda c: c["loop"].update(stop=6), lambda c: c["loop"].update(times=0), lambda c: c["loop"].update(start=4), lambda c: c.update(layers=[])])
def test_configurations_outside_the_design_are_refused(change):
    from llvq_b200.hybrid import HybridConfig
    c = copy.deepcopy(cases.UNEVEN)
    change(c)
    with pytest.raises(ValueError):
        HybridConfig.parse(c)


def test_registry_knows_the_design():
    from llvq_b200 import registry
    a = registry.architecture_of({"architecture": "Dozusun"})
    assert (a.container, a.dtypes) == ("folder", ("bfloat16", "float32"))


# ---- matrices, routes, caches ------------------------------------------------------------
def test_matrices_side_by_side_are_one_product():
    from llvq_b200.dense import ColumnMatrix
    parts = [torch.randn(5, k) for k in (7, 8, 1)]
    m = ColumnMatrix(parts, torch.float32, "cpu")
    assert m.at == [0, 8, 16] and m.k == m.ld == 20 and m.padded
    a = torch.zeros(20)
    for lo, p in zip(m.at, parts):
        a[lo:lo + p.shape[1]] = torch.arange(p.shape[1]) + 1.0
    assert torch.allclose(m.rows(0) @ a, sum(p @ (torch.arange(p.shape[1]) + 1.0) for p in parts))
    assert not ColumnMatrix([torch.randn(5, 8)], torch.float32, "cpu").padded
    with pytest.raises(ValueError):
        ColumnMatrix([torch.randn(5, 3), torch.randn(4, 3)], torch.float32, "cpu")


def test_key_value_rows_and_their_transposed_values():
    from llvq_b200.cache import KvRing
    r = KvRing(50, 7, 5, 2, 3, 5, torch.bfloat16, "cpu")
    assert (r.slots, r.kd, r.vd, r.ld) == (11, 8, 8, 32)
    r.rows.copy_(torch.randn(11, 32))
    vt = r.values_transposed(r.read(20, 29))
    assert vt.shape == (10, 16) and not vt[:, 9:].any()
    for j in range(9):
        row = r.rows[(20 + j) % 11]
        assert torch.equal(vt[:, j], torch.cat([row[16:21], row[24:29]]))


def test_bad_arguments_are_refused_without_a_gpu():
    from llvq_b200 import _lib
    L, bad = _lib.load_dense(), _lib.ERR_INVALID
    d = _lib.DenseGemv(dtype=_lib.DN_BF16, prologue=_lib.DN_NORM, n_out=4, k=10, ldw=16, w=16, y=16, x=16, norm_w=16, rows2=3, w2=16, norm_w2=16, y2=16, glu2=1)
    assert L.llvq_dn_gemv(C.byref(d), None) == bad and b"second rows" in L.llvq_dn_last_error()
    d.rows2, d.prologue = 4, _lib.DN_PLAIN
    assert L.llvq_dn_gemv(C.byref(d), None) == bad
    d.rows2, d.w_r, d.k_r, d.ld_r, d.route, d.token, d.top, d.matrices, d.route_rows = 0, 16, 9, 9, 16, 16, 1, 2, 5
    assert L.llvq_dn_gemv(C.byref(d), None) == bad and b"routed columns" in L.llvq_dn_last_error()
    d.top = 0
    assert L.llvq_dn_gemv(C.byref(d), None) == bad and b"route" in L.llvq_dn_last_error()
    a = _lib.DenseGqa(dtype=_lib.DN_F32, heads=4, kv_heads=3, dim=8, vdim=8, slots=8, ld=32, kd=8, vd=8, window=9, splits=1, scale=1.0, ring=16)
    assert L.llvq_dn_mixer_token(C.byref(a), None, 16, None) == bad and b"4 heads over 3" in L.llvq_dn_last_error()
    a.kv_heads, a.q, a.k, a.v, a.q_norm, a.k_norm, a.part, a.arrived, a.out = 2, *[16] * 8
    assert L.llvq_dn_mixer_token(C.byref(a), None, 16, None) == bad and b"window of 9 over 8" in L.llvq_dn_last_error()
    a.window = 8
    assert L.llvq_dn_gqa_rows(C.byref(a), 16, 16, 16, 40, 16, 0, 9, None) == bad        # nine rows into eight slots
    assert L.llvq_dn_gqa_prefill(C.byref(a), 16, 16, None, 0, 4, 4, 5, 2, 16, 0, None) == bad  # query 8 has no key
    assert L.llvq_dn_mixer_token(None, None, 16, None) == bad
    r = _lib.DenseLru(dtype=_lib.DN_F32, blocks=2, n=3, taps=0, ldw=4)
    assert L.llvq_dn_mixer_token(None, C.byref(r), 16, None) == bad
    e = _lib.DenseDelta(dtype=_lib.DN_F32, heads=2, kv_heads=1, dim=8, vdim=6, vp=6, taps=4)
    assert L.llvq_dn_delta_token(C.byref(e), 16, None) == bad
    assert L.llvq_dn_conv_rows(_lib.DN_F32, 16, 3, None, 16, None, 16, 16, 4, 4, 0, 1, None) == bad
    assert L.llvq_dn_gated_rows(_lib.DN_F32, 16, None, 16, 3, 1, 4, 1.0, 1.0, 0.0, 1.0, None) == bad
    assert L.llvq_dn_route_rows(16, 5, 0, 3, 16, 4, 16, 16, 16, None) == bad
    assert L.llvq_dn_add_norms_rows(_lib.DN_F32, 16, None, None, None, 0, 16, None, None, None, 1e-5, 1, 4, None) == bad


# ---- the plain implementation -----------------------------------------------------------
def test_delta_rule_writes_before_it_reads_and_overwrites_a_key():
    k = torch.tensor([[[1.0, 0.0]], [[0.0, 1.0]], [[1.0, 0.0]]], dtype=torch.float64)
    v = torch.tensor([[[2.0]], [[3.0]], [[5.0]]], dtype=torch.float64)
    one = torch.ones(3, 1, dtype=torch.float64)
    o, S = plain.delta_rule(k, k, v, one, one)
    assert o.flatten().tolist() == [2.0, 3.0, 5.0] and S[0].flatten().tolist() == [5.0, 3.0]
    o, S = plain.delta_rule(k, k, v, 0.5 * one, one)
    assert o.flatten().tolist() == [1.0, 1.5, 3.0]
    o, S = plain.delta_rule(k, k, v, one, 0.5 * one)
    assert S[0].flatten().tolist() == [5.0, 1.5]


def test_convolution_is_causal_and_its_last_column_is_the_current_token():
    x = torch.zeros(6, 1, dtype=torch.float64)
    x[2] = 1.0
    assert plain.causal_conv(x, torch.tensor([[3.0, 2.0, 1.0]], dtype=torch.float64)).flatten().tolist() == [0.0, 0.0, 1.0, 2.0, 3.0, 0.0]


def test_recurrence_starts_from_zero_without_a_special_case():
    one = torch.ones(3, 1, dtype=torch.float64)
    lam = torch.tensor([0.3], dtype=torch.float64)
    a = float(torch.exp(-8.0 * 0.5 * plain.softplus(lam)))
    S = plain.gated_recurrence(one, 0.5 * one, 0.25 * one, lam).flatten()
    x = (1 - a * a) ** 0.5 * 0.25
    assert torch.allclose(S, torch.tensor([x, x + a * x, x + a * (x + a * x)], dtype=torch.float64))


def _faults():
    def left(i, **kw):
        return lambda c, w: c["layers"][i]["mixer"]["left"].update(**kw)

    def weight(name, fn):
        return lambda c, w: w.update({name: fn(w[name])})
    yield "window one wider", left(1, mask={"size": 20})
    yield "window one narrower", left(1, mask={"size": 18})
    yield "window of one as two", left(4, mask={"size": 2})
    yield "score scale", left(2, scale=20 ** -0.5 * 1.05)
    yield "loop once more", lambda c, w: c["loop"].update(times=3)
    yield "eps", lambda c, w: c["norm"].update(eps=1e-5)
    yield "left scale", lambda c, w: c["layers"][2]["mixer"].update(left_scale=1.0)
    yield "right scale", lambda c, w: c["layers"][1]["mixer"].update(right_scale=1.0)
    for name in ("l1.mix.right.conv.b", "l1.mix.right.x.b", "l2.mix.right.y.b", "l4.mix.right.ra.b", "l1.mix.right.ri.b", "l0.mix.dt_bias", "l3.mix.A_log", "l1.mix.left.g"):
        yield name + " left out", weight(name, torch.zeros_like)
    for name in ("l0.norm1", "l3.norm2", "l1.mix.left.q.norm", "l2.mix.left.k.norm", "l0.mix.norm", "final.norm"):
        yield name + " left out", weight(name, torch.ones_like)
    yield "taps reversed", weight("l3.mix.k.conv", lambda t: t.flip(1))
    yield "an oldest tap lost", weight("l3.mix.v.conv", lambda t: torch.cat([torch.zeros_like(t[:, :1]), t[:, 1:]], 1))
    yield "gates swapped", lambda c, w: w.update({"l1.mix.right.ra": w["l1.mix.right.ri"], "l1.mix.right.ri": w["l1.mix.right.ra"]})
    yield "gate matrix transposed", weight("l1.mix.right.ra", lambda t: t.transpose(1, 2))
    yield "experts of the next token id", weight("l0.mlp.table", lambda t: t.roll(1, 0))


@pytest.mark.parametrize("name,fault", list(_faults()), ids=[n for n, _ in _faults()])
def test_the_random_models_show_a_planted_fault(name, fault):
    """Faults planted in the plain implementation move its logits by far more than the GPU tests' f32 tolerance."""
    w = cases.random_model(cases.UNEVEN, 11)
    toks = torch.randint(0, 203, (60,), generator=torch.Generator().manual_seed(4)).tolist()
    good = plain.forward(cases.UNEVEN, w, toks)
    c, w = copy.deepcopy(cases.UNEVEN), dict(w)
    fault(c, w)
    bad = plain.forward(c, w, toks)
    assert ((bad - good)[-1].norm() / good[-1].norm()).item() > 20 * 3e-5, name


def test_the_random_models_show_a_state_lost_far_back():
    """What a token wrote 150 positions ago still moves the logits."""
    w = cases.random_model(cases.EVEN, 11)
    toks = torch.randint(0, 500, (200,), generator=torch.Generator().manual_seed(4)).tolist()
    other = list(toks)
    other[20] = (other[20] + 1) % 500
    a, b = plain.forward(cases.EVEN, w, toks), plain.forward(cases.EVEN, w, other)
    assert ((a - b)[-1].norm() / a[-1].norm()).item() > 20 * 3e-5
