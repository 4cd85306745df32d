"""Host side of the latent-attention model and of the shared token loop: configuration, files, ring, feeding, trace
replay; and that the random models of the GPU tests would show the faults they look for. No GPU needed."""
import copy
import ctypes as C
import io
import json
import os
import re

import numpy as np
import pytest
import torch

import latent_cases as cases
from conftest import ROOT
from oracle import latent_lm as plain


# ---- library ---------------------------------------------------------------------
def test_dense_library_exports_every_declared_symbol():
    from llvq_b200 import _lib
    text = re.sub(r"/\*.*?\*/", "", open(os.path.join(ROOT, "include", "llvq_dense.h")).read(), flags=re.S)
    names = set(re.findall(r"\b(llvq_dn_[a-z0-9_]+)\s*\(", text))
    L = _lib.load_dense()
    assert names == set(_lib._DENSE_SIGNATURES)
    for n in names:
        assert hasattr(L, n)


def test_bad_arguments_are_refused_without_a_gpu():
    from llvq_b200 import _lib
    L = _lib.load_dense()
    bad = _lib.ERR_INVALID
    assert L.llvq_dn_gemv(None, None) == bad
    d = _lib.DenseGemv(dtype=_lib.DN_BF16, n_out=4, k=10, ldw=10, w=16, y=16, x=16)
    assert L.llvq_dn_gemv(C.byref(d), None) == bad and b"multiple of 8" in L.llvq_dn_last_error()
    d.ldw, d.prologue = 16, 9
    assert L.llvq_dn_gemv(C.byref(d), None) == bad and b"prologue" in L.llvq_dn_last_error()
    d.prologue, d.x, d.norm_w, d.a_out = _lib.DN_NORM, 32, 16, 32
    assert L.llvq_dn_gemv(C.byref(d), None) == bad  # the normed stream may not go where the stream is read from
    a = _lib.DenseLatent(dtype=_lib.DN_F32, heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=16, ldk=16, slots=8, ld=20, rot_dims=3, window=9, splits=1,
                         ring=16, cos_t=16, sin_t=16, uk=16, uv=16, qlat=16, part=16)
    assert L.llvq_dn_latent_decode(C.byref(a), 16, None) == bad and b"rotated" in L.llvq_dn_last_error()
    a.rot_dims = 4
    assert L.llvq_dn_latent_decode(C.byref(a), 16, None) == bad and b"window of 9 over 8" in L.llvq_dn_last_error()
    assert L.llvq_dn_latent_prefill(C.byref(a), 16, 16, 32, 16, 4, None, 0, 4, 4, 5, 2, 16, 0, None) == bad  # query 8 has no key
    assert L.llvq_dn_latent_prefill(C.byref(a), 16, 16, 32, 16, 4, 16, 8, 4, 4, 2, 2, 16, 0, None) == bad  # no transposed values in f32
    assert L.llvq_dn_latent_prefill_transposes(C.byref(a), 500) == 0
    assert L.llvq_dn_latent_rows(C.byref(a), 16, 64, 8, 16, 16, 0, 9, 0, None) == bad  # nine rows into eight slots
    assert L.llvq_dn_softcap(16, 4, 0.0, None) == bad
    with pytest.raises(_lib.LlvqError):
        _lib.check_dense(bad)


# ---- configuration and files -----------------------------------------------------
def test_configuration_is_read_as_written():
    from llvq_b200.latent import LatentConfig
    c = LatentConfig.parse(cases.UNEVEN)
    assert (c.width, c.vocab, c.alpha, c.softcap, c.eps, c.embed_scale) == (90, 203, 1.2, 7.0, 1e-3, 2.5)
    a = c.layers[1].attn
    assert (a.heads, a.dim, a.rot_dim, a.vdim, a.q_rank, a.kv_rank, a.window, a.rot_base, a.rot_dims) == (5, 17, 6, 9, 21, 30, 7, 500.0, 6)
    assert c.layers[2].attn.kv_from == 0 and c.layers[2].mlp is None and c.layers[3].mlp.limit == 2.5
    d = copy.deepcopy(cases.UNEVEN)
    d["logit_softcap"] = None
    del d["layers"][0]["mixer"]["mask"]
    assert LatentConfig.parse(d).softcap is None and LatentConfig.parse(d).layers[0].attn.window is None


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][2]["mixer"].update(kv_from=2), lambda c: c["layers"][2]["mixer"].update(kv_from=3),
    lambda c: c["layers"][3]["mixer"].update(kv_from=2), lambda c: c["layers"][2]["mixer"].update(kv_rank=55),
    lambda c: c["layers"][2]["mixer"]["rot"].update(base=9.0), lambda c: c["layers"][0].update(type="other"),
    lambda c: c["layers"][0]["mlp"].update(kind="routed"), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), lambda c: c.update(layers=[])])
def test_configurations_outside_the_design_are_refused(change):
    from llvq_b200.latent import LatentConfig
    c = copy.deepcopy(cases.UNEVEN)
    change(c)
    with pytest.raises(ValueError):
        LatentConfig.parse(c)


def test_registry_finds_the_class_by_config(tmp_path):
    from llvq_b200 import registry
    assert registry.architecture_of({"architecture": "Bikelix"}).dtypes == ("bfloat16", "float32")
    assert registry.architecture_of({"architectures": ["Qwen3ForCausalLM"]}).container == "archive"
    assert registry.architecture_of({"model_type": "qwen3"}).name == "qwen3"
    with pytest.raises(ValueError, match="no known architecture"):
        registry.architecture_of({"architecture": "Unheard"})
    p = cases.write_folder(tmp_path / "m", cases.EVEN, {"embed": torch.zeros(2, 2)})
    with pytest.raises(registry.UnsupportedDtype):
        registry.load_model(p, 16, "float16")
    q = cases.write_folder(tmp_path / "q", {"model_type": "qwen3"}, {"embed": torch.zeros(2, 2)})
    with pytest.raises(ValueError, match="served from a archive"):
        registry.load_model(q, 16)


def test_safetensors_round_trip_and_refusals(tmp_path):
    from llvq_b200.safetensors import SafetensorsFile, write_safetensors
    p = str(tmp_path / "a.safetensors")
    want = {"w": torch.randn(5, 3).bfloat16(), "i": torch.arange(7, dtype=torch.int32), "f": torch.randn(2, 2, 2), "none": torch.zeros(0, 4)}
    write_safetensors(p, want)
    f = SafetensorsFile(p)
    assert sorted(f.names()) == sorted(want) and "w" in f and "x" not in f
    for k, t in want.items():
        got = f.tensor(k)
        assert got.dtype == t.dtype and torch.equal(got, t)
    with pytest.raises(KeyError):
        f.tensor("x")
    raw = open(p, "rb").read()
    open(p, "wb").write(raw[:-3])
    with pytest.raises(ValueError):
        SafetensorsFile(p)
    open(p, "wb").write((10 ** 6).to_bytes(8, "little") + raw[8:])
    with pytest.raises(ValueError):
        SafetensorsFile(p)


# ---- ring ------------------------------------------------------------------------
@pytest.mark.parametrize("window,portion,capacity", [(1, 1, 50), (7, 1, 50), (7, 5, 50), (40, 30, 50), (1, 64, 50)])
def test_ring_holds_what_a_window_and_a_portion_can_see(window, portion, capacity):
    from llvq_b200.cache import LatentRing
    r = LatentRing(capacity, window, portion, 3, 2, torch.float32, "cpu")
    assert r.slots == min(capacity, window - 1 + portion) and r.ld == 8
    rng = np.random.default_rng(3)
    for _ in range(2):  # a second sequence in the same slots
        end = 0
        while end < capacity:
            n = int(rng.integers(1, portion + 1))
            n = min(n, capacity - end)
            for p in range(end, end + n):
                r.rows[p % r.slots] = float(p)
            end += n
            lo = max(0, end - n - window + 1)
            assert r.read(lo, end)[:, 0].tolist() == [float(p) for p in range(lo, end)]
    with pytest.raises(ValueError):
        r.read(0, r.slots + 1)


# ---- the shared loop and trace replay ---------------------------------------------
class Tally:
    """A model whose logits spell out what it was given: row p of a sequence is [p, sum of the tokens up to p, ...]."""

    def __new__(cls, capacity=40, chunk=6):
        from llvq_b200.token_loop import TokenLoop

        class T(TokenLoop):
            def __init__(self):
                self._init_loop(torch.device("cpu"), capacity, chunk)
                self.cache = torch.full((capacity,), -1)
                self.calls = []

            def _row(self, p):
                return [float(p), float(self.cache[:p + 1].sum()), 0.0]

            def hidden(self, tokens, pos, end):
                assert pos.tolist() == list(range(end - len(tokens), end))
                self.calls.append(("portion", len(tokens)))
                self.cache[pos] = tokens
                return torch.tensor([self._row(int(p)) for p in pos])

            def logits(self, x):
                return x

            def pick_last(self, x):
                return (x[-1, 1] % 7).long().reshape(1)

            def _eager_step(self):
                self.calls.append(("step", 1))
                p = int(self._pos)
                self.cache[p] = int(self._tok)
                self.last = torch.tensor(self._row(p))
                self._tok.copy_(self.pick_last(self.last[None]))
                self._pos += 1

            def _graph_step(self):
                self._eager_step()

            def step_logits(self):
                return self.last.clone()
        return T()


def test_feed_runs_only_what_it_is_given_and_generate_uses_the_same_steps():
    m = Tally()
    toks = [3, 5, 0, 2, 6, 1, 4, 4, 2, 6, 6, 1, 0]
    whole = m.feed(toks, list(range(13)))
    assert m.calls == [("portion", 6), ("portion", 6), ("portion", 1)]
    m.release()
    m.calls.clear()
    parts, at = [], 0
    for n in (1, 2, 7, 1, 1, 1):
        parts.append(m.feed(toks[at:at + n], list(range(n))))
        at += n
    assert torch.equal(torch.cat(parts), whole) and m.length == 13
    assert m.calls == [("step", 1), ("portion", 2), ("portion", 6), ("portion", 1), ("step", 1), ("step", 1), ("step", 1)]
    assert torch.equal(m.feed([1, 1, 1], [2, 0])[0], torch.tensor([15.0, float(sum(toks) + 3), 0.0]))  # the order asked for
    assert m.feed([1]) is None
    for bad in (lambda: m.feed([]), lambda: m.feed([1], [1]), lambda: m.feed([0] * 40)):
        with pytest.raises(ValueError):
            bad()
    out = m.generate(toks, 5)
    m2 = Tally()
    y = m2.feed(toks, [12])
    want = [int(m2.pick_last(y))]
    while len(want) < 5:
        want.append(int(m2.pick_last(m2.feed(want[-1:], [0]))))
    assert out == want


def test_trace_replay_writes_what_each_step_asks_for(tmp_path):
    from llvq_b200 import trace
    m, out = Tally(), io.StringIO()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [4], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [5], "want": [0]}], "end": ["b"]}]
    trace.run(m, [json.dumps(s) + "\n" for s in steps] + ["\n"], str(tmp_path), out)
    assert out.getvalue().split("\n") == ["done 0", "done 1", "done 2", ""]
    assert np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, 3).tolist() == [[2.0, 6.0, 0.0], [0.0, 1.0, 0.0]]
    assert not (tmp_path / "1.f32").exists()
    assert np.fromfile(tmp_path / "2.f32", "<f4").tolist() == [0.0, 5.0, 0.0]
    with pytest.raises(ValueError, match="holds the cache"):
        trace.run(m, [json.dumps({"step": k, "entries": [{"id": i, "tokens": [1], "want": []}], "end": []}) for k, i in enumerate("ab")], str(tmp_path), out)


def test_trace_runner_refuses_an_element_type_with_exit_code_3(tmp_path):
    from llvq_b200 import trace
    p = cases.write_folder(tmp_path / "m", cases.EVEN, {"embed": torch.zeros(2, 2)})
    assert trace.main(["--model", p, "--dtype", "float16", "--out", str(tmp_path)]) == 3


# ---- the plain implementation -----------------------------------------------------
def test_window_counts_the_position_itself():
    v = plain.window_mask(6, 3)
    assert v[5].tolist() == [False, False, False, True, True, True] and v[0].tolist() == [True] + [False] * 5
    assert plain.window_mask(6, None)[4].tolist() == [True] * 5 + [False]


def test_sink_takes_its_share_once():
    s = torch.zeros(1, 2, 2, dtype=torch.float64)
    p = plain.softmax_with_sink(s, plain.window_mask(2, 2), torch.tensor([np.log(3.0)]))
    assert torch.allclose(p[0], torch.tensor([[0.25, 0.0], [0.2, 0.2]], dtype=torch.float64))
    p = plain.softmax_with_sink(s, plain.window_mask(2, 2), None)
    assert torch.allclose(p[0, 1], torch.tensor([0.5, 0.5], dtype=torch.float64))


def test_rotation_keeps_relative_positions_and_passes_the_rest():
    x = torch.randn(9, 10, dtype=torch.float64)
    pos = torch.arange(9)
    r = plain.rotate(x[:1].expand(9, 10), pos, 6, 100.0)
    assert torch.equal(r[:, 6:], x[:1, 6:].expand(9, 4)) and torch.allclose(r[0], x[0])
    k = plain.rotate(x[1:2].expand(9, 10), pos, 6, 100.0)
    d = r[:, :6] @ k[:, :6].T
    assert torch.allclose(torch.diagonal(d, 2), d[0, 2].expand(7)) and torch.allclose(torch.diagonal(d, -3), d[3, 0].expand(6))
    assert abs(float(r[1, 0]) - float(x[0, 0] * np.cos(1) - x[0, 3] * np.sin(1))) < 1e-12


def _faults():
    def layer(i, **kw):
        return lambda c: c["layers"][i]["mixer"].update(**kw)
    yield "window one wider", layer(0, mask={"size": 20})
    yield "window one narrower", layer(0, mask={"size": 18})
    yield "shared cache with the owner's window", layer(2, mask={"size": 19})
    yield "window of one as two", layer(3, mask={"size": 2})
    yield "rotation base", layer(1, rot={"base": 10000.0, "dims": 6})
    yield "score scale", layer(0, scale=32 ** -0.5 * 1.05)
    yield "alpha", lambda c: c.update(postln_alpha=1.15)
    yield "soft cap", lambda c: c.update(logit_softcap=None)
    yield "embedding scale", lambda c: c["embedding"].update(scale=1.0)
    yield "eps", lambda c: c["norm"].update(eps=1e-5)
    yield "unit limit", lambda c: c["layers"][1]["mlp"].update(limit=2.5)


@pytest.mark.parametrize("name,fault", list(_faults()), ids=[n for n, _ in _faults()])
def test_the_random_models_show_a_planted_fault(name, fault):
    """Faults planted in the plain implementation move its logits by far more than the GPU tests' f32 tolerance."""
    w = plain.random_model(cases.UNEVEN, 11)
    toks = torch.randint(0, 203, (60,), generator=torch.Generator().manual_seed(4)).tolist()
    good = plain.forward(cases.UNEVEN, w, toks)
    c = copy.deepcopy(cases.UNEVEN)
    fault(c)
    bad = plain.forward(c, w, toks)
    assert ((bad - good)[-1].norm() / good[-1].norm()).item() > 50 * 3e-5, name


def test_the_random_models_show_a_missing_sink_or_bias():
    w = plain.random_model(cases.UNEVEN, 11)
    toks = list(range(50))
    good = plain.forward(cases.UNEVEN, w, toks)
    for name in ("l0.mix.sink", "l4.mix.sink", "l1.mlp.up.b", "l0.mlp.down.b", "l0.norm2", "l2.norm1", "l1.mix.dkv.norm", "l3.mix.dq.norm", "final.norm"):
        bad = dict(w)
        if name.endswith("sink"):
            bad[name] = torch.full_like(w[name], -1e4)
        else:
            bad[name] = torch.ones_like(w[name]) if name.endswith("dq.norm") or name.endswith("dkv.norm") else torch.zeros_like(w[name])
        y = plain.forward(cases.UNEVEN, bad, toks)
        assert ((y - good).norm() / good.norm()).item() > 50 * 3e-5, name
