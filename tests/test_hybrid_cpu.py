"""Configuration, registry, weight files and argument checks of the hybrid decoder: everything that needs no GPU, and the plain
statement's own consistency."""
import ctypes as C
import json

import numpy as np
import pytest

import ctorch_b200 as B
import hybrid_cases as H
import hybrid_oracle as O
from ctorch_b200 import trace


def host_model(c, dtype="bf16", weights=None):
    return B.LanguageModel(c, weights, dtype=dtype, device=None)


def test_registry_names_the_designs():
    assert B.architectures() == ["Lozepel", "Ripitar", "Rizovik", "Sinezen", "TransformerDecoder"]
    with pytest.raises(B.B200Error, match="unknown architecture 'Nothing'"):
        host_model({"architecture": "Nothing", "vocab": 4})


@pytest.mark.parametrize("name", H.CASES)
def test_parameters_follow_the_configuration(name):
    c = H.CASES[name]
    state = host_model(c).module.state()
    assert {n: t.shape for n, t in state.items()} == {n: tuple(s) for n, s in H.weight_shapes(c).items()}
    assert all(t.dtype == B.BF16 for t in state.values())


def broken(change):
    c = json.loads(json.dumps(H.CASES["mixed"]))
    change(c)
    return c


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][1].update(type="rnn"), "unknown layer type 'rnn'"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), r"layers\[1\]\.mixer\.state' is missing"),
    (lambda c: c["layers"][0]["mixer"].update(heads=2.5), r"heads' must be an integer"),
    (lambda c: c["layers"][0]["mixer"].update(heads=0), "must be a positive integer"),
    (lambda c: c["layers"][1]["mixer"].update(groups=3), "multiple of groups"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "multiple of norm_groups"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=12), "at most rot_dim"),
    (lambda c: c["layers"][2]["mlp"].update(kind="routed"), "unknown feed-forward kind 'routed'"),
    (lambda c: c["loop"].update(stop=5), "range of layers"),
    (lambda c: c.update(layers=[]), "at least one layer"),
    (lambda c: c.pop("logit_scale"), "'logit_scale' is missing"),
])
def test_configuration_errors_name_the_key(change, message):
    with pytest.raises(B.B200Error, match=message):
        host_model(broken(change))


def test_json_text_errors():
    out = C.c_void_p()
    for text in (b"{", b'{"a": 1,}', b'{"a": 01x}', b'[1, 2] 3', b'{"a" 1}', b'"\\q"'):
        assert B.lib().dl_model_create(text, B.options(B.BF16), C.byref(out)) == 1
        assert b"JSON" in B.lib().dl_last_error(), text


def test_weight_folder_round_trip(tmp_path):
    c = H.CASES["mixed"]
    w = H.make_weights(c, 3)
    H.write_folder(tmp_path, c, {**w, "table": np.arange(6).reshape(2, 3)})   # a tensor the design does not have is left alone
    model = B.LanguageModel.load(str(tmp_path), dtype="f32", device=None)
    for name, tensor in model.module.state().items():
        assert np.array_equal(tensor.numpy(), w[name]), name
    state = C.c_void_p()
    B.check(B.lib().dl_state_load_safetensors(str(tmp_path / "model.safetensors").encode(), C.byref(state)))
    names = [B.lib().dl_state_name(state, i).decode() for i in range(B.lib().dl_state_size(state))]
    t = C.c_void_p()
    B.check(B.lib().dl_state_tensor(state, names.index("table"), C.byref(t)))
    assert np.array_equal(B.Tensor(t).numpy(), np.arange(6).reshape(2, 3))
    B.lib().dl_state_release(state)


def test_damaged_weight_files_are_refused(tmp_path):
    c = H.CASES["ones"]
    w = H.make_weights(c)
    H.write_folder(tmp_path, c, w)
    path = tmp_path / "model.safetensors"
    good = path.read_bytes()
    for bad in (good[:-2], good[:40], b"\xff" * 8 + good[8:], good[:8] + b"x" + good[9:]):
        path.write_bytes(bad)
        with pytest.raises(B.B200Error):
            B.LanguageModel.load(str(tmp_path), device=None)
    del w["l0.mix.D"]
    H.write_folder(tmp_path, c, w)
    with pytest.raises(B.B200Error, match="l0.mix.D"):
        B.LanguageModel.load(str(tmp_path), device=None)
    w["l0.mix.D"] = np.ones(3)
    H.write_folder(tmp_path, c, w)
    with pytest.raises(B.B200Error, match="l0.mix.D"):
        B.LanguageModel.load(str(tmp_path), device=None)


def test_other_design_loads_through_the_same_registry(tmp_path):
    c = {"architecture": "TransformerDecoder", "vocab": 40, "layers": 1, "width": 16, "heads": 2, "kv_heads": 1, "ff": 24, "context": 32}
    names = [n for n in host_model(c).module.state_names() if "rotary" not in n]
    assert "tokens.weight" in names and "decoder.layer0.attention.query.weight" in names and "output.weight" not in names
    shapes = {n: t.shape for n, t in host_model(c).module.state().items()}
    H.write_folder(tmp_path, c, {n: np.random.default_rng(0).normal(size=shapes[n]) for n in names})
    assert B.LanguageModel.load(str(tmp_path), device=None).vocab == 40


def test_no_cpu_compute_path():
    model = host_model(H.CASES["ones"])
    with pytest.raises(B.B200Error, match="no CPU compute path"):
        model.new_cache(1, 8)


class FakeModel:
    """Records what the trace replay asks of a model."""
    vocab = 7

    def __init__(self):
        self.log, self.cache = [], None

    def new_cache(self, slots, capacity):
        self.cache = self
        self.log.append(("cache", slots, capacity))

    def release(self, slot):
        self.log.append(("release", slot))

    def run(self, entries):
        self.log.append(("run", [(s, list(t)) for s, t, _ in entries]))
        return np.zeros((sum(len(w) for _, _, w in entries), self.vocab), dtype=np.float32)


def test_trace_replay_assigns_and_returns_slots():
    model = FakeModel()
    replay = trace.Replay(model, 50)
    assert replay.step([{"id": "a", "tokens": [1, 2], "want": [1]}, {"id": "b", "tokens": [3], "want": []}], []).shape == (1, 7)
    replay.step([{"id": "b", "tokens": [4], "want": [0]}, {"id": "a", "tokens": [5], "want": [0]}], ["a"])
    with pytest.raises(ValueError):
        replay.step([{"id": "c", "tokens": [1], "want": []}, {"id": "d", "tokens": [1], "want": []}], [])
    replay.step([{"id": "b", "tokens": [6], "want": []}], ["b"])
    replay.step([{"id": "c", "tokens": [1], "want": []}], ["c"])
    assert model.log == [("cache", 2, 50), ("run", [(0, [1, 2]), (1, [3])]), ("run", [(1, [4]), (0, [5])]), ("release", 0),
                         ("run", [(1, [6])]), ("release", 1), ("run", [(0, [1])]), ("release", 0)]


# ---- the plain statement itself ---------------------------------------------------------------------------------
def test_statement_is_causal_and_sees_far_tokens():
    c = H.CASES["mixed"]
    w = H.make_weights(c, 5)
    ids = H.tokens(c, 40)
    base = O.forward(c, w, ids)
    changed = ids.copy()
    changed[30] = (changed[30] + 1) % c["vocab"]
    other = O.forward(c, w, changed)
    assert np.array_equal(base[:30], other[:30]) and np.abs(base[30:] - other[30:]).max() > 1e-2
    first = ids.copy()
    first[0] = (first[0] + 1) % c["vocab"]
    assert np.abs(base[39] - O.forward(c, w, first)[39]).max() > 1e-4


def test_statement_recurrence_matches_its_closed_form():
    """One head, one group: y_t = sum_s prod(decay) dt_s (C_t . B_s) x_s + D x_t."""
    rng = np.random.default_rng(0)
    T, P, N = 9, 3, 4
    x, Bm, Cm, dt = rng.normal(size=(T, 1, P)), rng.normal(size=(T, 1, N)), rng.normal(size=(T, 1, N)), rng.uniform(0.1, 1, (T, 1))
    a_log, d = np.array([0.3]), np.array([0.7])
    y = O.ssm_recurrence(x, Bm, Cm, dt, a_log, d)
    logs = np.cumsum(-np.exp(a_log) * dt[:, 0])
    for t in range(T):
        want = d * x[t, 0] + sum(np.exp(logs[t] - logs[s]) * dt[s, 0] * (Cm[t, 0] @ Bm[s, 0]) * x[s, 0] for s in range(t + 1))
        assert np.allclose(y[t, 0], want)


def test_statement_loop_order():
    c = H.CASES["mixed"]
    assert O.run_order(c) == [(0, None, False), (1, 0, True), (2, 0, False), (1, 1, True), (2, 1, False), (3, None, False)]
