"""Configuration, registry, weight files and argument checks of the parallel decoder: everything that needs no GPU, and the plain
statement's own checks."""
import json

import numpy as np
import pytest

import ctorch_b200 as B
import parallel_cases as P
import parallel_oracle as O


def host_model(c, dtype="bf16", weights=None):
    return B.LanguageModel(c, weights, dtype=dtype, device=None)


@pytest.mark.parametrize("name", P.CASES)
def test_parameters_follow_the_configuration(name):
    c = P.CASES[name]
    assert {n: t.shape for n, t in host_model(c).module.state().items()} == {n: tuple(s) for n, s in P.weight_shapes(c).items()}


def broken(change):
    c = json.loads(json.dumps(P.CASES["mixed"]))
    change(c)
    return c


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][1].update(type="rnn"), "unknown layer type 'rnn'"),
    (lambda c: c["layers"][1]["mixer"].pop("vdim"), r"layers\[1\]\.mixer\.vdim' is missing"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "at most dim"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "must be even"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "must be a positive integer"),
    (lambda c: c["layers"][1]["mlp"].update(kind="routed"), "unknown feed-forward kind 'routed'"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "exceeds the number of experts"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(experts=5000), "more than 1024 experts"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), r"mlp\.expert' is missing"),
    (lambda c: c["loop"].update(stop=5), "range of layers"),
    (lambda c: c["norm"].pop("eps"), "eps' is missing"),
    (lambda c: c.update(architecture="Ripitar", embedding={"scale": 1.0}, logit_scale=1.0), "unknown layer type 'attention'"),
])
def test_configuration_errors_name_the_key(change, message):
    with pytest.raises(B.B200Error, match=message):
        host_model(broken(change))


def test_weight_folder_round_trip(tmp_path):
    c = P.CASES["mixed"]
    w = P.make_weights(c, 3)
    P.write_folder(tmp_path, c, w)
    for name, tensor in B.LanguageModel.load(str(tmp_path), dtype="f32", device=None).module.state().items():
        assert np.array_equal(tensor.numpy(), w[name]), name
    del w["l1.mlp.e5.down"]
    P.write_folder(tmp_path, c, w)
    with pytest.raises(B.B200Error, match="l1.mlp.e5.down"):
        B.LanguageModel.load(str(tmp_path), device=None)


def test_no_cpu_compute_path():
    with pytest.raises(B.B200Error, match="no CPU compute path"):
        host_model(P.CASES["ones"]).new_cache(1, 8)


# ---- the statement itself ---------------------------------------------------------------------------------------
def test_chunks_are_counted_from_the_start():
    seen = [[j for j in range(12) if O.chunk_visible(i, j, 5)] for i in range(12)]
    assert seen[4] == [0, 1, 2, 3, 4] and seen[5] == [5] and seen[9] == [5, 6, 7, 8, 9] and seen[11] == [10, 11]
    assert all(O.chunk_visible(i, j, None) == (j <= i) for i in range(6) for j in range(6))


def test_statement_distinguishes_the_mechanisms():
    """Every mechanism matters to the logits of the test weights: the mistake is planted in the statement's configuration or weights."""
    c, w = P.CASES["mixed"], P.make_weights(P.CASES["mixed"])
    ids = P.tokens(c, 40)
    want = O.forward(c, w, ids)

    def differs(config, weights):
        return np.abs(O.forward(config, weights, ids) - want).max() / np.abs(want).max()

    for layer, key, value in ((0, ("mask", "size"), 17), (1, ("mask", "size"), 8), (0, ("rot", "dims"), 16), (1, ("rot", "base"), 700.0), (2, ("scale",), 0.25)):
        d = json.loads(json.dumps(c))
        at = d["layers"][layer]["mixer"]
        for k in key[:-1]:
            at = at[k]
        at[key[-1]] = value
        assert differs(d, w) > 1e-2, (layer, key)
    for d in (dict(c, loop={"start": 1, "stop": 2, "times": 2}), dict(c, loop={"start": 1, "stop": 3, "times": 3}), dict(c, norm={"eps": 0.3})):
        assert differs(d, w) > 1e-2
    one = json.loads(json.dumps(c))
    one["layers"][1]["mlp"]["router"]["top"] = 1
    assert differs(one, w) > 1e-2
    for name in ("l0.mix.q.norm", "l2.mix.k.norm", "l1.norm1", "final.norm"):
        assert differs(c, {**w, name: np.ones_like(w[name])}) > 1e-2, name
    for name in ("l0.mix.g", "l1.mlp.router", "l1.mlp.shared.up"):
        assert differs(c, {**w, name: np.zeros_like(w[name])}) > 1e-2, name


def test_the_weight_multiplies_the_experts_input():
    w = {"e0.up": np.array([[2.0]]), "e0.down": np.array([[1.0]]), "router": np.array([[0.0]])}
    h = np.array([[3.0]])
    got = O.mixture(h, w, "", {"router": {"top": 1}})
    assert np.allclose(got, O.gelu_exact(np.array(3.0))) and not np.allclose(got, 0.5 * O.gelu_exact(np.array(6.0)))
