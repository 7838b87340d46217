"""Configuration, registry, weight files and argument checks of the sandwich decoder: everything that needs no GPU, and the plain
statement's own checks."""
import json

import numpy as np
import pytest

import ctorch_b200 as B
import sandwich_cases as S
import sandwich_oracle as O


def host_model(c, dtype="bf16", weights=None):
    return B.LanguageModel(c, weights, dtype=dtype, device=None)


def changed(change, name="mixed"):
    c = json.loads(json.dumps(S.CASES[name]))
    change(c)
    return c


@pytest.mark.parametrize("name", S.CASES)
def test_parameters_follow_the_configuration(name):
    c = S.CASES[name]
    assert {n: t.shape for n, t in host_model(c).module.state().items()} == {n: tuple(s) for n, s in S.weight_shapes(c).items()}


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][1].update(type="attention_3"), "unknown layer type 'attention_3'"),
    (lambda c: c["layers"][0].update(type="mamba2"), "unknown layer type 'mamba2'"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_heads"), r"layers\[0\]\.mixer\.kv_heads' is missing"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(vdim=8), "values that are the keys"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "at most dim"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7), "must be even"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=0), "'softcap' must be positive"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "'kv_from' must name an earlier attention layer"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=0), "'kv_from' must name an earlier attention layer"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=-1), "number of a layer"),
    (lambda c: c["layers"][2]["mixer"]["right"]["decay"].pop(), "one number per head"),
    (lambda c: c["layers"][2]["mixer"].pop("left_scale"), "left_scale' is missing"),
    (lambda c: c["layers"][2]["mixer"]["right"].update(dim=600), "exceeds 512"),
    (lambda c: c["layers"][1]["mlp"].pop("limit"), r"mlp\.limit' is missing"),
    (lambda c: c["layers"][1]["mlp"].update(limit=-1.0), "'limit' must be positive"),
    (lambda c: c["layers"][0]["mlp"].update(kind="routed"), "unknown feed-forward kind 'routed'"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "exceeds the number of experts"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(identity=-1), "negative number of identity experts"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(experts=1000, identity=25), "more than 1024 experts"),
    (lambda c: c["layers"][0]["mlp"].update(shared={"ff": 8}), "shared expert"),
    (lambda c: c["embedding"].pop("bigram"), r"embedding\.bigram' is missing"),
    (lambda c: c["embedding"]["bigram"].update(buckets=0), "must be a positive integer"),
    (lambda c: c.update(logit_softcap=-3.0), "'logit_softcap' must be positive"),
    (lambda c: c.update(loop={"start": 0, "stop": 1, "times": 2}), "looped layers"),
    (lambda c: c["norm"].pop("eps"), "eps' is missing"),
])
def test_configuration_errors_name_the_key(change, message):
    with pytest.raises(B.B200Error, match=message):
        host_model(changed(change))


def test_layers_without_optional_parts():
    """No rotation, no cap, no identity experts, no feed-forward: the configuration may leave them out."""
    def drop(c):
        c["layers"][1]["mixer"].pop("softcap")
        c["layers"][1]["mixer"].pop("rot")
        c["layers"][0]["mlp"]["router"].pop("identity")
        c["layers"][2].pop("mlp")
        c["layers"][1]["mixer"]["kv_from"] = None
    state = host_model(changed(drop)).module.state()
    assert state["l0.mlp.router"].shape == (6, 64) and "l2.norm2" not in state and "l1.mix.k" in state


def test_weight_folder_round_trip(tmp_path):
    c = S.CASES["mixed"]
    w = S.make_weights(c, 3)
    S.write_folder(tmp_path, c, w)
    for name, tensor in B.LanguageModel.load(str(tmp_path), dtype="f32", device=None).module.state().items():
        assert np.array_equal(tensor.numpy(), w[name]), name
    del w["l2.mix.left.sink"]
    S.write_folder(tmp_path, c, w)
    with pytest.raises(B.B200Error, match="l2.mix.left.sink"):
        B.LanguageModel.load(str(tmp_path), device=None)


def test_no_cpu_compute_path():
    with pytest.raises(B.B200Error, match="no CPU compute path"):
        host_model(S.CASES["ones"]).new_cache(1, 8)


# ---- the statement itself ---------------------------------------------------------------------------------------
def test_statement_distinguishes_the_mechanisms():
    """Every mechanism matters to the logits of the test weights: the mistake is planted in the statement's configuration or weights."""
    c, w = S.CASES["mixed"], S.make_weights(S.CASES["mixed"])
    ids = S.tokens(c, 40)
    want = O.forward(c, w, ids)

    def differs(config, weights):
        return np.abs(O.forward(config, weights, ids) - want).max() / np.abs(want).max()

    for layer, path, value in ((0, ("mixer", "rot", "dims"), 16), (1, ("mixer", "rot", "base"), 700.0), (0, ("mixer", "scale"), 0.2), (1, ("mixer", "softcap"), 2.0), (3, ("mixer", "softcap"), None),
                               (2, ("mixer", "left_scale"), 0.5), (2, ("mixer", "right_scale"), 1.2), (2, ("mixer", "right", "decay"), [0.5, 0.9, 0.95]), (1, ("mlp", "limit"), 1.4),
                               (0, ("mlp", "router", "top"), 1), (4, ("mlp", "limit"), 0.8)):
        def plant(d):
            at = d["layers"][layer]
            for k in path[:-1]:
                at = at[k]
            at[path[-1]] = value
        assert differs(changed(plant), w) > 3e-3, (layer, path)
    for key, value in (("norm", {"eps": 0.3}), ("logit_softcap", 3.2), ("embedding", {"bigram": {"buckets": 61, "mul_prev": 7, "mul_cur": 31}})):
        assert differs(dict(c, **{key: value}), w) > 1e-2, key
    zeroed = ("l0.norm1", "l0.norm1b", "l1.norm2", "l1.norm2b", "final.norm", "l0.mix.q.b", "l0.mix.k.b", "l0.mix.g", "l1.mix.sink", "l2.mix.left.sink", "l2.mix.left.g", "l2.mix.right.g",
              "l0.mlp.correction", "l0.mlp.router", "bigram", "l3.mix.sink")
    for name in zeroed:
        assert differs(c, {**w, name: np.zeros_like(w[name])}) > 1e-2, name
    for name in ("l2.mix.left.q.norm", "l2.mix.left.k.norm", "l2.mix.right.norm"):
        assert differs(c, {**w, name: np.ones_like(w[name])}) > 3e-3, name
    first = w["bigram"].copy()
    first[-1] = 0
    assert differs(c, {**w, "bigram": first}) > 1e-2


def test_sinks_take_their_share():
    assert np.allclose(O.sink_softmax(np.zeros((1, 3)), 0.0), 0.25)          # one added to the denominator
    assert np.allclose(O.sink_softmax(np.array([[0.0, -np.inf]]), np.log(3.0)), [[0.25, 0.0]])
    assert np.allclose(O.sink_softmax(np.array([[1e4, 0.0]]), 0.0), [[1.0, 0.0]])


def test_pair_rows():
    spec = {"buckets": 10, "mul_prev": 7, "mul_cur": 3}
    assert O.pair_row(None, 4, spec) == 10 and O.pair_row(2, 4, spec) == 6 and O.pair_row(4, 2, spec) == 4


def test_choice_is_corrected_and_weights_are_not():
    logits = np.log(np.array([[0.5, 0.3, 0.2]]))
    chosen, score = O.route(logits, np.array([0.0, 0.0, 0.4]), 2)
    assert chosen.tolist() == [[2, 0]] and np.allclose(score, [[0.2, 0.5]])
    w = {"router": logits.T, "correction": np.array([0.0, 0.0, 0.4]), "e0.gate": np.array([[1.0]]), "e0.up": np.array([[2.0]]), "e0.down": np.array([[1.0]])}
    got = O.mixture(np.array([[1.0]]), w, "", {"router": {"experts": 1, "identity": 2, "top": 2}})
    assert np.allclose(got, 0.2 + 0.5 * 2.0 * O.silu(1.0))


def test_unrotated_keys_serve_as_values():
    h = np.eye(2)
    w = {"q": np.zeros((2, 2)), "q.b": np.zeros(2), "k": 5.0 * np.eye(2), "k.b": np.array([1.0, 2.0]), "g": np.zeros((1, 2)), "o": np.eye(2)}
    m = {"heads": 1, "kv_heads": 1, "rot": {"dims": 2, "base": 10.0}, "scale": 1.0}
    got = O.attention_keys_as_values(h, w, "", m)
    assert np.allclose(got[0], 0.5 * np.array([6.0, 2.0]) / 2) and np.allclose(got[1], 0.5 * np.array([7.0, 9.0]) / 3)


def test_clamped_units_by_hand():
    got = O.clamped_units(np.array([5.0, -5.0, 0.5]), np.array([9.0, -9.0, 0.25]), 2.0)
    want = [2.0 * 3.0 / (1 + np.exp(-3.404)), -5.0 * -1.0 / (1 + np.exp(8.51)), 0.5 * 1.25 / (1 + np.exp(-0.851))]
    assert np.allclose(got, want)
