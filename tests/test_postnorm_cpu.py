"""Configuration, registry, weight files and argument checks of the post-norm decoder: everything that needs no GPU, and the plain
statement's own checks."""
import json

import numpy as np
import pytest

import ctorch_b200 as B
import postnorm_cases as S
import postnorm_oracle as O


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
    (lambda c: c["layers"][1]["mixer"].pop("kv_heads"), r"layers\[1\]\.mixer\.kv_heads' is missing"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), r"mixer\.conv' is missing"),
    (lambda c: c["layers"][0]["mixer"].update(dim=600), "'dim' exceeds 512"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "must be a positive integer"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(pool=0), "must be a positive integer"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=2), "not combined with pooled blocks"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(keep_first=-1), "must not be negative"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=26), "at most dim"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7), "must be even"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("factor"), r"scaling\.factor' is missing"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].update(factor=0.0), "'factor' must be positive"),
    (lambda c: c["layers"][3].update(weights_of=7), "'weights_of' must name a layer with weights"),
    (lambda c: c["layers"][3].update(weights_of=3), "'weights_of' must name a layer with weights"),
    (lambda c: c["layers"][3].update(weights_of=1), "'weights_of' must name a layer of the same type"),
    (lambda c: c["layers"][0]["mlp"].update(kind="routed"), "unknown feed-forward kind 'routed'"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "exceeds the number of experts"),
    (lambda c: c.pop("residual_mult"), "residual_mult' is missing"),
    (lambda c: c.update(loop={"start": 0, "stop": 1, "times": 2}), "looped layers"),
    (lambda c: c["norm"].pop("eps"), "eps' is missing"),
])
def test_configuration_errors_name_the_key(change, message):
    with pytest.raises(B.B200Error, match=message):
        host_model(changed(change))


def test_layers_without_optional_parts():
    """No feed-forward, no stretched positions, a window alone."""
    def drop(c):
        c["layers"][1].pop("mlp")
        c["layers"][1]["mixer"]["mask"].pop("pool")
        c["layers"][2]["mixer"]["rot"].pop("scaling")
        c["layers"][2]["mixer"]["mask"].pop("keep_first")
    state = host_model(changed(drop)).module.state()
    assert "l1.norm2" not in state and "l1.mlp.router" not in state and "l2.mix.talk" in state and "l3.norm1" not in state and "head" not in state


def test_weight_folder_round_trip(tmp_path):
    c = S.CASES["mixed"]
    w = S.make_weights(c, 3)
    S.write_folder(tmp_path, c, w)
    for name, tensor in B.LanguageModel.load(str(tmp_path), dtype="f32", device=None).module.state().items():
        assert np.array_equal(tensor.numpy(), w[name]), name
    del w["l2.mix.talk"]
    S.write_folder(tmp_path, c, w)
    with pytest.raises(B.B200Error, match="l2.mix.talk"):
        B.LanguageModel.load(str(tmp_path), device=None)


def test_no_cpu_compute_path():
    with pytest.raises(B.B200Error, match="no CPU compute path"):
        host_model(S.CASES["ones"]).new_cache(1, 8)


# ---- the statement itself ---------------------------------------------------------------------------------------
def test_statement_distinguishes_the_mechanisms():
    """Every mechanism matters to the logits of the test weights: the mistake is planted in the statement's configuration or weights."""
    c, w = S.CASES["mixed"], S.make_weights(S.CASES["mixed"])
    ids = S.tokens(c, 60)
    want = O.forward(c, w, ids)

    def differs(config, weights):
        return np.abs(O.forward(config, weights, ids) - want).max() / np.abs(want).max()

    for layer, path, value in ((1, ("mixer", "rot", "dims"), 16), (1, ("mixer", "rot", "base"), 700.0), (1, ("mixer", "scale"), 0.2), (1, ("mixer", "mask", "size"), 21),
                               (1, ("mixer", "mask", "pool"), 5), (1, ("mixer", "mask", "pool"), 64), (2, ("mixer", "mask", "size"), 17), (2, ("mixer", "mask", "keep_first"), 2),
                               (2, ("mixer", "mask", "keep_first"), 0), (2, ("mixer", "rot", "scaling", "factor"), 2.0), (0, ("mlp", "router", "top"), 1)):
        def plant(d):
            at = d["layers"][layer]
            for k in path[:-1]:
                at = at[k]
            at[path[-1]] = value
        assert differs(changed(plant), w) > 3e-3, (layer, path)
    for key, value in (("norm", {"eps": 0.3}), ("residual_mult", 0.78)):
        assert differs(dict(c, **{key: value}), w) > 1e-2, key
    assert differs(changed(lambda d: d["layers"].pop()), w) > 1e-2
    for name in ("l0.norm1", "l1.norm2", "final.norm", "l0.mix.b", "l0.mix.a", "l0.mix.dt_bias", "l0.mix.A_log", "l0.mix.g", "l1.mix.g", "l0.mlp.router", "l0.mlp.router.b"):
        assert differs(c, {**w, name: np.zeros_like(w[name])}) > 1e-2, name
    for name in ("l1.mix.q.norm", "l1.mix.k.norm", "l2.mix.q.norm", "l2.mix.k.norm", "l0.mix.norm"):
        assert differs(c, {**w, name: np.ones_like(w[name])}) > 3e-3, name
    assert differs(c, {**w, "l2.mix.talk": np.eye(6)}) > 1e-2 and differs(c, {**w, "l2.mix.talk": w["l2.mix.talk"].T}) > 1e-2
    for name in ("q", "k", "v"):
        assert differs(c, {**w, f"l0.mix.{name}.conv": w[f"l0.mix.{name}.conv"][:, ::-1]}) > 1e-2, name


def test_window_edges_by_hand():
    seen = O.seen_tokens(8, 3, 2)
    assert np.flatnonzero(seen[7]).tolist() == [0, 1, 5, 6, 7] and np.flatnonzero(seen[3]).tolist() == [0, 1, 2, 3] and np.flatnonzero(seen[0]).tolist() == [0]
    blocks = O.seen_blocks(12, 4, 3)      # block 0 holds 0 .. 2: seen once 2 <= i - 4; block 1 holds 3 .. 5
    assert [np.flatnonzero(row).tolist() for row in blocks[[5, 6, 8, 9]]] == [[], [0], [0], [0, 1]]
    assert np.allclose(O.block_means(np.arange(14.0).reshape(7, 2), 3), [[2, 3], [8, 9]])


def test_tokens_and_blocks_share_one_softmax():
    """Three keys of one score each: the window's two tokens and the block of the two before them."""
    k = np.array([[[1.0, 0], [0, 1.0], [1.0, 0], [0, 1.0]]])
    weights = O.pooled_window_weights(np.zeros((1, 4, 2)), k, 1.0, 2, 2)
    assert np.allclose(weights[0, 3], [0, 0, 1 / 3, 1 / 3, 1 / 3, 0]) and np.allclose(weights[0, 2], [0, 0.5, 0.5, 0, 0, 0])


def test_halves_turn_together():
    x = np.array([[1.0, 2.0, 3.0, 4.0, 5.0]])
    got = O.rotate_halves(x, np.array([3]), 4, 100.0, 2.0)
    for i, angle in ((0, 1.5), (1, 0.15)):
        c, s = np.cos(angle), np.sin(angle)
        assert np.allclose(got[0, [i, i + 2]], [x[0, i] * c - x[0, i + 2] * s, x[0, i + 2] * c + x[0, i] * s])
    assert got[0, 4] == 5.0


def test_mixed_weights_meet_their_own_values():
    """Head h takes the other heads' weights to the values of its own kv head."""
    weights = np.array([[[1.0, 0.0]], [[0.0, 1.0]]])
    mixed = O.mixed_heads(weights, np.array([[0.5, 2.0], [0.0, -1.0]]))
    assert np.allclose(mixed, [[[0.5, 2.0]], [[0.0, -1.0]]])


def test_delta_rule_replaces_what_a_key_holds():
    """With beta 1 and decay 1 the state answers a unit key with the last value written under it, and keeps what orthogonal keys hold."""
    k = np.array([[1.0, 0], [0, 1.0], [1.0, 0], [0, 1.0]])[:, None]
    v = np.array([[1.0, 2, 3], [4, 5, 6], [7, 8, 9], [0, 0, 0]])[:, None]
    q = np.array([[1.0, 0], [1.0, 0], [1.0, 0], [1.0, 0]])[:, None]
    beta, g = np.array([1.0, 1, 1, 0])[:, None], np.array([1.0, 1, 1, 0.5])[:, None]
    out, S_ = O.delta_rule(q, k, v, beta, g)
    assert np.allclose(out[:, 0], [[1, 2, 3], [1, 2, 3], [7, 8, 9], [3.5, 4, 4.5]]) and np.allclose(S_[0, 1], [2, 2.5, 3])


def test_choice_and_weights_take_the_bias():
    z = np.array([[0.0, 1.0, 2.0]])
    chosen, score = O.route(z + np.array([3.0, 0.0, 0.0]), 2)
    assert chosen.tolist() == [[0, 2]] and np.allclose(score, [[np.e / (1 + np.e), 1 / (1 + np.e)]])
