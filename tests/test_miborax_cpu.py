"""CPU: the Miborax oracle's mechanisms, the configuration reader, the registry and the planning of shared caches."""
import copy
import json

import numpy as np
import pytest

import miborax_models as M
from oracle import miborax_np as O


def small():
    return M.make(M.config([M.window(6), M.window(9, kv_from=0, heads=2, vdim=8), M.full(), M.window(4, kv_from=0, mlp=None)],
                           vocab=37, width=44), seed=2)


def test_layer_norm_centres_and_adds_its_bias():
    x = np.random.default_rng(0).standard_normal((3, 10)) + 5
    y = O.layer_norm(x, np.ones(10), np.zeros(10), 0.0)
    assert np.allclose(y.mean(-1), 0) and np.allclose((y * y).mean(-1), 1)
    assert np.allclose(O.layer_norm(x, 2 * np.ones(10), 3 * np.ones(10), 0.0), 2 * y + 3)


def test_rotation_turns_neighbouring_pairs_and_keeps_relative_scores():
    g = np.random.default_rng(1)
    q, k = g.standard_normal((2, 1, 8))
    one = O.rotate(np.array([[1.0, 0, 0, 0]]), [3], 100.0, 4)[0]
    assert np.allclose(one, [np.cos(3), np.sin(3), 0, 0])
    assert np.allclose(O.rotate(np.array([[0, 0, 1.0, 0]]), [3], 100.0, 4)[0], [0, 0, np.cos(0.3), np.sin(0.3)])
    a = (O.rotate(q, [9], 50.0, 8) * O.rotate(k, [4], 50.0, 8)).sum()
    b = (O.rotate(q, [25], 50.0, 8) * O.rotate(k, [20], 50.0, 8)).sum()
    assert np.isclose(a, b) and np.array_equal(O.rotate(q, [9], 50.0, 4)[..., 4:], q[..., 4:])


def test_a_sink_takes_weight_and_has_no_value():
    s = np.array([1.0, 2.0, 0.5])
    p = O.sink_softmax(s, 2.0)
    assert np.allclose(p, np.exp(s) / (np.exp(s).sum() + np.exp(2.0)))
    assert np.allclose(O.sink_softmax(s, None).sum(), 1) and O.sink_softmax(s, 80.0).sum() < 1e-30


def test_a_window_holds_its_own_position_and_those_before():
    assert [j for j in range(12) if O.visible(7, j, 3)] == [5, 6, 7]
    assert [j for j in range(12) if O.visible(7, j, None)] == list(range(8))
    v = np.eye(9)
    out = O.attention_head(np.zeros((9, 2)), np.zeros((9, 2)), v, 1.0, None, 4)
    assert np.array_equal(np.flatnonzero(out[8]), [5, 6, 7, 8]) and np.array_equal(np.flatnonzero(out[1]), [0, 1])


def test_routing_takes_the_largest_and_weighs_those_alone():
    r = dict(O.routes(np.array([0.0, 3.0, 1.0, 2.0]), 2))
    assert set(r) == {1, 3} and np.isclose(r[1], 1 / (1 + np.exp(-1.0)))
    assert [e for e, _ in O.routes(np.array([1.0, 1.0, 1.0]), 2)] == [0, 1]


def test_a_prompt_is_causal_and_windows_forget():
    m = small()
    a = np.arange(20) % 37
    b = a.copy()
    b[11] = 36
    la, lb = O.forward(m, a), O.forward(m, b)
    assert np.array_equal(la[:11], lb[:11]) and not np.allclose(la[11:], lb[11:])
    one = M.make(M.config([M.window(5)], vocab=37, width=44), seed=5)
    la, lb = O.forward(one, a), O.forward(one, b)
    assert np.allclose(la[16:], lb[16:]) and all(not np.allclose(la[i], lb[i]) for i in range(11, 16))


def test_config_reader_takes_every_branch_and_rejects_others():
    from rotor_b200.miborax import MiboraxConfig
    cfg = small()["cfg"]
    c = MiboraxConfig.from_dict(cfg)
    assert (c.vocab, c.width, c.embed_scale) == (37, 44, 3.0)
    assert [l.window for l in c.layers] == [6, 9, 0, 4] and [l.kv_from for l in c.layers] == [None, 0, None, 0]
    assert [l.q_rank for l in c.layers] == [None, None, 36, None] and [l.gated for l in c.layers] == [False, False, True, False]
    assert c.layers[3].mlp is None and (c.layers[2].mlp.experts, c.layers[2].mlp.top) == (5, 2)
    for change in (lambda e: e.update(type="attention"), lambda e: e["mlp"].update(kind="dense"), lambda e: e["mixer"]["rot"].update(dims=4)):
        bad = copy.deepcopy(cfg)
        change(bad["layers"][0])
        with pytest.raises(ValueError):
            MiboraxConfig.from_dict(bad)


def test_runs_that_share_a_cache_are_tied_to_its_owner():
    from rotor_b200.decoder_model import Latent, LayerSpec, plan_runs

    def spec(kv_from=None, rank=8, base=10.0):
        a = Latent(rank, 4, base, None, None, dkv=object() if kv_from is None else None, kv_from=kv_from)
        return LayerSpec(1, 1, 8, 8, 1.0, None, None, None, None, None, latent=a)

    runs = plan_runs([spec(), spec(0), spec(), spec(2), spec(0)], range(5))
    assert [None if r.source is None else runs.index(r.source) for r in runs] == [None, 0, None, 2, 0]
    for bad in ([spec(1), spec()], [spec(), spec(0, rank=16)], [spec(), spec(0, base=11.0)], [spec(), spec(0), spec(1)]):
        with pytest.raises(ValueError):
            plan_runs(bad, range(len(bad)))


def test_registry_and_command_line_know_the_design(tmp_path, capsys):
    from rotor_b200 import registry
    from rotor_b200.__main__ import main
    assert "Miborax" in registry.architectures()
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Miborax"}))
    assert main(["info", "--model", str(tmp_path)]) == 0
    assert capsys.readouterr().out.strip().endswith("Miborax")


def test_the_seeded_models_route_without_close_calls():
    m = small()
    w = {n: np.asarray(a, dtype=np.float64) for n, a in m["w"].items()}
    x = w["embed"] * m["cfg"]["embedding"]["scale"]
    z = np.sort(O.linear(w["l0.mlp.router"], O.layer_norm(x, w["l0.norm2"], w["l0.norm2.b"], 1e-4)) + w["l0.mlp.router.b"], axis=-1)
    assert np.diff(z, axis=-1).min() > 0.15
