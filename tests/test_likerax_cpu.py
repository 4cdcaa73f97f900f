"""CPU: the Likerax oracle's mechanisms, the configuration reader, the registry and the command line."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import likerax_models as M
from oracle import likerax_np as L

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def small(**kw):
    return M.make(M.config([M.layer(chunk=7), M.layer(heads=3, kv_heads=1, dim=20, vdim=12, chunk=5, ff=None)],
                           vocab=41, width=36, streams=2, **kw), seed=3)


def test_one_stream_with_unit_connections_is_the_ordinary_residual():
    x, y = np.random.default_rng(0).standard_normal((2, 5, 8))
    one = np.ones(1)
    got = L.hyper_connection([x], one, np.ones((1, 1)), one, lambda u: y * u)
    assert np.allclose(got[0], x + y * x)


def test_mix_is_indexed_from_to():
    a, b = np.ones((1, 4)), 10 * np.ones((1, 4))
    new = L.hyper_connection([a, b], [1, 0], [[1, 2], [3, 4]], [0, 0], lambda u: u)
    assert new[0][0, 0] == 1 * 1 + 3 * 10 and new[1][0, 0] == 2 * 1 + 4 * 10


def test_positions_see_their_own_chunk_only():
    seen = [[j for j in range(12) if L.visible(i, j, 5)] for i in range(12)]
    assert seen[4] == [0, 1, 2, 3, 4] and seen[5] == [5] and seen[11] == [10, 11]
    assert [j for j in range(12) if L.visible(6, j, None)] == list(range(7))


def test_distance_bias_favours_near_keys():
    g = np.random.default_rng(1)
    q = np.zeros((6, 4))
    v = np.eye(6)
    out = L.attention_head(q, g.standard_normal((6, 4)), v, 1.0, 0.5, None)
    assert np.allclose(out[5], np.exp(-0.5 * (5 - np.arange(6))) / np.exp(-0.5 * np.arange(6)).sum())


def test_a_prompt_is_causal_and_a_chunk_forgets_the_one_before():
    m = small()
    a = np.arange(14) % 41
    la = L.forward(m, a)
    b = a.copy()
    b[9] = 40
    lb = L.forward(m, b)
    assert np.array_equal(la[:9], lb[:9]) and not np.allclose(la[9:], lb[9:])
    # one layer with chunks of 7: what lies before position 7 does not reach it
    one = M.make(M.config([M.layer(chunk=7)], vocab=41, width=36, streams=2), seed=5)
    c = a.copy()
    c[6] = 40
    assert np.allclose(L.forward(one, a)[7:], L.forward(one, c)[7:])
    assert not np.allclose(L.forward(one, a)[6], L.forward(one, c)[6])


def test_a_loop_equals_the_layers_written_out():
    looped = small(loop=(0, 1, 3))
    flat = {"cfg": dict(looped["cfg"]), "w": {}}
    flat["cfg"].pop("loop")
    order = L.layer_order(looped["cfg"])
    assert order == [0, 0, 0, 1]
    flat["cfg"]["layers"] = [looped["cfg"]["layers"][i] for i in order]
    for n, a in looped["w"].items():
        if not n.startswith("l"):
            flat["w"][n] = a
    for k, i in enumerate(order):
        for n, a in looped["w"].items():
            if n.startswith(f"l{i}."):
                flat["w"][f"l{k}." + n.split(".", 1)[1]] = a
    t = np.arange(11)
    assert np.allclose(L.forward(looped, t), L.forward(flat, t))


def test_run_order_and_slopes_of_the_reader():
    from rotor_b200.likerax import distance_slopes, run_order
    assert run_order(4) == [0, 1, 2, 3]
    assert run_order(4, {"start": 1, "stop": 3, "times": 2}) == [0, 1, 2, 1, 2, 3]
    assert run_order(3, {"start": 0, "stop": 3, "times": 1}) == [0, 1, 2]
    with pytest.raises(ValueError):
        run_order(2, {"start": 1, "stop": 3, "times": 2})
    assert distance_slopes(8)[0] == 0.5 and np.isclose(distance_slopes(6)[5], 2.0 ** -8)


def test_config_reader_takes_every_branch_and_rejects_others():
    from rotor_b200.likerax import LikeraxConfig
    c = LikeraxConfig.from_dict(small(loop=(0, 2, 2))["cfg"])
    assert (c.vocab, c.width, c.streams, c.order) == (41, 36, 2, [0, 1, 0, 1])
    assert c.layers[1].ff is None and c.layers[0].chunk == 7 and c.layers[1].vdim == 12
    bad = small()["cfg"]
    bad["layers"][0]["type"] = "convolution"
    with pytest.raises(ValueError):
        LikeraxConfig.from_dict(bad)
    bad = small()["cfg"]
    bad["layers"][0]["mlp"]["kind"] = "experts"
    with pytest.raises(ValueError):
        LikeraxConfig.from_dict(bad)


def test_registry_knows_both_families_and_refuses_others(tmp_path):
    from rotor_b200 import registry
    assert {"BitNet", "Likerax"} <= set(registry.architectures())
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unheard"}))
    with pytest.raises(ValueError, match="Unheard"):
        registry.load_model(tmp_path)
    (tmp_path / "config.json").write_text(json.dumps({"vocab_size": 8, "hidden_size": 8}))
    with pytest.raises(registry.UnsupportedDtype):
        registry.load_model(tmp_path, dtype="float32")


def test_trace_of_a_design_without_float32_exits_with_3(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"vocab_size": 8, "hidden_size": 8}))
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32",
                        "--out", str(tmp_path), "--max-tokens", "16"], input="", capture_output=True, text=True)
    assert r.returncode == 3, r.stderr


def test_command_line_info(tmp_path, capsys):
    from rotor_b200.__main__ import main
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Likerax"}))
    assert main(["info", "--model", str(tmp_path)]) == 0
    out = capsys.readouterr().out
    assert "BitNet" in out and out.strip().endswith("Likerax")


def test_trace_session_keeps_one_request_and_its_length():
    from rotor_b200.trace import TraceSession

    class Recorder:
        vocab_size = 3

        def __init__(self):
            self.calls = []

        def forward_rows_device(self, tokens, past, rows):
            import torch
            self.calls.append((list(tokens), past, list(rows)))
            return torch.zeros((len(rows), 3))

    m = Recorder()
    s = TraceSession(m)
    assert s.step([{"id": "a", "tokens": [1, 2, 3], "want": [2]}]).shape == (1, 3)
    assert s.step([{"id": "a", "tokens": [4], "want": []}], ["a"]).shape == (0, 3)
    s.step([{"id": "b", "tokens": [5, 6], "want": [0, 1]}])
    with pytest.raises(ValueError):
        s.step([{"id": "c", "tokens": [7], "want": []}])
    assert m.calls == [([1, 2, 3], 0, [2]), ([4], 3, []), ([5, 6], 0, [0, 1])]
