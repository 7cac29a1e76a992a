"""Degedra on the CPU: configuration, registry, checkpoint reader and writer, slots, the oracle's own
consistency, and the host-side packing."""
import json

import pytest
import torch

from degedra_cases import A, CONFIGS, ids, layer, mixed_config, model, oracle
import degedra_oracle as O


def test_config_round_trip():
    from mi50grad_b200.config import degedra_config_from_dict, degedra_config_to_dict
    for make in CONFIGS.values():
        cfg = make()
        assert degedra_config_from_dict(json.loads(json.dumps(degedra_config_to_dict(cfg)))) == cfg
    assert [mixed_config().weight_layer(i) for i in range(6)] == [0, 1, 0, 3, 1, 3]


def test_config_rejects_what_it_cannot_run():
    from mi50grad_b200.config import DegedraConfig, degedra_config_from_dict, degedra_config_to_dict
    c = degedra_config_to_dict(mixed_config())
    for path, val in ((("type",), "other"), (("mixer", "left", "vdim"), 7), (("mlp", "kind"), "other"),
                      (("mixer", "left", "kv_heads"), 5), (("mixer", "right", "norm_groups"), 7)):
        bad = json.loads(json.dumps(c))
        d = bad["layers"][0]
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = val
        with pytest.raises(ValueError):
            degedra_config_from_dict(bad)
    a, s = A(2, 1, 16, 16, 4), (2, 8, 8, 1, 2, 1)
    with pytest.raises(ValueError):
        DegedraConfig(32, 10, 1e-5, [layer(a, s, of=1), layer(a, s, of=0)])


def test_registry_and_loader(tmp_path):
    from mi50grad_b200.loaders import load_any
    from mi50grad_b200.models.mixer_weights import named_tensors, write_mixer_checkpoint
    from mi50grad_b200.models.registry import ARCHITECTURES, architecture_of, load_model_config
    cfg, mw = model("mixed")
    write_mixer_checkpoint(mw, tmp_path)
    assert architecture_of(tmp_path).name == "Degedra" and load_model_config(tmp_path) == cfg
    got = load_any(tmp_path).load_model()
    a, b = named_tensors(mw), named_tensors(got)
    assert a.keys() == b.keys() and all(torch.equal(a[k], b[k]) for k in a)
    assert "l2.norm1" not in a and got.layers[2] is got.layers[0] and got.layers[1].down is None
    assert ARCHITECTURES["Qwen3.5"].tensor_parallel and not ARCHITECTURES["Degedra"].tensor_parallel
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "nothing"}))
    with pytest.raises(ValueError):
        architecture_of(tmp_path)
    (tmp_path / "config.json").write_text(json.dumps({"text_config": {}}))
    assert architecture_of(tmp_path).name == "Qwen3.5"


def test_loader_checks_shapes(tmp_path):
    from mi50grad_b200.loaders.mixer import DegedraLoader
    from mi50grad_b200.models.mixer_weights import write_mixer_checkpoint
    cfg, mw = model("odd_width")
    mw.layers[1].k = mw.layers[1].k[:-1]
    write_mixer_checkpoint(mw, tmp_path)
    ld = DegedraLoader(tmp_path)
    ld.load_layer(0)
    with pytest.raises(ValueError):
        ld.load_layer(1)


def test_trace_runner_refuses_a_type_the_model_has_not(tmp_path, capsys):
    from mi50grad_b200.generate.trace import main
    (tmp_path / "config.json").write_text(json.dumps({"text_config": {}}))
    assert main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "8"]) == 3


def test_slots_are_handed_out_and_reused():
    from mi50grad_b200.engine.state import MixerStates
    st = MixerStates(mixed_config(), 32, 2, "cpu", torch.float32)
    a, b = st.acquire(), st.acquire()
    assert {a, b} == {0, 1}
    with pytest.raises(RuntimeError):
        st.acquire()
    st.set_length(b, 5)
    for t in st.S + st.conv:
        t.fill_(3.0)
    st.release(b)
    with pytest.raises(ValueError):
        st.release(b)
    assert st.acquire() == b and st.length(b) == 0
    assert all(float(t[b].abs().sum()) == 0 and float(t[a].abs().min()) == 3 for t in st.S)
    sd = st.state_dict(a)
    st.reset()
    st.load_state_dict(sd, a)
    assert all(float(t[a].abs().min()) == 3 for t in st.S)


def test_states_count_their_bytes():
    cfg = mixed_config()
    from mi50grad_b200.engine.state import MixerStates
    st = MixerStates(cfg, 64, 3, "cpu", torch.bfloat16)
    assert st.nbytes() == cfg.cache_bytes(64, 3, 2) + cfg.state_bytes(3, 2)


def test_gate_up_interleave():
    from mi50grad_b200.engine.mixer_engine import gemv_outputs_per_cta, interleave_dense_gate_up
    g, u = torch.randn(19, 6), torch.randn(19, 6)
    w = interleave_dense_gate_up(g, u)
    assert w.shape == (48, 6)
    for j in range(24):
        r = (j // 8) * 16 + j % 8
        want = (g[j], u[j]) if j < 19 else (torch.zeros(6), torch.zeros(6))
        assert torch.equal(w[r], want[0]) and torch.equal(w[r + 8], want[1])
    for n in (1, 7, 500, 5000, 50000, 200000):
        assert gemv_outputs_per_cta(n, True) in (16, 32, 64, 128)
        assert gemv_outputs_per_cta(n, False) in (8, 16, 32) and gemv_outputs_per_cta(n, False, True) in (16, 32)


@pytest.mark.parametrize("name", ["mixed", "odd_width"])
def test_oracle_portions_equal_whole(name):
    cfg, mw = model(name)
    t = ids(cfg, 50)
    o = oracle(mw)
    whole = o.forward(t)
    o.reset()
    parts = torch.cat([o.forward(t[a:b]) for a, b in ((0, 2), (2, 3), (3, 20), (20, 21), (21, 50))])
    assert torch.allclose(whole, parts, atol=1e-10)


def test_oracle_window_and_rotation_by_hand():
    # one key far outside, one just outside, one just inside the window, all with large scores
    q, k, v = torch.zeros(1, 1, 4), torch.zeros(10, 1, 4), torch.zeros(10, 1, 4)
    q[0, 0, 0] = 1.0
    for j, val in ((0, 50.0), (5, 40.0), (6, 30.0)):
        k[j, 0, 0], v[j, 0, 1] = val, val
    out = O.window_attention(q, k, v, 1.0, 4, q0=9)
    assert abs(float(out[0, 0, 1]) - 30.0) < 1e-4
    assert abs(float(O.window_attention(q, k, v, 1.0, 5, q0=9)[0, 0, 1]) - 40.0) < 1e-3
    x = torch.arange(1.0, 7.0).reshape(1, 1, 6)
    r = O.rotate_half(x, torch.tensor([3]), 4, 100.0)
    import math
    for i, f in ((0, 1.0), (1, 0.1)):
        c, s = math.cos(3 * f), math.sin(3 * f)
        assert abs(float(r[0, 0, i]) - (x[0, 0, i] * c - x[0, 0, i + 2] * s)) < 1e-5
        assert abs(float(r[0, 0, i + 2]) - (x[0, 0, i + 2] * c + x[0, 0, i] * s)) < 1e-5
    assert torch.equal(r[0, 0, 4:], x[0, 0, 4:])


def test_oracle_recurrence_by_hand():
    # one head, state and column of size one: S = a S + dt B x
    x, B, C, dt = torch.tensor([[[2.0]], [[3.0]]]), torch.tensor([[[0.5]], [[1.0]]]), torch.ones(2, 1, 1), torch.tensor([[0.1], [0.2]])
    y, S = O.ssd_recurrence(x, B, C, dt, torch.zeros(1), torch.tensor([10.0]), torch.full((1, 1, 1), 4.0))
    import math
    s1 = math.exp(-0.1) * 4 + 0.1 * 0.5 * 2
    s2 = math.exp(-0.2) * s1 + 0.2 * 3
    assert abs(float(y[0]) - (s1 + 20)) < 1e-5 and abs(float(y[1]) - (s2 + 30)) < 1e-5 and abs(float(S) - s2) < 1e-6
