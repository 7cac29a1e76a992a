"""Vekerax on the CPU: configuration, registry, checkpoint reader and writer, slots, and the oracle's own
consistency."""
import dataclasses
import json
import math

import pytest
import torch

from degedra_cases import ids
from vekerax_cases import A, CONFIGS, R, layer, mixed_config, model, oracle
import vekerax_oracle as O


def test_config_round_trip():
    from mi50grad_b200.config import vekerax_config_from_dict, vekerax_config_to_dict
    for make in CONFIGS.values():
        cfg = make()
        d = json.loads(json.dumps(vekerax_config_to_dict(cfg)))
        assert vekerax_config_from_dict(d) == cfg
        assert cfg.run_order() == O.layer_order(d)
    assert mixed_config().run_order() == [0, 1, 2, 3, 1, 2, 3, 4] and mixed_config().num_hidden_layers == 5
    assert [a is not None for a, _ in mixed_config().run_mixers()] == [False, True, True, False, True, True, False, True]


def test_config_rejects_what_it_cannot_run():
    from mi50grad_b200.config import VekeraxConfig, vekerax_config_from_dict, vekerax_config_to_dict
    c = vekerax_config_to_dict(mixed_config())
    for path, val in (((1, "type"), "other"), ((1, "mixer", "kv_heads"), 5), ((1, "mlp", "kind"), "other"), ((0, "mixer", "decay"), [0.5]),
                      ((0, "mixer", "decay"), [0.5, 0.5, 0.5, 0.5, 1.5]), ((1, "mixer", "vdim"), 300)):
        bad = json.loads(json.dumps(c))
        d = bad["layers"][path[0]]
        for k in path[1:-1]:
            d = d[k]
        d[path[-1]] = val
        with pytest.raises(ValueError):
            vekerax_config_from_dict(bad)
    for kw in (dict(loop=(1, 3, 2)), dict(loop=(2, 1, 2)), dict(streams=99)):
        with pytest.raises(ValueError):
            VekeraxConfig(32, 10, 1e-5, [layer(A(2, 1, 16, 16, 4)), layer(R(2, 8, 8))], **kw)


@pytest.mark.parametrize("name", CONFIGS)
def test_registry_and_loader(tmp_path, name):
    from mi50grad_b200.loaders import load_any
    from mi50grad_b200.models.registry import ARCHITECTURES, architecture_of, load_model_config
    from mi50grad_b200.models.vekerax_weights import named_tensors, write_vekerax_checkpoint
    cfg, mw = model(name)
    write_vekerax_checkpoint(mw, tmp_path)
    assert architecture_of(tmp_path).name == "Vekerax" and load_model_config(tmp_path) == cfg
    ld = load_any(tmp_path)
    a, b = named_tensors(mw), named_tensors(ld.load_model())
    assert a.keys() == b.keys() and all(torch.equal(a[k], b[k]) for k in a)
    assert torch.equal(ld.load_lm_head(), mw.embed)
    assert ("l0.hc1.mix" in a) == (cfg.streams > 0)
    assert ARCHITECTURES["Vekerax"].dtypes == ("bfloat16", "float32") and not ARCHITECTURES["Vekerax"].tensor_parallel


def test_loader_checks_shapes(tmp_path):
    from mi50grad_b200.loaders.mixer import VekeraxLoader
    from mi50grad_b200.models.vekerax_weights import write_vekerax_checkpoint
    cfg, mw = model("mixed")
    mw.layers[1].v = mw.layers[1].v[:-1]
    write_vekerax_checkpoint(mw, tmp_path)
    ld = VekeraxLoader(tmp_path)
    ld.load_layer(0)
    with pytest.raises(ValueError):
        ld.load_layer(1)


def test_every_run_has_its_own_history():
    from mi50grad_b200.engine.state import MixerStates
    cfg = mixed_config()
    st = MixerStates(cfg, 32, 2, "cpu", torch.bfloat16)
    assert len(st.k) == len(st.S) == 8
    assert st.k[1].shape == (2, 32, 2, 40) and st.v[1].shape == (2, 32, 2, 24) and st.S[1].numel() == 0
    assert st.S[0].shape == (2, 5, 17, 33) and st.k[0].numel() == 0
    assert st.nbytes() == cfg.cache_bytes(32, 2, 2) + cfg.state_bytes(2, 2)
    assert len({t.data_ptr() for t in st.k if t.numel()}) == 5
    b = st.acquire()
    st.set_length(b, 5)
    for t in st.S:
        t.fill_(3.0)
    sd = st.state_dict(b)
    st.release(b)
    assert st.acquire() == b and st.length(b) == 0 and all(float(t[b].abs().sum()) == 0 for t in st.S)
    st.load_state_dict(sd, b)
    assert st.length(b) == 5 and all(float(t[b].abs().min()) == 3 for t in st.S if t.numel())


@pytest.mark.parametrize("name", CONFIGS)
def test_oracle_portions_equal_whole(name):
    cfg, mw = model(name)
    t = ids(cfg, 50)
    o = oracle(mw)
    whole = o.forward(t)
    o.reset()
    parts = torch.cat([o.forward(t[a:b]) for a, b in ((0, 2), (2, 3), (3, 20), (20, 21), (21, 50))])
    assert torch.allclose(whole, parts, atol=1e-10)


def test_visibility_by_hand():
    see = lambda i, **kw: [j for j in range(i + 2) if O.visible(i, j, **kw)]
    assert see(9, window=3, keep=2) == [0, 1, 7, 8, 9]
    assert see(3, window=3, keep=2) == [0, 1, 2, 3]
    assert see(0, window=3, keep=2) == [0] and see(4, window=None, keep=0) == [0, 1, 2, 3, 4]
    assert see(5, window=2, keep=4) == [0, 1, 2, 3, 4, 5] and see(6, window=1, keep=0) == [6]


def test_sink_and_cap_by_hand():
    # two keys with scores 2 and -1 (scale 0.5), cap 4: weights over e^s1 + e^s2 + e^sink; the sink is neither scaled nor capped
    q, k, v = torch.ones(1, 1, 1), torch.tensor([4.0, -2.0]).reshape(2, 1, 1), torch.tensor([1.0, 10.0]).reshape(2, 1, 1)
    out = float(O.sink_attention(q, k, v, 0.5, 4.0, None, 0, torch.tensor([5.0]), q0=1))
    s = [4 * math.tanh(2 / 4), 4 * math.tanh(-1 / 4)]
    e = [math.exp(x) for x in s]
    assert abs(out - (e[0] + 10 * e[1]) / (e[0] + e[1] + math.exp(5.0))) < 1e-5


def test_recurrence_and_gate_by_hand():
    o, S = O.decayed_outer_recurrence(torch.tensor([[[2.0]], [[3.0]]]), torch.tensor([[[0.5]], [[4.0]]]), torch.tensor([[[1.0]], [[-1.0]]]),
                                      [0.25], torch.full((1, 1, 1), 8.0))
    assert abs(float(o[0]) - 2 * 2.5) < 1e-6 and abs(float(S) - (0.25 * 2.5 - 4)) < 1e-6 and abs(float(o[1]) - 3 * (0.625 - 4)) < 1e-6
    y = O.norm_then_gate(torch.tensor([[3.0, -4.0]]), torch.tensor([[0.0, 1.0]]), torch.tensor([2.0, 1.0]), 0.0)
    r = math.sqrt(12.5)
    assert abs(float(y[0, 0]) - 3 / r) < 1e-6 and abs(float(y[0, 1]) + 4 / r / (1 + math.exp(-1))) < 1e-6


def test_streams_by_hand():
    # row of M: where a part comes from; column: where it goes
    xs = torch.tensor([1.0, 10.0]).reshape(2, 1, 1)
    M, b = torch.tensor([[1.0, 2.0], [3.0, 4.0]]), torch.tensor([0.5, -1.0])
    new = O.streams_out(xs, M, b, 0.1, torch.tensor([[20.0]]))
    assert abs(float(new[0]) - (1 + 30 + 1)) < 1e-5 and abs(float(new[1]) - (2 + 40 - 2)) < 1e-5
    assert float(O.streams_in(xs, torch.tensor([2.0, 0.5]))) == 7.0


def test_plain_residual_equals_one_neutral_stream():
    """A model without hyper-connections is one with a single stream whose weights are all one."""
    cfg, mw = model("bare")
    one = dataclasses.replace(cfg, streams=1)
    ones = {f"hc{q}_{n}": torch.ones(*s) for q in (1, 2) for n, s in (("in", (1,)), ("out", (1,)), ("mix", (1, 1)))}
    m2 = dataclasses.replace(mw, config=one, layers=[dataclasses.replace(l, **ones) for l in mw.layers])
    t = ids(cfg, 30)
    assert torch.allclose(oracle(mw).forward(t), oracle(m2).forward(t), atol=1e-12)
