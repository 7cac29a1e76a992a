"""The Vekerax decoder in the engine against the plain implementation: prompts, decoding through the cache,
portions, batches, slots used again, generation through the public entry points."""
import dataclasses
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from degedra_cases import close, ids, row_errors
from vekerax_cases import CONFIGS, A, R, layer, model, oracle

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BOTH = ["bfloat16", "float32"]


def engine(mw, dtype, max_seq=320, **kw):
    from mi50grad_b200.engine.vekerax_engine import VekeraxEngine
    e = VekeraxEngine(mw.config, max_seq_len=max_seq, dtype=dtype, **kw)
    e.load_model(mw)
    return e


_cache = {}


def setup(name, dtype):
    """(config, weights, engine, tokens, oracle logits of a 200-token request), built once."""
    if name not in _cache:
        cfg, mw = model(name)
        t = ids(cfg, 200, seed=1)
        _cache[name] = [cfg, mw, t, oracle(mw).forward(t), {}]
    cfg, mw, t, ref, eng = _cache[name]
    if dtype not in eng:
        eng[dtype] = engine(mw, dtype, max_batch=3)
    eng[dtype].reset()
    return cfg, mw, eng[dtype], t, ref


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", CONFIGS)
def test_whole_prompt(name, dtype):
    cfg, mw, eng, t, ref = setup(name, dtype)
    assert close(eng.forward_tokens(t, want=range(200)), ref, dtype)
    eng.check_status()
    x = []
    oracle(mw).forward(t[:40], x)
    eng.reset()
    eng.forward_tokens(t[:40])
    got = eng.buf["p_h"][39].double().cpu()
    assert float((got - x[-1][-1]).abs().max() / x[-1][-1].abs().max()) < {"bfloat16": 0.1, "float32": 3e-5}[dtype]
    short = []
    for n in (1, 2, 8, 9, 17):
        eng.reset()
        short.append(eng.forward_tokens(t[:n], want=range(n)))
    assert close(torch.cat(short), torch.cat([ref[:s.shape[0]] for s in short]), dtype)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", CONFIGS)
def test_every_run_of_a_layer(name, dtype):
    """The residual streams' sum after each run, from models cut off behind it."""
    cfg, mw = model(name)
    t, x = ids(cfg, 33, seed=4), []
    oracle(mw).forward(t, x)
    order = cfg.run_order()
    for r in range(1, len(order) + 1):
        c = dataclasses.replace(cfg, layers=[cfg.layers[i] for i in order[:r]], loop=None)
        e = engine(dataclasses.replace(mw, config=c, layers=[mw.layers[i] for i in order[:r]]), dtype, max_seq=64)
        e.forward_tokens(t)
        a = e.buf["p_h"][:33].double().cpu()
        e.reset()
        e.step_tokens(t[:1])
        b = e.residual_stream(1).double().cpu()
        for got, want in ((a, x[r - 1]), (b, x[r - 1][:1])):
            assert float((got - want).abs().max() / x[r - 1].abs().max()) < {"bfloat16": 0.1, "float32": 3e-5}[dtype], r


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", CONFIGS)
def test_token_by_token(name, dtype):
    cfg, mw, eng, t, ref = setup(name, dtype)
    n = 120 if name != "odd_width" else 200
    lg = torch.cat([eng.forward_tokens([tok], want=[0]) for tok in t[:n]])
    assert close(lg, ref[:n], dtype)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", CONFIGS)
@pytest.mark.parametrize("sizes", [[2] * 100, [2, 7, 9, 31, 1, 64, 3, 16, 33, 34], [100, 1, 1, 2, 63, 1, 32], [65, 64, 71]])
def test_portions(name, dtype, sizes):
    cfg, mw, eng, t, ref = setup(name, dtype)
    assert sum(sizes) == 200
    out, i = [], 0
    for n in sizes:
        out.append(eng.forward_tokens(t[i:i + n], 2, want=range(n)))
        i += n
    assert close(torch.cat(out), ref, dtype)


@pytest.mark.parametrize("dtype", BOTH)
def test_prompt_longer_than_a_launch(dtype):
    cfg, mw = model("plain", seed=3, window=40, keep=3)
    t = ids(cfg, 700, seed=2)
    ref = oracle(mw).forward(t)
    assert close(engine(mw, dtype, max_seq=704).forward_tokens(t, want=range(0, 700, 7)), ref[::7], dtype)


@pytest.mark.parametrize("dtype", BOTH)
def test_batches_equal_single_requests(dtype):
    """Unequal requests decoded together against each alone: few rows, and more sequences than the few-row
    kernels take."""
    cfg, mw = model("mixed", seed=5)
    eng = engine(mw, dtype, max_seq=128, max_batch=11)
    lens = [1, 70, 2, 33, 9, 16, 8, 64, 65, 40, 5]
    prompts = [ids(cfg, n, seed=n) for n in lens]
    alone, logits = [], []
    for p in prompts:
        eng.reset(0)
        first = eng.prefill_tokens(p, 0)
        alone.append([first] + eng.decode_tokens(6, [0])[:, 0].tolist())
        logits.append(eng.logits(1)[0].clone())
    for group in ([3, 0, 7], list(range(8)), list(range(11))):
        for graph in (True, False):
            eng.reset()
            first = [eng.prefill_tokens(prompts[s], s) for s in group]
            out = eng.decode_tokens(6, group, graph=graph).cpu()
            lg = eng.buf["p_logits" if len(group) > 8 else "logits"][:len(group), :cfg.vocab_size]
            for j, s in enumerate(group):
                got = [first[j]] + out[:, j].tolist()
                if dtype == "float32":
                    assert got == alone[s]
                if got == alone[s]:
                    assert close(lg[j:j + 1], logits[s][None], dtype)
        assert [eng.states.length(s) for s in group] == [lens[s] + 6 for s in group]


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("name", ["mixed", "plain"])
def test_slots_used_again(name, dtype):
    cfg, mw, eng, t, ref = setup(name, dtype)
    a = eng.states.acquire()
    eng.forward_tokens(ids(cfg, 150, seed=8), a)
    for tok in ids(cfg, 5, seed=9):
        eng.forward_tokens([tok], a)
    eng.states.release(a)
    b = eng.states.acquire()
    assert b == a
    got = torch.cat([eng.forward_tokens(t[:60], b, want=range(60)), eng.forward_tokens([t[60]], b, want=[0])])
    eng.states.release(b)
    assert close(got, ref[:61], dtype)
    fresh = engine(mw, dtype)
    assert torch.equal(got, torch.cat([fresh.forward_tokens(t[:60], want=range(60)), fresh.forward_tokens([t[60]], want=[0])]))


@pytest.mark.parametrize("dtype", BOTH)
def test_snapshot_restore_and_dry_run(dtype):
    cfg, mw, eng, t, ref = setup("mixed", dtype)
    eng.forward_tokens(t[:40])
    snap, sd = eng.states.snapshot(0), eng.states.state_dict(0)
    a = eng.forward_tokens(t[40:80], want=range(40))
    eng.states.restore(snap)
    eng.step_tokens(t[100:105], commit=False)
    assert eng.states.length(0) == 40
    assert torch.equal(a, eng.forward_tokens(t[40:80], want=range(40)))
    eng.reset()
    eng.states.load_state_dict(sd, 1)
    assert torch.equal(eng.forward_tokens(t[40:80], 1, want=range(40)), a)


@pytest.mark.parametrize("dtype", BOTH)
def test_far_keys_stand_out_in_the_model(dtype):
    """One attention layer whose queries match single keys sharply: a token repeated far back, in front of and
    behind the window's edge, and a kept first token; prompts, portions and decoding."""
    from mi50grad_b200.config import VekeraxConfig
    from mi50grad_b200.models.vekerax_weights import random_vekerax_model
    window, keep = 33, 3
    cfg = VekeraxConfig(64, 200, 1e-5, [layer(A(4, 2, 32, 16, window, keep, 30.0, 1.0), 48), layer(R(2, 16, 16, 0.9, 0.999), 48)],
                        embedding_scale=8.0, residual_mult=1.0, streams=2)
    mw = random_vekerax_model(cfg, 6)
    # queries are keys with the width's columns permuted: token 100 + j asks for token j (and not for itself)
    w, perm = mw.layers[0], torch.randperm(64, generator=torch.Generator().manual_seed(0))
    w.q = torch.empty(128, 64, dtype=torch.bfloat16)
    w.q[:, perm] = torch.cat([w.k[:32], w.k[:32], w.k[32:], w.k[32:]])
    w.q_norm, w.k_norm, w.norm1, w.sink = *(torch.ones(n).bfloat16() for n in (32, 32, 64)), -5 * torch.ones(4).bfloat16()
    mw.embed[100 + perm.new_tensor(range(100))[:, None], perm[None]] = mw.embed[:100].clone()
    t = list(range(100))
    for i, j in ((60, 60 - window + 1), (61, 61 - window), (70, keep - 1), (71, keep), (90, 90 - window + 1), (91, 91 - window), (95, 0)):
        t[i] = 100 + t[j]
    o = oracle(mw)
    ref = o.forward(t)
    eng = engine(mw, dtype, max_seq=128)
    for cuts in ([100], [59, 1, 1, 8, 1, 1, 19, 10], [50] + [1] * 50, [2] * 50):
        eng.reset()
        out, i = [], 0
        for n in cuts:
            out.append(eng.forward_tokens(t[i:i + n], want=range(n)))
            i += n
        assert close(torch.cat(out), ref, dtype)
    # a window or a count of kept tokens that is one off is far outside the tolerance at those places
    for places, a in (([60, 90], dict(window=window - 1)), ([61, 91], dict(window=window + 1)), ([70], dict(keep_first=keep - 1)),
                      ([71], dict(keep_first=keep + 1)), ([95], dict(keep_first=0))):
        l0 = dataclasses.replace(cfg.layers[0], mixer=dataclasses.replace(cfg.layers[0].mixer, **a))
        wrong = oracle(dataclasses.replace(mw, config=dataclasses.replace(cfg, layers=[l0, cfg.layers[1]]))).forward(t)
        assert float(row_errors(wrong, ref)[places].min()) > 0.25, (places, a)


@pytest.mark.parametrize("dtype", BOTH)
def test_long_decoding(dtype):
    """Far beyond the window, with a sharp soft-max (large attention scale), forced tokens."""
    cfg, mw = model("mixed", seed=11)
    for i, l in enumerate(cfg.layers):
        if l.attention is not None:
            cfg.layers[i] = dataclasses.replace(l, mixer=dataclasses.replace(l.mixer, scale=0.5, window=23 + 20 * i, softcap=25.0))
    t = ids(cfg, 420, seed=4)
    ref = oracle(mw).forward(t)
    eng = engine(mw, dtype, max_seq=420)
    eng.forward_tokens(t[:20])
    assert close(torch.cat([eng.forward_tokens([tok], want=[0]) for tok in t[20:]]), ref[20:], dtype, 2.0)
    with pytest.raises(ValueError):
        eng.forward_tokens([1])


def test_greedy_generation_matches_the_oracle(tmp_path):
    from mi50grad_b200.generate.generate import TextGenerator, load_and_generate
    from mi50grad_b200.generate.sampler import SamplingParams
    from mi50grad_b200.models.registry import build_engine
    from mi50grad_b200.models.vekerax_weights import write_vekerax_checkpoint
    cfg, mw = model("mixed", seed=7)
    write_vekerax_checkpoint(mw, tmp_path)
    eng, _ = build_engine(str(tmp_path), max_seq_len=160, dtype="float32")
    gen = TextGenerator(eng)
    o = oracle(mw)
    for n in (1, 5, 40):
        p = ids(cfg, n, seed=n)
        want = o.greedy(p, 24)
        assert gen.generate_ids(p, SamplingParams(temperature=0.0, max_tokens=24)) == want
        assert eng.generate_tokens(p, 24) == want and eng.generate_tokens(p, 24, graph=False) == want
    # bf16 through the one-call entry point: every token is the oracle's choice up to rounding
    p = ids(cfg, 30, seed=30)
    text = load_and_generate(str(tmp_path), p, max_tokens=16, temperature=0.0, max_seq_len=96)
    got = [int(x) for x in text.split()]
    assert len(got) == 16
    lg = oracle(mw).forward(p + got[:-1])[len(p) - 1:]
    gap = lg.max(-1).values - lg.gather(1, torch.tensor(got)[:, None])[:, 0]
    assert float(gap.max() / lg.pow(2).mean().sqrt()) < 0.15


def test_sampling_on_the_device():
    from mi50grad_b200.generate.generate import TextGenerator
    from mi50grad_b200.generate.sampler import SamplingParams
    cfg, mw, eng, t, ref = setup("plain", "bfloat16")
    gen = TextGenerator(eng)
    par = SamplingParams(temperature=0.8, top_k=20, top_p=0.9, repetition_penalty=1.1, max_tokens=12, seed=3)
    a, b = gen.generate_ids(t[:20], par), gen.generate_ids(t[:20], par)
    assert a == b and len(a) == 12 and all(0 <= x < cfg.vocab_size for x in a)


def test_scores_and_embedding_interface():
    cfg, mw, eng, t, ref = setup("mixed", "float32")
    lp = eng.score_tokens(t[:100])
    want = torch.log_softmax(ref[:99], -1).gather(1, torch.tensor(t[1:100])[:, None])[:, 0]
    assert float((lp.double().cpu() - want).abs().max()) < 1e-3
    eng.reset()
    emb = lambda s: mw.embed[torch.tensor(s)].float()           # rows of the table: the engine scales them
    hid = eng.prefill_step(emb(t[:40]))
    assert row_errors(eng.compute_logits(hid)[None], ref[39:40]).max() < 1e-4
    hid = eng.decode_step(emb(t[40:41])[0])
    assert row_errors(eng.compute_logits(hid)[None], ref[40:41]).max() < 1e-4
    h = eng.forward_embeddings(emb(t[41:44]))
    assert row_errors(eng.compute_logits(h[2])[None], ref[43:44]).max() < 1e-4
    with pytest.raises(NotImplementedError):
        eng.spec_step([[1]], [[-1]])


def test_lazy_rows_make_no_difference(monkeypatch):
    """Streams updated in the projections against streams updated by a launch of their own."""
    cfg, mw, eng, t, ref = setup("mixed", "float32")
    monkeypatch.setenv("B200GRAD_LAZY_ROWS", "8")
    fused = engine(mw, "float32")
    monkeypatch.setenv("B200GRAD_LAZY_ROWS", "0")
    apart = engine(mw, "float32")
    for n in (1, 5, 8):
        for e in (fused, apart):
            e.reset()
            assert close(e.forward_tokens(t[:n], want=range(n)), ref[:n], "float32")


def test_guard_bands_stay_clean():
    from mi50grad_b200.config import EngineConfig
    for name in CONFIGS:
        cfg, mw = model(name)
        for dtype in BOTH:
            eng = engine(mw, dtype, engine_config=EngineConfig(debug_guards=True, use_graph=False), max_batch=10)
            for n in (1, 3, 13, 40, 150):
                eng.reset(0)
                eng.forward_tokens(ids(cfg, n), want=[0, n - 1])
                eng.decode_tokens(2, [0])
                eng.check_guards()
            for s in range(10):
                eng.prefill_tokens(ids(cfg, 3 + s), s)
            eng.decode_tokens(2, list(range(10)))
            eng.check_guards()


@pytest.mark.parametrize("dtype", BOTH)
def test_trace_runner(tmp_path, dtype):
    from mi50grad_b200.models.vekerax_weights import write_vekerax_checkpoint
    cfg, mw = model("bare", seed=2)
    write_vekerax_checkpoint(mw, tmp_path / "m")
    (tmp_path / "out").mkdir()
    t, u = ids(cfg, 60, seed=1), ids(cfg, 20, seed=2)
    steps = [[("a", t[:33], [0, 32])], [("a", t[33:34], [0])], [("b", u[:2], [])], [("a", t[34:60], [1, 25]), ("b", u[2:], [17, 3])]]
    lines = [json.dumps({"step": i, "entries": [{"id": n, "tokens": x, "want": w} for n, x, w in st],
                         "end": ["a", "b"] if i == 3 else []}) for i, st in enumerate(steps)]
    lines.append(json.dumps({"step": 4, "entries": [{"id": "c", "tokens": u, "want": [19]}], "end": ["c"]}))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype,
                        "--out", str(tmp_path / "out"), "--max-tokens", "80"], input="\n".join(lines) + "\n",
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    read = lambda i, n: torch.from_numpy(np.fromfile(tmp_path / "out" / f"{i}.f32", dtype="<f4")).reshape(n, cfg.vocab_size)
    ra, rb = oracle(mw).forward(t), oracle(mw).forward(u)
    assert close(read(0, 2), ra[[0, 32]], dtype) and close(read(1, 1), ra[[33]], dtype)
    assert not (tmp_path / "out" / "2.f32").exists()
    assert close(read(3, 4), torch.cat([ra[[35, 59]], rb[[19, 5]]]), dtype)
    assert close(read(4, 1), rb[[19]], dtype)
