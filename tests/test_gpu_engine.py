"""The CUDA engine against the fp32 oracle on the tiny hybrid model."""
import pytest
import torch

from helpers import cosine

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def setup():
    from mi50grad_b200.config import tiny_config
    from mi50grad_b200.engine.engine import InferenceEngine
    from mi50grad_b200.models.oracle import OracleEngine
    from mi50grad_b200.models.weights import random_model
    cfg = tiny_config()
    mw = random_model(cfg, 0)
    eng = InferenceEngine(cfg, max_seq_len=256, max_batch=2)
    eng.load_model(mw)
    return cfg, mw, eng, OracleEngine(mw, max_seq_len=256, max_batch=2)


def _prompt(cfg, n=16, seed=0):
    return torch.randint(0, cfg.vocab_size, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def test_hidden_states_match_oracle(setup):
    cfg, mw, eng, orc = setup
    eng.states.reset(); orc.reset()
    ids = _prompt(cfg, 13)
    x_ref = orc.forward(orc.embed(ids))
    hs = []
    for i in range(0, len(ids), 8):
        eng.step_tokens(ids[i:i + 8], logits=False)
        hs.append(eng.residual_stream(len(ids[i:i + 8])).clone())
    x = torch.cat(hs).cpu()
    for r in range(len(ids)):
        assert cosine(x[r], x_ref[r]) > 0.999, f"row {r}"
    assert (x - x_ref).abs().max() / x_ref.abs().max() < 2e-2
    assert eng.states.length(0) == 13


def test_greedy_tokens_and_logits_match_oracle(setup):
    cfg, mw, eng, orc = setup
    orc.reset()
    ids = _prompt(cfg, 16)
    ref_toks, ref_logits = orc.greedy_generate(ids, 8)
    toks = eng.generate_tokens(ids, 8, graph=False)
    assert toks == ref_toks
    lg = eng.logits(1)[0].cpu()
    assert cosine(lg, ref_logits[-1]) > 0.999


def test_graph_replay_equals_eager_bitwise(setup):
    cfg, mw, eng, orc = setup
    ids = _prompt(cfg, 9, seed=3)
    a = eng.generate_tokens(ids, 12, graph=False)
    la = eng.logits(1).clone()
    b = eng.generate_tokens(ids, 12, graph=True)
    lb = eng.logits(1).clone()
    assert a == b and torch.equal(la, lb)
    assert eng.states.length(0) == 9 + 11
    # replay many tokens without collecting
    eng.decode_tokens(5, collect=False)
    assert eng.states.length(0) == 9 + 16


def test_embedding_in_hidden_out_api(setup):
    cfg, mw, eng, orc = setup
    eng.states.reset(); orc.reset()
    ids = _prompt(cfg, 6, seed=4)
    emb = orc.embed(ids)
    h_ref = orc.prefill_step(emb)
    h = eng.prefill_step(emb.numpy())
    assert h.dtype.name == "float16" and cosine(torch.from_numpy(h).float(), h_ref) > 0.999
    e1 = orc.embed([5])[0]
    d_ref = orc.decode_step(e1, position=6)
    d = eng.decode_step(e1.numpy(), position=6)
    assert cosine(torch.from_numpy(d).float(), d_ref) > 0.999
    lg = eng.compute_logits(d)
    assert cosine(torch.from_numpy(lg), orc.compute_logits(d_ref)) > 0.999
    # a long prompt given as embeddings takes the tensor-core path (not eight rows per decode-sized step)
    eng.states.reset(); orc.reset()
    ids = _prompt(cfg, 40, seed=9)
    emb = orc.embed(ids)
    h_ref = orc.prefill_step(emb)
    h = eng.prefill_step(emb.numpy())
    assert cosine(torch.from_numpy(h).float(), h_ref) > 0.999 and eng.states.length(0) == 40
    e1 = orc.embed([7])[0]
    assert cosine(torch.from_numpy(eng.decode_step(e1.numpy(), position=40)).float(),
                  orc.decode_step(e1, position=40)) > 0.999


def test_two_sequences_with_independent_lengths(setup):
    cfg, mw, eng, orc = setup
    eng.states.reset(); orc.reset()
    p0, p1 = _prompt(cfg, 11, seed=5), _prompt(cfg, 4, seed=6)
    t0 = eng.prefill_tokens(p0, seq=0)
    t1 = eng.prefill_tokens(p1, seq=1)
    out = eng.decode_tokens(5, seqs=[0, 1], graph=True).cpu()
    r0, _ = orc.greedy_generate(p0, 6, seq=0)
    r1, _ = orc.greedy_generate(p1, 6, seq=1)
    assert [t0] + out[:, 0].tolist() == r0
    assert [t1] + out[:, 1].tolist() == r1
    assert eng.states.lengths() == [16, 9]


def test_decoding_a_slot_other_than_the_first(setup):
    """The step advances the sequences it decodes, whichever slots they are in."""
    cfg, mw, eng, orc = setup
    eng.states.reset(); orc.reset()
    p = _prompt(cfg, 9, seed=11)
    t = eng.prefill_tokens(p, seq=1)
    out = eng.decode_tokens(6, seqs=[1], graph=True).cpu()
    ref, _ = orc.greedy_generate(p, 7, seq=1)
    assert [t] + out[:, 0].tolist() == ref and eng.states.lengths() == [0, 15]


def test_snapshot_restore_rolls_back_deltanet(setup):
    cfg, mw, eng, orc = setup
    ids = _prompt(cfg, 10, seed=7)
    eng.states.reset()
    eng.prefill_tokens(ids)
    snap = eng.states.snapshot(0)
    a = eng.decode_tokens(4).cpu()
    eng.states.restore(snap)
    b = eng.decode_tokens(4).cpu()
    assert torch.equal(a, b)
    sd = eng.states.state_dict(0)
    eng.states.reset()
    eng.states.load_state_dict(sd)
    c = eng.decode_tokens(2).cpu()
    eng.states.restore(snap); eng.decode_tokens(4)
    d = eng.decode_tokens(2).cpu()
    assert torch.equal(c, d)


def test_fp16_attention_checkpoint_variant():
    from mi50grad_b200.config import tiny_config
    from mi50grad_b200.engine.engine import InferenceEngine
    from mi50grad_b200.models.oracle import OracleEngine
    from mi50grad_b200.models.weights import random_model
    cfg = tiny_config()
    mw = random_model(cfg, 1, int4_attention=False)
    eng = InferenceEngine(cfg, max_seq_len=128)
    eng.load_model(mw)
    orc = OracleEngine(mw, max_seq_len=128)
    ids = _prompt(cfg, 12, seed=8)
    ref, _ = orc.greedy_generate(ids, 6)
    assert eng.generate_tokens(ids, 6) == ref


def test_generator_samples_on_device(setup):
    from mi50grad_b200.generate.generate import TextGenerator
    from mi50grad_b200.generate.sampler import SamplingParams
    cfg, mw, eng, orc = setup
    gen = TextGenerator(eng)
    prm = SamplingParams(temperature=0.8, top_k=20, top_p=0.9, repetition_penalty=1.2, max_tokens=10, seed=5)
    a = gen.generate_ids(_prompt(cfg, 9, seed=11), prm)
    b = gen.generate_ids(_prompt(cfg, 9, seed=11), prm)
    assert a == b and len(a) == 10 and all(0 <= t < cfg.vocab_size for t in a)
    c = gen.generate_ids(_prompt(cfg, 9, seed=11), SamplingParams(temperature=0.8, top_k=20, top_p=0.9, max_tokens=10, seed=6))
    assert c != a or len(set(a)) == 1
    # unseeded: every call draws its own seed, as the host sampler does, so two generations differ
    free = SamplingParams(temperature=1.5, top_k=0, top_p=1.0, max_tokens=16)
    u1 = gen.generate_ids(_prompt(cfg, 9, seed=11), free)
    u2 = gen.generate_ids(_prompt(cfg, 9, seed=11), free)
    u3 = gen.generate_ids(_prompt(cfg, 9, seed=11), free)
    assert not (u1 == u2 == u3)
    # the repetition penalty reaches every distinct past token, however many there are
    from mi50grad_b200.generate.sampler import filtered_probs
    from mi50grad_b200.ops import kernels as K
    g = torch.Generator().manual_seed(3)
    logits = torch.randn(1, 4096, generator=g) * 3
    past = torch.randperm(4096, generator=g)[:2500].tolist()
    pp = SamplingParams(temperature=1.0, top_k=50, top_p=0.95, repetition_penalty=1.7)
    ref = filtered_probs(logits[0].numpy(), pp, past)
    pt = torch.tensor([sorted(set(past))], dtype=torch.int32, device="cuda")
    ids, probs = K.sample_top_p(logits.cuda().clone(), 1.0, 50, 0.95, 1.7, pt,
                                torch.tensor([pt.shape[1]], dtype=torch.int32, device="cuda"), seed=1, debug=True)[1:3]
    got = {int(i): float(p_) for i, p_ in zip(ids[0].tolist(), probs[0].tolist()) if i >= 0}
    assert set(got) == set(int(i) for i in ref.nonzero()[0])
    assert all(abs(got[i] - float(ref[i])) < 2e-5 for i in got)
    # after a short prompt (several rows in one step) the logits offered to the sampler are the last row's
    first = gen.prefill(_prompt(cfg, 5, seed=12))
    assert int(eng.logits(1)[0].argmax()) == first
    assert int(eng.compute_logits(None).argmax()) == first
    first = gen.prefill(_prompt(cfg, 21, seed=13))
    assert int(eng.compute_logits(None).argmax()) == first


def test_debug_guards_see_no_out_of_bounds_write():
    """Every work buffer between poisoned bands: decode, verify and many-row steps leave them intact."""
    from mi50grad_b200.config import EngineConfig, tiny_config
    from mi50grad_b200.engine.engine import InferenceEngine
    from mi50grad_b200.models.weights import random_model
    cfg = tiny_config()
    eng = InferenceEngine(cfg, max_seq_len=128, max_batch=3, engine_config=EngineConfig(debug_guards=True))
    eng.load_model(random_model(cfg, 0))
    for i in range(3):
        eng.prefill_tokens(_prompt(cfg, 20 + i, seed=40 + i), seq=i)     # tensor-core path
        eng.check_guards()
    eng.decode_tokens(3, seqs=[0, 1, 2], graph=False)
    eng.spec_step([[1, 2, 3], [4, 5, 6], [7, 8, 9]], [[-1, 0, 1]] * 3, [0, 1, 2])   # 12 rows: many-row verify
    eng.spec_step([[1, 2]], [[-1, -1]], [0])
    assert eng._guards is not None and len(eng._guards.names()) > 30


@pytest.mark.parametrize("fmt", ["gptq", "awq"])
def test_load_and_generate_from_checkpoint_directory(tmp_path, fmt):
    """Checkpoint on disk -> loaders -> engine -> tokens, through the public one-call API."""
    from mi50grad_b200.config import tiny_config
    from mi50grad_b200.generate.generate import load_and_generate, load_and_generate_eagle
    from mi50grad_b200.models.oracle import OracleEngine
    from mi50grad_b200.models.weights import random_model, write_checkpoint
    cfg = tiny_config()
    mw = random_model(cfg, 3)
    if fmt == "awq":                                           # the zero-less variant: no zero points anywhere
        from mi50grad_b200.utils.quant import Int4Linear
        for lw in mw.layers:
            for name, v in vars(lw).items():
                if isinstance(v, Int4Linear):
                    v.zeros = None
    write_checkpoint(mw, str(tmp_path), fmt)
    ids = _prompt(cfg, 18, seed=21)
    ref, _ = OracleEngine(mw, max_seq_len=128).greedy_generate(ids, 6)
    out = load_and_generate(str(tmp_path), ids, max_tokens=6, temperature=0.0, max_seq_len=128)
    assert out == " ".join(str(t) for t in ref)
    if fmt == "gptq":
        out2 = load_and_generate_eagle(str(tmp_path), ids, max_tokens=6, k_draft=3, max_seq_len=128)
        assert out2 == ref


def test_prompt_longer_than_one_prefill_launch(setup):
    """A 130-token prompt in launches of 48 rows: the chunked scan carries state and conv history
    across launches, attention sees the rows of earlier launches through the cache."""
    cfg, mw, eng, orc = setup
    eng._ensure_driver()
    saved = eng.max_prefill
    try:
        eng.max_prefill = 48
        ids = _prompt(cfg, 130, seed=17)
        orc.reset()
        ref, _ = orc.greedy_generate(ids, 5)
        assert eng.generate_tokens(ids, 5, graph=False) == ref
        assert eng.states.length(0) == 130 + 4
    finally:
        eng.max_prefill = saved


def test_score_tokens_matches_oracle(setup):
    cfg, mw, eng, orc = setup
    ids = _prompt(cfg, 45, seed=23)
    ref = orc.score_tokens(ids)
    got = eng.score_tokens(ids).cpu()
    assert got.shape == ref.shape
    assert (got - ref).abs().max() < 0.05 and abs(eng.perplexity(ids) / orc.perplexity(ids) - 1) < 0.02


@pytest.mark.parametrize("fmt", ["w8a8", "w4a8"])
def test_whole_model_int8_activation_formats(fmt):
    """quant_format w8a8 / w4a8: the FFN of every layer runs on the INT8-activation kernels (decode steps
    and the many-row prefill path); hidden states stay close to the w4a16 engine's and greedy tokens of
    the fp32 oracle are reproduced on a well-separated prompt (reference: tests/test_engine_w8a8_w4a8.py)."""
    from mi50grad_b200.config import tiny_config
    from mi50grad_b200.engine.engine import InferenceEngine
    from mi50grad_b200.models.weights import random_model
    cfg = tiny_config(intermediate_size=768)          # the W4A8 product needs K % 128 == 0 (down: K = FFN width)
    mw = random_model(cfg, 0)
    base = InferenceEngine(cfg, max_seq_len=128)
    base.load_model(mw)
    eng = InferenceEngine(cfg, max_seq_len=128, quant_format=fmt)
    eng.load_model(mw)
    ids = _prompt(cfg, 13, seed=4)
    for e in (base, eng):
        e.states.reset()
        e.step_tokens(ids[:8], logits=False)
        e.step_tokens(ids[8:], logits=True)
    n = len(ids) - 8
    h0, h1 = base.residual_stream(n).float().cpu(), eng.residual_stream(n).float().cpu()
    for r in range(n):
        assert cosine(h1[r], h0[r]) > 0.995, (fmt, r, cosine(h1[r], h0[r]))
    lg0, lg1 = base.logits(n)[n - 1].float().cpu(), eng.logits(n)[n - 1].float().cpu()
    assert cosine(lg1, lg0) > 0.99
    # the many-row path (tensor-core projections + the same INT8 FFN) agrees with the step path
    eng.states.reset()
    first = eng.prefill_tokens(_prompt(cfg, 40, seed=5))
    eng2 = InferenceEngine(cfg, max_seq_len=128, quant_format=fmt)
    eng2.load_model(mw)
    p40 = _prompt(cfg, 40, seed=5)
    for i in range(0, 40, 8):
        out = eng2.step_tokens(p40[i:i + 8], logits=i + 8 >= 40)
    assert cosine(eng.residual_stream(1)[0].float().cpu(), eng2.residual_stream(8)[7].float().cpu()) > 0.995
    assert eng.launches_per_step() > 0 and 0 <= first < cfg.vocab_size
