"""bench.py's command-line contract that can be checked without a GPU."""
import json
import os
import subprocess
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_reference_arm_reports_unavailable():
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bench.py"), "--impl", "reference", "--gpus", "1",
                        "--steps", "4", "--warmup", "3"], capture_output=True, text=True, timeout=120)
    assert r.returncode == 0
    d = json.loads(r.stdout.strip().splitlines()[-1])
    assert d["impl"] == "reference" and "unavailable" in d and "\n" not in d["unavailable"]


def test_arguments_and_docstring():
    src = open(os.path.join(ROOT, "bench.py")).read()
    for flag in ("--gpus", "--steps", "--warmup", "--impl"):
        assert flag in src
    for key in ('"metric"', '"value"', '"unit"', '"n_gpus"', '"ms_per_step"', '"higher_is_better"', '"scaling"',
                '"vs_baseline"', '"dtype"', '"data"', '"config"', '"clocks"', '"e2e"', '"gpu_launches"'):
        assert key in src, key


def test_degedra_mode_compares_models_of_equal_size():
    src = open(os.path.join(ROOT, "bench.py")).read()
    assert '"degedra"' in src and 'default="decode"' in src
    from mi50grad_b200.bench.degedra import SIZES, degedra_config, hybrid_config
    for size in SIZES:
        d, h = degedra_config(size), hybrid_config(size)
        l = d.layers[0]
        assert (d.hidden_size, l.ff, len(d.layers), d.vocab_size) == (h.hidden_size, h.intermediate_size, h.num_hidden_layers, h.vocab_size)
        assert l.attention.heads * l.attention.dim == h.full_attn_q_dim
        assert l.ssd.inner == h.linear_attn_value_dim


def test_vekerax_mode_compares_models_of_equal_size():
    src = open(os.path.join(ROOT, "bench.py")).read()
    assert '"vekerax": ("vekerax", "degedra")' in src
    from mi50grad_b200.bench.degedra import SIZES, degedra_config, vekerax_config
    for size in SIZES:
        v, d = vekerax_config(size), degedra_config(size)
        assert (v.hidden_size, v.vocab_size, len(v.layers), v.layers[0].ff) == (d.hidden_size, d.vocab_size, len(d.layers), d.layers[0].ff)
        a, r, l = v.layers[0].attention, v.layers[1].recurrence, d.layers[0]
        assert (a.heads, a.kv_heads, a.dim, a.vd, a.window) == (l.attention.heads, l.attention.kv_heads, l.attention.dim, l.attention.vd, l.attention.window)
        assert r.heads * r.state * r.vdim == l.ssd.heads * l.ssd.state * l.ssd.vdim and r.inner == l.ssd.inner
