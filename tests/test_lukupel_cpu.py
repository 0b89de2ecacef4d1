"""CPU: the Lukupel configuration reader and registry entry, the argument blocks of its kernels against a C compiler, and
the plain restatement's own invariants (tests/lukupel_oracle.py)."""
import ctypes as C
import math
import os
import subprocess

import pytest
import torch

import lukupel_oracle as O

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def small_config():
    att = {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 6, "scale": 0.3, "mask": {"size": 5}, "rot": {"base": 100.0, "dims": 4, "scaling": {"factor": 2.0}}}
    mem = {"heads": 3, "dim": 5, "vdim": 7, "gate_cap": 6.0}
    dense = {"kind": "dense", "ff": 20}
    return {"architecture": "Lukupel", "vocab": 30, "width": 16, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0}, "residual_mult": 0.4, "logit_softcap": 9.0,
            "layers": [{"type": "mlstm", "mixer": mem, "mlp": None}, {"type": "attention", "mixer": att, "mlp": dense},
                       {"type": "mlstm", "mixer": dict(mem), "mlp": None, "weights_of": 0}, {"type": "attention", "mixer": dict(att), "mlp": dict(dense), "weights_of": 1},
                       {"type": "attention", "mixer": dict(att), "mlp": dict(dense), "weights_of": 3}]}


def test_config_reader_and_registry():
    from lit_llama_b200 import LukupelConfig, registry

    assert "Lukupel" in registry.architectures()
    c = LukupelConfig.from_dict(small_config())
    assert (c.vocab, c.width, c.eps, c.embedding_scale, c.residual_mult, c.logit_softcap, len(c.layers)) == (30, 16, 1e-5, 3.0, 0.4, 9.0, 5)
    assert [c.owner(i) for i in range(5)] == [0, 1, 0, 1, 1] == [O.owner(c.layers, i) for i in range(5)]
    assert LukupelConfig.from_dict(c.to_dict()) == c
    for breaker in (lambda d: d["layers"][0].update(type="convolution"), lambda d: d["layers"][1]["mlp"].update(kind="maxout"),
                    lambda d: d["layers"][2].update(weights_of=2), lambda d: d["layers"][3].update(weights_of=4), lambda d: d["layers"][2].update(weights_of=9),
                    lambda d: d["layers"][2].update(weights_of=1), lambda d: d["layers"][3]["mixer"].update(scale=0.1),
                    lambda d: d.update(architecture="Other")):
        d = small_config()
        breaker(d)
        with pytest.raises(ValueError):
            LukupelConfig.from_dict(d)
    plain = {"vocab": 4, "width": 8, "norm": {"eps": 1e-6}, "layers": []}
    c = LukupelConfig.from_dict(plain)
    assert (c.embedding_scale, c.residual_mult, c.logit_softcap) == (1.0, 1.0, 0.0)


def test_argument_blocks_match_the_header(tmp_path):
    from lit_llama_b200 import _seqlib as S

    prog = tmp_path / "layout.c"
    prog.write_text('#include <stdio.h>\n#include <stddef.h>\n#include "b2l_seq.h"\nint main(void){printf("%zu %zu %zu %zu %zu %zu %zu %zu %zu %zu %zu\\n", '
                    "sizeof(b2l_seq_mlstm_args), offsetof(b2l_seq_mlstm_args, b_i), offsetof(b2l_seq_mlstm_args, eps), offsetof(b2l_seq_mlstm_args, meta), "
                    "offsetof(b2l_seq_mlstm_args, nq), offsetof(b2l_seq_mlstm_args, act_dtype), sizeof(b2l_seq_scan_args), offsetof(b2l_seq_scan_args, ones), "
                    "offsetof(b2l_seq_scan_args, out_ones), sizeof(b2l_seq_qkv_prep_args), offsetof(b2l_seq_qkv_prep_args, unit_rms));return 0;}\n")
    exe = tmp_path / "layout"
    subprocess.run(["gcc", "-I", os.path.join(ROOT, "include"), str(prog), "-o", str(exe)], check=True)
    out = [int(v) for v in subprocess.run([str(exe)], check=True, capture_output=True, text=True).stdout.split()]
    A, B, Q = S.MlstmArgs, S.ScanArgs, S.QkvPrepArgs
    assert out == [C.sizeof(A), A.b_i.offset, A.eps.offset, A.meta.offset, A.nq.offset, A.act_dtype.offset, C.sizeof(B), B.ones.offset, B.out_ones.offset, C.sizeof(Q),
                   Q.unit_rms.offset]
    names = {k for k in S.EXPORTS if "mlstm" in k}
    assert names == {"b2l_seq_mlstm_step", "b2l_seq_mlstm_gates", "b2l_seq_mlstm_readout"}


def test_rotation_frequencies_match_the_package():
    from lit_llama_b200.mixers import rope_frequencies

    for dims, base, factor in ((8, 100.0, None), (32, 3e5, 6.0), (2, 1e4, 1.0)):
        rot = {"dims": dims, "base": base}
        if factor:
            rot["scaling"] = {"factor": factor}
        g, m = rope_frequencies(dims, base, rot.get("scaling"))
        assert m == 1.0 and torch.allclose(torch.tensor(O.frequencies(rot), dtype=torch.float32), g, rtol=1e-6)
        assert float(g[0]) == pytest.approx(1.0 / (factor or 1.0))


def test_shared_mixers_keep_their_own_names():
    from lit_llama_b200.mixers import share_weights

    class One:
        name, w = "a", torch.ones(3)

    class Several(One):
        branches = [One(), One()]

    twin = share_weights(One(), "b")
    assert twin.name == "b" and twin.w is One.w and One().name == "a"
    with pytest.raises(ValueError):
        share_weights(Several(), "b")


def test_oracle_invariants():
    g = torch.Generator().manual_seed(0)
    # rotations keep the length, so the norm after them may be taken before; the norm leaves a root mean square of one
    v = torch.randn(8, generator=g, dtype=torch.float64)
    r = O.rotate(v, 7, O.frequencies({"dims": 6, "base": 50.0, "scaling": {"factor": 3.0}}))
    assert float(r.norm()) == pytest.approx(float(v.norm())) and torch.equal(r[6:], v[6:]) and not torch.allclose(r, v)
    assert float((O.unit_rms(r, 0.0) ** 2).mean()) == pytest.approx(1.0)
    # chunks are counted from position 0
    assert [O.visible_from(p, 5) for p in (0, 4, 5, 9, 10, 14)] == [0, 0, 5, 5, 10, 10] and O.visible_from(77, None) == 0
    # the running maximum is a matter of range alone: an unstabilised recurrence gives the same read-outs
    T, K, V = 40, 4, 3
    q, k, x = (torch.randn(T, n, generator=g, dtype=torch.float64) for n in (K, K, V))
    li, lf = torch.randn(T, generator=g, dtype=torch.float64), -torch.rand(T, generator=g, dtype=torch.float64)
    S, n, m = torch.zeros(K, V, dtype=torch.float64), torch.zeros(K, dtype=torch.float64), 0.0
    got = O.matrix_memory(q, k, x, li, lf)
    for t in range(T):
        S = math.exp(float(lf[t])) * S + math.exp(float(li[t])) * torch.outer(k[t], x[t])
        n = math.exp(float(lf[t])) * n + math.exp(float(li[t])) * k[t]
        m = max(m + float(lf[t]), float(li[t]))
        want = S.T @ q[t] / (max(abs(float(n @ q[t])), 1.0) + 1e-6 * math.exp(m))
        assert torch.allclose(got[t], want, rtol=1e-9)
    # a closed forget gate leaves the current token alone: its value, up to the sign of q . k
    lf[:] = -60.0
    li[:] = 5.0
    got = O.matrix_memory(q, k, x, li, lf)
    dots = (q * k).sum(-1)
    big = dots.abs() > 0.1
    assert torch.allclose(got[big], torch.sign(dots[big])[:, None] * x[big], rtol=1e-4)
    # the square of relu
    W = {"up": torch.eye(3), "down": torch.eye(3)}
    assert O.dense_ff(torch.tensor([[-2.0, 0.0, 3.0]], dtype=torch.float64), W, "").tolist() == [[0.0, 0.0, 9.0]]


def test_oracle_whole_model_is_causal_and_runs_shared_layers_again():
    from lit_llama_b200.lukupel import random_weights

    cfg = small_config()
    W = random_weights(cfg, "cpu", dtype=torch.float32, seed=2)
    assert not any(k.startswith(("l2.", "l3.", "l4.")) for k in W)
    toks = [3, 1, 4, 1, 5, 9, 2, 6, 5, 3, 5, 8]
    cap = []
    out = O.model(toks, cfg, W, capture=cap)
    assert out.shape == (12, 30) and len(cap) == 5 and bool(torch.isfinite(out).all()) and float(out.abs().max()) < 9.0
    again = O.model(toks[:7] + [0] + toks[8:], cfg, W)
    assert torch.allclose(again[:7], out[:7]) and not torch.allclose(again[7:], out[7:])
    once = dict(cfg, layers=cfg["layers"][:2])
    assert not torch.allclose(O.model(toks, once, W), out)
