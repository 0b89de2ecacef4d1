"""CPU: the Malulorn configuration reader and registry entry, the argument blocks of its kernels against a C compiler, and
the plain restatement's own invariants (tests/malulorn_oracle.py)."""
import copy
import ctypes as C
import math
import os
import subprocess

import pytest
import torch

import malulorn_oracle as O

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def small_config():
    att = {"heads": 4, "kv_heads": 2, "dim": 6, "vdim": 5, "scale": 0.4, "q_temp": {"coef": 0.2, "every": 3}}
    lat = {"heads": 2, "dim": 5, "rot_dim": 4, "vdim": 3, "kv_rank": 7, "scale": 0.3, "rot": {"base": 50.0, "dims": 4}}
    moe = {"kind": "moe", "expert": {"ff": 6}, "router": {"experts": 5, "top": 2}, "shared": {"ff": 9}}
    return {"architecture": "Malulorn", "vocab": 30, "width": 16, "norm": {"eps": 1e-5}, "loop": {"start": 1, "stop": 3, "times": 2},
            "layers": [{"type": "attention", "mixer": att, "mlp": moe}, {"type": "latent_attention", "mixer": lat, "mlp": None},
                       {"type": "attention", "mixer": att, "mlp": moe}, {"type": "latent_attention", "mixer": lat, "mlp": moe}]}


def test_config_reader_and_registry():
    from lit_llama_b200 import MalulornConfig, registry

    assert "Malulorn" in registry.architectures()
    c = MalulornConfig.from_dict(small_config())
    assert (c.vocab, c.width, c.eps, len(c.layers), c.loop) == (30, 16, 1e-5, 4, {"start": 1, "stop": 3, "times": 2})
    assert c.runs() == [(0, 0, False), (1, 0, True), (2, 0, False), (1, 1, True), (2, 1, False), (3, 0, False)]
    assert MalulornConfig.from_dict(c.to_dict()) == c
    for breaker in (lambda d: d["layers"][0].update(type="convolution"), lambda d: d["layers"][0]["mlp"].update(kind="dense"),
                    lambda d: d["loop"].update(stop=5), lambda d: d["loop"].update(start=3), lambda d: d["loop"].update(times=0),
                    lambda d: d["layers"][1]["mixer"]["rot"].update(dims=2), lambda d: d.update(architecture="Other")):
        d = copy.deepcopy(small_config())
        breaker(d)
        with pytest.raises(ValueError):
            MalulornConfig.from_dict(d)
    d = small_config()
    d.pop("loop")
    c = MalulornConfig.from_dict(d)
    assert c.loop is None and c.runs() == [(i, 0, False) for i in range(4)]
    d["loop"] = {"start": 0, "stop": 4, "times": 1}
    assert MalulornConfig.from_dict(d).runs() == [(0, 0, True), (1, 0, False), (2, 0, False), (3, 0, False)]


def test_argument_blocks_match_the_header(tmp_path):
    from lit_llama_b200 import _seqlib as S

    fields = {"b2l_seq_latent_operands_args": (S.LatentOperandsArgs, ("w_kv", "rot_mult", "cache", "q_full", "q_lat", "act_dtype")),
              "b2l_seq_residual_args": (S.ResidualArgs, ("y2", "split", "h", "eps", "D", "act_dtype")),
              "b2l_seq_latent_attn_args": (S.LatentAttnArgs, ("window", "gate", "ldg", "partial")),
              "b2l_seq_qkv_prep_args": (S.QkvPrepArgs, ("unit_rms", "temp_coef", "temp_every"))}
    items, want = [], []
    for name, (cls, names) in fields.items():
        items.append(f"sizeof({name})")
        want.append(C.sizeof(cls))
        for f in names:
            items.append(f"offsetof({name}, {f})")
            want.append(getattr(cls, f).offset)
    prog = tmp_path / "layout.c"
    prog.write_text('#include <stdio.h>\n#include <stddef.h>\n#include "b2l_seq.h"\nint main(void){' +
                    "".join(f'printf("%zu\\n", {i});' for i in items) + "return 0;}\n")
    exe = tmp_path / "layout"
    subprocess.run(["gcc", "-I", os.path.join(ROOT, "include"), str(prog), "-o", str(exe)], check=True)
    assert [int(v) for v in subprocess.run([str(exe)], check=True, capture_output=True, text=True).stdout.split()] == want


def small_weights(cfg, seed=1):
    from lit_llama_b200.malulorn import random_weights

    return random_weights(cfg, "cpu", dtype=torch.float32, seed=seed)


def test_oracle_is_causal_and_reads_every_position():
    cfg = small_config()
    W = small_weights(cfg)
    toks = torch.randint(0, 30, (14,), generator=torch.Generator().manual_seed(3)).tolist()
    base = O.model(toks, cfg, W)
    for at in (0, 5, 13):
        other = list(toks)
        other[at] = (other[at] + 1) % 30
        got = O.model(other, cfg, W)
        assert torch.equal(got[:at], base[:at])
        assert all(float((got[t] - base[t]).abs().max()) > 1e-9 for t in range(at, 14))
    assert torch.allclose(O.model(toks[:9], cfg, W), base[:9], atol=1e-12)


def test_oracle_loop_is_the_layers_written_out():
    """One pass with W_in = [1 | 0] and no step vector is the model without a loop; each pass sees the embedding again."""
    cfg = small_config()
    W = small_weights(cfg)
    toks = [3, 8, 1, 29, 4]
    plain = {k: v for k, v in cfg.items() if k != "loop"}
    cfg["loop"] = {"start": 1, "stop": 3, "times": 1}
    W["loop.in"] = torch.cat([torch.eye(16), torch.zeros(16, 16)], dim=1)
    W["loop.step"] = torch.zeros(1, 16)
    assert torch.allclose(O.model(toks, cfg, W), O.model(toks, plain, W), atol=1e-12)
    W["loop.in"] = torch.cat([torch.zeros(16, 16), torch.eye(16)], dim=1)          # a pass starts from the embedding output alone
    cap = []
    O.model(toks, cfg, W, capture=cap)
    skip = dict(plain, layers=plain["layers"][1:])
    W2 = {k.replace("l1.", "l0.", 1) if k.startswith("l1.") else k.replace("l2.", "l1.", 1) if k.startswith("l2.") else
          k.replace("l3.", "l2.", 1) if k.startswith("l3.") else k: v for k, v in W.items() if not k.startswith("l0.")}
    cap2 = []
    O.model(toks, skip, W2, capture=cap2)
    assert torch.allclose(cap[1], cap2[0], atol=1e-12) and torch.allclose(cap[3], cap2[2], atol=1e-12)


def test_oracle_softmax_and_temperature():
    s = torch.tensor([[0.0, 0.0, 5.0], [-2.0, 700.0, 9.0]], dtype=torch.float64)
    w = O.softmax_plus_one(s, torch.tensor([[False, False, True], [False, False, False]]))
    assert torch.allclose(w[0], torch.tensor([1 / 3, 1 / 3, 0.0], dtype=torch.float64)) and float(w[1, 1]) == pytest.approx(1.0)
    assert O.query_temperature(0, 0.5, 4) == 1.0 and O.query_temperature(2, 0.5, 4) == 1.0
    assert O.query_temperature(3, 0.5, 4) == pytest.approx(1 + 0.5 * math.log(2)) == O.query_temperature(6, 0.5, 4)
    assert O.query_temperature(7, 0.5, 4) == pytest.approx(1 + 0.5 * math.log(3))
    assert O.query_temperature(0, 0.5, 1) == pytest.approx(1 + 0.5 * math.log(2))


def test_host_side_refusals():
    from lit_llama_b200 import mixers as M

    W = {"m." + k: torch.zeros(*s) for k, s in (("q", (8, 4)), ("k", (8, 4)), ("v", (8, 4)), ("g", (2, 4)), ("o", (4, 8)))}
    kw = dict(heads=2, kv_heads=2, dim=4, vdim=4, scale=1.0, eps=1e-6, max_positions=8, norm_over="head")
    att = M.LocalAttention("a", W, "m.", gate="head", sink=True, q_temp={"coef": 0.1, "every": 16.0}, **kw)
    assert (att.temp_every, att.sink, att.gate_per_channel, att.ring, att.window) == (16, 1, 0, 8, 0)
    for bad in ({"coef": 0.1, "every": 0}, {"coef": 0.1, "every": 2.5}):
        with pytest.raises(ValueError):
            M.LocalAttention("a", W, "m.", gate="head", sink=True, q_temp=bad, **kw)
    with pytest.raises(ValueError):
        M.LocalAttention("a", W, "m.", gate="row", **kw)
    with pytest.raises(AssertionError):
        M.LocalAttention("a", W, "m.", gate="channel", **kw)                    # the gate has one row per head
    with pytest.raises(ValueError):
        M.LoopInjection(torch.zeros(4, 7), torch.zeros(2, 4))
    with pytest.raises(ValueError):
        M.LoopInjection(torch.zeros(4, 8), torch.zeros(2, 5))
    E = {"router": torch.zeros(2, 4), "router.b": torch.zeros(2)}
    for e in ("e0", "e1", "shared"):
        E.update({f"{e}.gate": torch.zeros(3, 4), f"{e}.up": torch.zeros(3, 4), f"{e}.down": torch.zeros(4, 3)})
    kw = dict(experts=2, identity=0, top=1, groups=1, keep=1, ff=3, score="chosen_softmax")
    assert M.MoEFeedForward(E, "", shared_ff=3, **kw).shared.ff == 3 and M.MoEFeedForward(E, "", **kw).shared is None
    with pytest.raises(ValueError):
        M.MoEFeedForward(E, "", renormalize=False, **kw)
    with pytest.raises(AssertionError):
        M.MoEFeedForward(E, "", shared_ff=4, **kw)
