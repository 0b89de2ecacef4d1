"""GPU: the Malulorn model family and its mechanisms against the plain restatement in tests/malulorn_oracle.py (float64), on
small random models of several shapes: each mechanism alone, whole prompts against token-by-token decoding and portions of
many sizes, interleaved requests, reused cache slots, keys that stand out far back, at chunk and tile borders and on both
sides of the causal edge, long decoding, greedy generation through the engine's scheduler, trace replay."""
import ctypes as C
import io
import json
import math
import sys

import pytest
import torch

import malulorn_oracle as O

pytestmark = pytest.mark.gpu

DEV = "cuda"
TOL = 2e-5


def _pkg():
    import lit_llama_b200 as P
    from lit_llama_b200 import _seqlib as S
    from lit_llama_b200 import mixers as M
    return P, S, M


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).norm() / (want.norm() + 1e-30))


# ----------------------------------------------------------------------------- configurations (none is a served model's)
def moe(experts, top, ff, shared=0):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return dict(m, shared={"ff": shared}) if shared else m


def attn(heads, kv, dim, vdim, scale, coef, every, mlp):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
                                           "q_temp": {"coef": coef, "every": every}}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, rank, scale, base, mlp):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
                                                  "rot": {"base": base, "dims": rot_dim}}, "mlp": mlp}


def config(vocab, width, layers, loop, eps=1e-6):
    d = {"architecture": "Malulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    return dict(d, loop=dict(zip(("start", "stop", "times"), loop))) if loop else d


def cfg_a():
    """Odd sizes everywhere, three query heads per kv head, three passes over a stretch in the middle, looped layers without
    a feed-forward, one without a shared expert."""
    return config(131, 72, [attn(3, 1, 10, 14, 0.6, 0.7, 5, moe(6, 2, 20, 28)), latent(3, 11, 6, 13, 35, 0.4, 900.0, None),
                            attn(4, 2, 7, 9, 0.5, 0.2, 16, moe(5, 3, 18)), latent(2, 8, 4, 10, 12, 0.5, 50.0, moe(4, 1, 26, 10)),
                            attn(2, 2, 12, 6, 0.4, -0.1, 9, None)], (1, 4, 3), eps=1e-5)


def cfg_b():
    """Shapes that take the tiled attention kernel, the expanded latent form and the grouped expert products: 16-byte rows,
    portions of hundreds of tokens; the whole stack runs twice."""
    f = moe(8, 3, 48, 64)
    return config(200, 128, [attn(8, 2, 32, 48, 0.2, 0.25, 64, f), latent(4, 32, 16, 24, 72, 0.15, 3e5, f), attn(4, 4, 24, 64, 0.25, 0.1, 100, f)], (0, 3, 2))


def cfg_c():
    """What a served model may happen to make equal or one: one head, kv heads = heads, key size = value size, a step of one
    position, no temperature, one expert, every expert chosen, one pass over one layer, the last one."""
    return config(90, 64, [attn(1, 1, 16, 16, 0.3, 0.3, 1, moe(3, 3, 16, 16)), latent(1, 16, 16, 16, 16, 0.25, 1e4, moe(1, 1, 24, 8)),
                           attn(4, 4, 8, 8, 0.9, 0.0, 7, moe(5, 1, 32, 40)), latent(5, 8, 2, 4, 150, 0.3, 10.0, moe(4, 2, 64, 32))], (3, 4, 1))


def cfg_d():
    """No loop; a latent above 256 entries; many heads (a portion of a few tokens does not count as few queries)."""
    return config(60, 56, [latent(6, 6, 8, 5, 264, 0.4, 400.0, moe(7, 4, 12, 30)), attn(80, 4, 6, 4, 0.5, 0.4, 3, None)], None)


CONFIGS = {"a": cfg_a, "b": cfg_b, "c": cfg_c, "d": cfg_d}


def random_weights(cfg, seed=1):
    """bf16-representable float32 tensors on the CPU under the family's tensor names."""
    from lit_llama_b200.malulorn import random_weights as rw

    return {k: v.bfloat16().float() for k, v in rw(cfg, "cpu", dtype=torch.float32, seed=seed).items()}


def build(cfg, dtype, seed=1, n_slots=3, max_positions=512):
    P, S, M = _pkg()
    W = random_weights(cfg, seed)
    model = P.Malulorn(P.MalulornConfig.from_dict(cfg), {k: v.to(DEV, dtype) for k, v in W.items()}, max_positions=max_positions)
    return model, P.Engine(model, n_slots=n_slots), W


def tokens_of(cfg, n, seed=5):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_whole(engine, toks, rid="w"):
    return engine.step([{"id": rid, "tokens": toks, "want": list(range(len(toks)))}], [rid])[0]


def run_pieces(engine, toks, sizes, rid="p"):
    """The prompt in portions of the given sizes (cycled), every position's logits."""
    outs, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[i % len(sizes)], len(toks) - at)
        outs.append(engine.step([{"id": rid, "tokens": toks[at:at + n], "want": list(range(n))}], [rid] if at + n == len(toks) else [])[0])
        at, i = at + n, i + 1
    return torch.cat(outs)


# ----------------------------------------------------------------------------- whole models against the oracle
@pytest.mark.parametrize("name", ["a", "b", "c", "d"])
def test_model_matches_the_oracle_layer_by_layer_f32(name):
    cfg = CONFIGS[name]()
    model, engine, W = build(cfg, torch.float32)
    toks = tokens_of(cfg, 200 if name == "b" else 75)      # long enough for the expanded latent form
    cap = []
    want = O.model(toks, cfg, W, capture=cap)
    model.capture_layers = []
    got = run_whole(engine, toks)
    assert len(model.capture_layers) == len(cap) == len(model.runs)
    for i, (g, w) in enumerate(zip(model.capture_layers, cap)):
        assert rel(g, w) < TOL, (name, "layer run", i, rel(g, w))
    assert rel(got, want) < TOL


@pytest.mark.parametrize("name", ["a", "b", "c", "d"])
def test_model_bf16_is_close_to_the_oracle(name):
    cfg = CONFIGS[name]()
    model, engine, W = build(cfg, torch.bfloat16)
    toks = tokens_of(cfg, 80)
    got = run_whole(engine, toks)
    assert rel(got, O.model(toks, cfg, W)) < 0.1, rel(got, O.model(toks, cfg, W))      # a routing flip on a close call moves one token a lot
    assert rel(run_pieces(engine, toks, [7, 1, 2, 13]), got) < 0.05


@pytest.mark.parametrize("name", ["a", "b", "c", "d"])
def test_portions_and_single_tokens_equal_the_whole_prompt(name):
    cfg = CONFIGS[name]()
    n = 400 if name == "b" else 80
    model, engine, W = build(cfg, torch.float32)
    toks = tokens_of(cfg, n)
    whole = run_whole(engine, toks)
    if name != "b":
        assert rel(whole, O.model(toks, cfg, W)) < TOL
    for sizes in ([1], [2], [3, 2, 17, 1, 5, 4], [33, 64], [n - 9, 1, 1, 2]):
        if name == "b" and sizes == [1]:
            sizes = [n - 140, 1]            # a long first portion, then 140 tokens one by one: chunks of 64 keys are passed while decoding
        got = run_pieces(engine, toks, sizes)
        assert rel(got, whole) < TOL, (name, sizes, rel(got, whole))


def test_long_prompt_matches_the_oracle():
    cfg = cfg_b()
    model, engine, W = build(cfg, torch.float32)
    toks = tokens_of(cfg, 310, seed=9)
    want = O.model(toks, cfg, W)
    assert rel(run_whole(engine, toks), want) < TOL
    assert rel(run_pieces(engine, toks, [261, 1, 2, 1, 1]), want) < TOL


def test_interleaved_requests_and_reused_slots():
    cfg = cfg_a()
    model, engine, W = build(cfg, torch.float32, n_slots=2)
    prompts = [tokens_of(cfg, n, seed=s) for n, s in ((23, 1), (5, 2), (41, 3), (1, 4), (12, 5))]
    alone = [run_whole(engine, p, rid=("alone", i)) for i, p in enumerate(prompts)]
    for i, p in enumerate(prompts):
        assert rel(alone[i], O.model(p, cfg, W)) < TOL
    # two at a time in the two slots, unequal portions in turns; finished requests hand their slot to the next one
    got = {i: [] for i in range(len(prompts))}
    at = {i: 0 for i in range(len(prompts))}
    waiting, live = list(range(len(prompts))), []
    step = 0
    while waiting or live:
        while waiting and len(live) < 2:
            live.append(waiting.pop(0))
        for i in list(live):
            n = min([3, 1, 7, 2][step % 4], len(prompts[i]) - at[i])
            step += 1
            end = at[i] + n == len(prompts[i])
            got[i].append(engine.step([{"id": i, "tokens": prompts[i][at[i]:at[i] + n], "want": list(range(n))}], [i] if end else [])[0])
            at[i] += n
            if end:
                live.remove(i)
    assert engine.pool.reused >= 3
    for i in range(len(prompts)):
        assert rel(torch.cat(got[i]), alone[i]) < TOL, i
    # one step with several entries of unequal length against each alone
    outs = engine.step([{"id": ("m", i), "tokens": p, "want": list(range(len(p)))} for i, p in enumerate(prompts[:2])], [("m", 0), ("m", 1)])
    for i in range(2):
        assert rel(outs[i], alone[i]) < TOL


def test_long_decoding_through_the_captured_step():
    cfg = cfg_a()
    model, engine, W = build(cfg, torch.float32)
    toks = tokens_of(cfg, 220)
    want = O.model(toks, cfg, W)
    first = engine.step([{"id": "d", "tokens": toks[:20], "want": [19]}])[0]
    outs = [first] + [engine.step([{"id": "d", "tokens": [t], "want": [0]}])[0] for t in toks[20:]]
    assert engine._graph is not None
    assert rel(torch.cat(outs), want[19:]) < TOL
    # the same captured step serves another request in another slot from its first token on
    outs2 = [engine.step([{"id": "e", "tokens": [t], "want": [0]}])[0] for t in toks[:40]]
    assert rel(torch.cat(outs2), want[:40]) < TOL


@pytest.mark.parametrize("name", ["a", "c"])
def test_first_tokens_of_a_sequence(name):
    """One-token and two-token sequences in a slot that a longer request used before."""
    cfg = CONFIGS[name]()
    model, engine, W = build(cfg, torch.float32, n_slots=1)
    run_whole(engine, tokens_of(cfg, 30, seed=2))
    for toks in ([7], [7, 7], [cfg["vocab"] - 1, 0], tokens_of(cfg, 3), tokens_of(cfg, 8)):
        want = O.model(toks, cfg, W)
        assert rel(run_whole(engine, toks), want) < TOL
        assert rel(run_pieces(engine, toks, [1]), want) < TOL
        assert rel(run_pieces(engine, toks, [2, 1]), want) < TOL
    assert engine.pool.reused >= 10


def test_every_pass_has_its_own_cache_over_the_same_weights():
    cfg = cfg_a()
    model, engine, W = build(cfg, torch.float32)
    for i, layer in enumerate(model.layers):
        assert len(layer.mixers) == (3 if 1 <= i < 4 else 1)
        assert all(m.w_in is layer.mixers[0].w_in for m in layer.mixers)
        names = [n for m in layer.mixers for n in m.state_specs()]
        assert len(names) == len(set(names))
    assert len(model.state_specs()) == 2 * 3 + 2 * 1 * 3 + 2 + 2      # looped: two latent caches and one key / value pair, three passes each
    toks = tokens_of(cfg, 12)
    want = O.model(toks, cfg, W)
    engine.step([{"id": "x", "tokens": toks[:11], "want": []}])
    good = engine.step([{"id": "x", "tokens": toks[11:], "want": [0]}], ["x"])[0]
    assert rel(good, want[11:]) < TOL
    engine.step([{"id": "y", "tokens": toks[:11], "want": []}])          # another pass's keys in place of its own: the result must notice
    engine.pool.tensors["l1.pass2.kv"].copy_(engine.pool.tensors["l1.pass1.kv"])
    bad = engine.step([{"id": "y", "tokens": toks[11:], "want": [0]}], ["y"])[0]
    assert rel(bad, want[11:]) > 1e-3


def test_position_limit():
    P, S, M = _pkg()
    cfg = cfg_c()
    model, engine, W = build(cfg, torch.float32, max_positions=16)
    toks = tokens_of(cfg, 20)
    want = O.model(toks[:16], cfg, W)
    got = [engine.step([{"id": "x", "tokens": toks[:14], "want": list(range(14))}])[0]] + [engine.step([{"id": "x", "tokens": [t], "want": [0]}])[0] for t in toks[14:16]]
    assert rel(torch.cat(got), want) < TOL                                # the last positions that fit
    with pytest.raises(P.state.PoolFull):
        engine.step([{"id": "x", "tokens": toks[16:17], "want": [0]}])


def test_greedy_generation_through_the_scheduler():
    cfg = cfg_a()
    model, engine, W = build(cfg, torch.float32, n_slots=2)
    engine.prefill_chunk = 6
    prompts = [tokens_of(cfg, n, seed=s) for n, s in ((9, 11), (17, 12), (3, 13))]
    for i, p in enumerate(prompts):
        engine.add_request(i, p, 12)
    out = engine.run()
    checked = 0
    for i, p in enumerate(prompts):
        seq = list(p)
        for _ in range(12):
            lg = O.model(seq, cfg, W)[-1]
            top2 = lg.topk(2).values
            if float(top2[0] - top2[1]) < 1e-3:          # a close call decides nothing about the framework
                break
            seq.append(int(lg.argmax()))
        n = len(seq) - len(p)
        checked += n
        assert out[i][:n] == seq[len(p):], (i, out[i], seq[len(p):])
    assert checked > 20
    assert engine.generate(prompts[0], 4)[:len(prompts[0])] == prompts[0]


def test_sampled_generation_runs_and_respects_eos():
    cfg = cfg_c()
    model, engine, W = build(cfg, torch.bfloat16)
    torch.manual_seed(0)
    prompt = tokens_of(cfg, 9)
    out = engine.generate(prompt, 12, temperature=0.8, top_k=5)
    assert len(out) == 21 and all(0 <= t < cfg["vocab"] for t in out)
    first = engine.generate(prompt, 4)[9]
    assert engine.generate(prompt, 12, eos_id=first) == prompt + [first]


def save(cfg, W, path):
    from lit_llama_b200.checkpoint_io import write_safetensors

    (path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(path / "model.safetensors"), {k: v.bfloat16() for k, v in W.items()})


def test_registry_loads_a_saved_model(tmp_path):
    P, S, M = _pkg()
    cfg = cfg_b()
    W = random_weights(cfg, seed=3)
    save(cfg, W, tmp_path)
    toks = tokens_of(cfg, 12)
    want = O.model(toks, cfg, W)
    for dtype, tol in ((torch.float32, TOL), (torch.bfloat16, 0.1)):
        model = P.load_model(str(tmp_path), dtype=dtype, device=DEV, max_positions=64)
        assert type(model).__name__ == "Malulorn" and model.max_positions == 64
        assert rel(run_whole(P.Engine(model, n_slots=1), toks), want) < tol


def test_trace_replay(tmp_path, monkeypatch, capsys):
    """Given tokens through the trace program: files for the steps that want logits, a line for every step."""
    import numpy as np
    from lit_llama_b200 import trace

    cfg = cfg_a()
    W = random_weights(cfg, seed=4)
    save(cfg, W, tmp_path)
    a, b = tokens_of(cfg, 21, seed=1), tokens_of(cfg, 6, seed=2)
    steps = [([("a", a[:9], [0, 8])], []), ([("a", a[9:11], [])], []), ([("a", a[11:20], [4])], []), ([("a", a[20:], [0])], ["a"]), ([("b", b, [5, 1])], ["b"])]
    lines = [json.dumps({"step": i, "entries": [{"id": r, "tokens": t, "want": w} for r, t, w in entries], "end": end}) for i, (entries, end) in enumerate(steps)]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(lines) + "\n"))
    assert trace.main(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path / "out"), "--max-tokens", "24"]) == 0
    assert [l for l in capsys.readouterr().out.split("\n") if l.startswith("done ")] == [f"done {i}" for i in range(5)]
    wa, wb = O.model(a, cfg, W), O.model(b, cfg, W)
    want = {0: wa[[0, 8]], 2: wa[[15]], 3: wa[[20]], 4: wb[[5, 1]]}
    assert sorted(int(p.stem) for p in (tmp_path / "out").glob("*.f32")) == sorted(want)
    for i, w in want.items():
        got = torch.from_numpy(np.fromfile(str(tmp_path / "out" / f"{i}.f32"), dtype="<f4")).view(w.shape)
        assert rel(got, w) < TOL, i


# ----------------------------------------------------------------------------- mechanisms alone
def _ctx(M, P, mixer, T, pos0, dtype, slot=0, pool=None, hint=True):
    pool = pool or P.SequenceStatePool(mixer.state_specs(), 2, torch.device(DEV))
    meta = torch.tensor([slot, pos0], dtype=torch.int32, device=DEV)
    return M.StepContext(T, meta, pool.tensors, dtype, pos_hint=pos0 if hint else None, slot_hint=slot if hint else None), pool, meta


def _pieces(M, P, mixer, h, sizes, dtype=torch.float32, slot=1, hint=True):
    """A mixer over portions of h, one after the other in one slot; single tokens without host hints, as in the captured step."""
    pool, outs, at = None, [], 0
    for n in sizes:
        ctx, pool, _ = _ctx(M, P, mixer, n, at, dtype, slot=slot, pool=pool, hint=hint and n > 1)
        outs.append(mixer.forward(h[at:at + n].to(DEV, dtype), ctx))
        at += n
    assert at == h.shape[0]
    return torch.cat(outs)


def _attention_layer(M, m, max_positions=400):
    """The attention mixer with projections that copy columns of h: h = [q | k | v | g], W_o the identity."""
    H, G, K, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rows = [H * K, G * K, G * V, H]
    D, at, W = sum(rows), 0, {}
    for n, r in zip("qkvg", rows):
        W["m." + n] = torch.eye(D)[at:at + r].contiguous()
        at += r
    W["m.o"] = torch.eye(H * V)
    mixer = M.LocalAttention("x", {k: v.to(DEV) for k, v in W.items()}, "m.", heads=H, kv_heads=G, dim=K, vdim=V, scale=m["scale"], eps=1e-6,
                             max_positions=max_positions, norm_over="head", gate="head", sink=True, q_temp=m["q_temp"])
    return mixer, {k: v.double() for k, v in W.items()}, D


SHAPES = [(3, 1, 10, 14, 0.5, 0.7, 5), (8, 2, 32, 48, 0.2, 0.25, 64), (1, 1, 16, 16, 0.3, 0.3, 1), (4, 4, 24, 128, 0.25, -0.1, 100), (6, 2, 13, 7, 0.4, 0.0, 3),
          (2, 1, 64, 200, 0.1, 0.5, 33)]


@pytest.mark.parametrize("shape", SHAPES)
def test_attention_alone(shape):
    P, S, M = _pkg()
    m = dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), shape[:5]), q_temp={"coef": shape[5], "every": shape[6]})
    mixer, W, D = _attention_layer(M, m)
    T = 330
    h = torch.randn(T, D, generator=torch.Generator().manual_seed(3)).bfloat16().float()
    want = O.attention(h.double(), W, "m.", m)
    assert rel(_pieces(M, P, mixer, h, [T]), want) < TOL                       # one portion: query tiles where the shape allows
    assert rel(_pieces(M, P, mixer, h, [250] + [1] * 80), want) < TOL          # chunks of keys, merged; the ring written by single tokens
    assert rel(_pieces(M, P, mixer, h, [2, 3, 64, 1, 17, 2, 128, 13, 100]), want) < TOL


@pytest.mark.parametrize("shape", SHAPES)
def test_attention_finds_a_standout_key_at_every_border(shape):
    """One key along a direction of its own, read by every query after it: at the first position, on both sides of tile (32,
    64) and chunk (64) borders, far back; a query before it must not see it, the query on it must."""
    P, S, M = _pkg()
    m = dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), shape[:5]), q_temp={"coef": max(shape[5], 0.0), "every": shape[6]})
    H, G, K, V = shape[:4]
    mixer, W, D = _attention_layer(M, m)
    T = 200
    g = torch.Generator().manual_seed(4)
    for target in (0, 1, 31, 32, 63, 64, 127, 128, 150, T - 1):
        h = 0.1 * torch.randn(T, D, generator=g)
        u = torch.randn(K, generator=g)
        u = u / u.norm()
        q, k, v = h[:, :H * K].view(T, H, K), h[:, H * K:H * K + G * K].view(T, G, K), h[:, H * K + G * K:H * K + G * (K + V)].view(T, G, V)
        q += 6.0 * u / math.sqrt(m["scale"])
        k -= (k @ u)[..., None] * u                                      # no other key has a component along u
        k[target] = 6.0 * u / math.sqrt(m["scale"])                      # score 36 against at most a few
        v[target] = 5.0
        want = O.attention(h.double(), W, "m.", m)
        gate = torch.sigmoid(h[:, -H:].double())
        share = (want.view(T, H, V).mean(-1) / gate) / 5.0
        assert float(share[target:].min()) > 0.95 and (target == 0 or float(share[:target].abs().max()) < 0.1)
        assert rel(_pieces(M, P, mixer, h, [T]), want) < TOL, target
        assert rel(_pieces(M, P, mixer, h, [120, 2] + [1] * 78), want) < TOL, target


def test_attention_denominator_takes_its_share():
    """All scores zero: weights 1 / (n + 1); scores far below zero: nothing comes out; far above: the one does not matter."""
    P, S, M = _pkg()
    m = {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 32, "scale": 1.0, "q_temp": {"coef": 0.0, "every": 4}}
    mixer, W, D = _attention_layer(M, m)
    T, nq, nk = 90, 64, 32
    h = torch.randn(T, D)
    for level in (0.0, -80.0, 80.0, -3.0):
        h[:, :nq] = level / 16.0
        h[:, nq:nq + nk] = 1.0
        v = h[:, nq + nk:nq + nk + 64].view(T, 2, 32).double()
        gate = torch.sigmoid(h[:, -4:].double())
        for sizes in ([T], [40] + [1] * 50):
            got = _pieces(M, P, mixer, h, sizes).view(T, 4, 32).double().cpu()
            for t in (0, 1, 31, 32, 63, 64, 89):
                n = t + 1
                w = 1.0 / (n + math.exp(-level))
                want = w * v[:t + 1].sum(0).repeat_interleave(2, 0) * gate[t][:, None]
                assert torch.allclose(got[t], want, rtol=1e-4, atol=1e-6), (level, sizes, t)


@pytest.mark.parametrize("coef,every", [(0.35, 96), (0.5, 1), (-0.2, 3), (0.1, 1000), (0.0, 7)])
def test_query_temperature_steps_at_its_positions(coef, every):
    P, S, M = _pkg()
    H, G, K, T = 3, 1, 10, 9
    proj = torch.randn(T, (H + 2 * G) * K)
    pd = proj.to(DEV)
    for pos0 in (0, every - 5 if every > 5 else 0, 10 * every - 4, 77 * every - 3, 100000):
        if pos0 < 0:
            continue
        q, k = torch.empty(T, H * K, device=DEV), torch.empty(T, G * K, device=DEV)
        meta = torch.tensor([0, pos0], dtype=torch.int32, device=DEV)
        a = S.QkvPrepArgs(proj=pd.data_ptr(), ld=(H + 2 * G) * K, q_off=0, k_off=H * K, v_off=(H + G) * K, eps=1e-6, rot_mult=1.0, meta=meta.data_ptr(),
                          q_out=q.data_ptr(), k_out=k.data_ptr(), T=T, heads=H, kv_heads=G, K=K, V=K, act_dtype=S.B2L_F32, temp_coef=coef, temp_every=every)
        S.check(S.lib().b2l_seq_qkv_prep(C.byref(a), torch.cuda.current_stream().cuda_stream), "prep")
        temp = torch.tensor([O.query_temperature(pos0 + t, coef, every) for t in range(T)], dtype=torch.float64)
        assert torch.allclose(q.double().cpu(), proj[:, :H * K].double() * temp[:, None], rtol=1e-6, atol=1e-7), (pos0,)
        assert torch.equal(k.cpu(), proj[:, H * K:(H + G) * K])


LATENTS = [(3, 20, 12, 28, 36), (1, 8, 2, 4, 70), (6, 16, 16, 16, 150), (2, 4, 6, 300, 260), (5, 33, 4, 9, 129), (4, 32, 16, 64, 512)]


def _latent_weights(m, D, seed=2):
    g = torch.Generator().manual_seed(seed)

    def lin(o, i, gain=1.0):
        return (gain * torch.randn(o, i, generator=g) / math.sqrt(i)).bfloat16().float()

    H, dn, dr, dv, rk = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    return {"m.q": lin(H * (dn + dr), D, 2.0), "m.dkv": lin(rk + dr, D), "m.dkv.norm": (1 + 0.2 * torch.randn(rk, generator=g)).bfloat16().float(),
            "m.uk": lin(H * dn, rk, 2.0), "m.uv": lin(H * dv, rk), "m.g": lin(H * dv, D, 2.0), "m.o": lin(D, H * dv)}


def _latent_layer(M, m, W, eps, dtype=torch.float32):
    return M.LatentAttention("x", {k: v.to(DEV, dtype) for k, v in W.items()}, "m.", heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"],
                             q_rank=None, kv_rank=m["kv_rank"], scale=m["scale"], eps=eps, rot=m["rot"], max_positions=256, gate=True)


@pytest.mark.parametrize("sizes", LATENTS)
def test_latent_attention_alone(sizes):
    P, S, M = _pkg()
    m = dict(zip(("heads", "dim", "rot_dim", "vdim", "kv_rank"), sizes), scale=0.2, rot={"base": 777.0, "dims": sizes[2]})
    D, T, eps = 48, 150, 1e-5
    W = _latent_weights(m, D)
    h = torch.randn(T, D, generator=torch.Generator().manual_seed(6)).bfloat16().float()
    Wd = {k: v.double() for k, v in W.items()}
    want = O.latent_attention(h.double(), Wd, "m.", m, eps)
    mixer = _latent_layer(M, m, W, eps)
    assert rel(_pieces(M, P, mixer, h, [T]), want) < TOL                       # keys and values expanded per head, gate on the stores
    assert rel(_pieces(M, P, mixer, h, [70] + [1] * 80), want) < TOL           # a few tokens: W_uk and W_uv inside the framework's kernels
    assert rel(_pieces(M, P, mixer, h, [5, 3, 2, 64, 4, 1, 50, 21]), want) < TOL
    mixer.expand_from = 10 ** 9
    assert rel(_pieces(M, P, mixer, h, [T]), want) < TOL                       # the same portion in the latent space
    b = _latent_layer(M, m, W, eps, torch.bfloat16)
    for pieces in ([T], [5] * 30, [1] * T):
        assert rel(_pieces(M, P, b, h, pieces, torch.bfloat16), want) < 0.03, pieces


@pytest.mark.parametrize("sizes", [LATENTS[0], LATENTS[2], LATENTS[4]])
def test_latent_attention_finds_a_standout_key_at_every_border(sizes):
    """Queries that point at one position's key (unrotated part): far back, on both sides of tile and split borders, on the
    query's own position, and not before it.  h = [q | c', k_r | g] with copying projections."""
    P, S, M = _pkg()
    H, dn, dr, dv, rk = sizes
    m = dict(zip(("heads", "dim", "rot_dim", "vdim", "kv_rank"), sizes), scale=1.0, rot={"base": 777.0, "dims": dr})
    nq, T = H * (dn + dr), 180
    D = nq + rk + dr + H * dv
    W = _latent_weights(m, D)
    eye = torch.eye(D)
    W["m.q"], W["m.dkv"], W["m.g"], W["m.o"] = eye[:nq].contiguous(), eye[nq:nq + rk + dr].contiguous(), eye[nq + rk + dr:].contiguous(), torch.eye(H * dv)
    mixer = _latent_layer(M, m, W, 1e-6)
    Wd = {k: v.double() for k, v in W.items()}
    g = torch.Generator().manual_seed(8)
    for target in (0, 1, 31, 32, 33, 63, 64, 95, 96, 133, T - 2, T - 1):
        h = 0.3 * torch.randn(T, D, generator=g)
        c = O.rms_unit(h[:, nq:nq + rk].double(), 1e-6) * Wd["m.dkv.norm"]
        keys = (c @ Wd["m.uk"].T).view(T, H, dn)
        others = torch.cat([keys[:target], keys[target + 1:]])
        q = h[:, :nq].view(T, H, dn + dr)
        for hd in range(H):                                              # away from the mean of the other keys, towards the target's
            d = keys[target, hd] - others[:, hd].mean(0)
            gap = float((keys[target, hd] @ d) - (others[:, hd] @ d).max())
            q[:, hd, :dn] = (d * (30.0 / max(gap, 1e-2))).float() if gap > 0.2 else 0.0
        want = O.latent_attention(h.double(), Wd, "m.", m, 1e-6)
        val = (c @ Wd["m.uv"].T).view(T, H, dv)
        hit = [(want.view(T, H, dv)[:, hd] / torch.sigmoid(h[:, nq + rk + dr:].double()).view(T, H, dv)[:, hd] - val[target, hd]).norm(dim=-1) / val[target, hd].norm()
               for hd in range(H) if float(q[0, hd, :dn].abs().max()) > 0]
        assert hit, "no head points at the target"
        for d in hit:
            assert float(d[target:].max()) < 1e-3 and (target == 0 or float(d[:target].min()) > 0.1)
        assert rel(_pieces(M, P, mixer, h, [T]), want) < 5e-5, target
        assert rel(_pieces(M, P, mixer, h, [100, 2, 7] + [1] * 71), want) < 5e-5, target


@pytest.mark.parametrize("E,top,ff,shared", [(6, 2, 24, 36), (4, 1, 16, 8), (5, 5, 10, 31), (40, 6, 32, 64), (1, 1, 8, 16), (7, 3, 26, 0)])
def test_router_and_experts(E, top, ff, shared):
    P, S, M = _pkg()
    D, T = 40, 60
    f = moe(E, top, ff, shared)
    g = torch.Generator().manual_seed(6)

    def lin(o, i):
        return (torch.randn(o, i, generator=g) / math.sqrt(i)).bfloat16().float()

    W = {"router": 2.0 * lin(E, D), "router.b": torch.randn(E, generator=g).bfloat16().float()}      # a bias that changes choices and weights
    for n, w in [(f"e{e}", ff) for e in range(E)] + ([("shared", shared)] if shared else []):
        W.update({n + ".gate": lin(w, D), n + ".up": lin(w, D), n + ".down": lin(D, w)})
    h = torch.randn(T, D, generator=g).bfloat16().float()
    Wd = {k: v.double() for k, v in W.items()}
    idx_want, w_want = O.route(h.double(), Wd, "", f["router"])
    z = h.double() @ Wd["router"].T + Wd["router.b"]
    srt = z.sort(dim=-1).values
    clear = (srt[:, 1:] - srt[:, :-1]).min(dim=-1).values > 1e-5 if E > 1 else torch.ones(T, dtype=torch.bool)
    assert int(clear.sum()) > T // 2
    if E > top:
        assert not torch.equal(idx_want, (h.double() @ Wd["router"].T).topk(top, dim=-1).indices)
    layer = M.MoEFeedForward({k: v.to(DEV) for k, v in W.items()}, "", experts=E, identity=0, top=top, groups=1, keep=1, ff=ff, score="chosen_softmax",
                             shared_ff=shared)
    want = O.experts(h.double(), Wd, "", f)

    def ctx(n):
        return M.StepContext(n, torch.zeros(2, dtype=torch.int32, device=DEV), {}, torch.float32)

    for n in (T, 3, 1):                       # sorted portions; logits and routing in one launch
        idx, wgt = layer.route(h[:n].to(DEV), ctx(n))
        assert torch.equal(idx.cpu().long()[clear[:n]], idx_want[:n][clear[:n]])
        assert torch.allclose(wgt.cpu().double()[clear[:n]], w_want[:n][clear[:n]], rtol=1e-5, atol=1e-7)
        assert torch.allclose(wgt.sum(-1), torch.ones(n, device=DEV), atol=1e-6)
        assert rel(layer.forward(h[:n].to(DEV), ctx(n)).cpu()[clear[:n]], want[:n][clear[:n]]) < TOL
    few = torch.cat([layer.forward(h[t:t + 4].to(DEV), ctx(4)) for t in range(0, 12, 4)]).cpu()
    assert rel(few[clear[:12]], want[:12][clear[:12]]) < TOL


def test_softmax_over_chosen_logits_far_apart():
    """Logits hundreds apart: the choice follows the logits where a softmax over all experts has nothing left to compare, and
    the chosen weights are exact."""
    P, S, M = _pkg()
    z = torch.tensor([[-300.0, 0.0, -120.0, -121.0, -500.0, -119.5], [1e4, -1e4, 9999.0, 0.0, 9998.5, -5.0]])
    bias = torch.tensor([0.0, 0.5, 0.0, 2.0, 0.0, 0.0])
    zd, bd = z.to(DEV), bias.to(DEV)
    idx, wgt = torch.empty(2, 4, dtype=torch.int32, device=DEV), torch.empty(2, 4, device=DEV)
    S.check(S.lib().b2l_seq_moe_route(zd.data_ptr(), 6, bd.data_ptr(), 6, 1, 1, 4, S.SCORE_CHOSEN_SOFTMAX, 1, 1, 1.0, idx.data_ptr(), wgt.data_ptr(), 2, None), "route")
    v, want = (z + bias).double().topk(4, dim=-1)
    assert torch.equal(idx.cpu().long(), want)
    assert torch.allclose(wgt.cpu().double(), torch.softmax(v, -1), rtol=1e-5, atol=1e-30)
    with pytest.raises(RuntimeError):
        S.check(S.lib().b2l_seq_moe_route(zd.data_ptr(), 6, None, 6, 1, 1, 4, S.SCORE_CHOSEN_SOFTMAX, 0, 1, 1.0, idx.data_ptr(), wgt.data_ptr(), 2, None), "route")


@pytest.mark.parametrize("D", [72, 256, 300, 1000, 1022, 2048, 2050, 4096, 4100, 6002, 9000])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_residual_step(D, dtype):
    P, S, M = _pkg()
    T, eps = 5, 1e-3
    g = torch.Generator().manual_seed(D)

    def r(*s):
        return torch.randn(*s, generator=g)

    x, base, y1, y2, vec, w, b = r(T, D) * 3, r(T, D), r(T, D).to(dtype), r(T, D).to(dtype), r(D).to(dtype), (1 + 0.2 * r(D)).to(dtype), r(D).to(dtype)
    ctx = M.StepContext(T, torch.zeros(2, dtype=torch.int32, device=DEV), {}, dtype)
    tol = 1e-6 if dtype == torch.float32 else 4e-3

    def d(t):
        return t.to(DEV)

    for kw in (dict(y1=y1), dict(y1=y1, y2=y2), dict(base=base, vec=vec), dict(y1=y1, y2=y2, base=base, vec=vec), dict()):
        xs = x.double() + sum(v.double() for v in kw.values())
        out = torch.empty(T, D, device=DEV)
        h = M.residual_step(d(x), out, ctx, norm=d(w), bias=d(b), kind="layer", eps=eps, **{k: d(v) for k, v in kw.items()})
        assert rel(out, xs) < 1e-6
        assert rel(h, O.layer_norm(xs, w.double(), b.double(), eps)) < tol
        h = M.residual_step(d(x), out, ctx, norm=d(w), kind="rms", eps=eps, **{k: d(v) for k, v in kw.items()})
        assert rel(h, O.rms_unit(xs, eps) * w.double()) < tol
        own = d(x)                                                     # in place, no norm; and the split form
        s = M.residual_step(own, own, ctx, split=True, **{k: d(v) for k, v in kw.items()})
        assert rel(own, xs) < 1e-6 and s.shape == (T, 2 * D)
        if dtype == torch.bfloat16:
            assert torch.equal(s[:, :D], own.to(dtype)) and torch.equal(s[:, D:], (own - own.to(dtype).float()).to(dtype))
            assert rel(s[:, :D].double() + s[:, D:].double(), xs) < 2e-5
        if D <= 4096:
            assert torch.equal(M.residual_step(d(x), None, ctx, split=True, **{k: d(v) for k, v in kw.items()}), s)


@pytest.mark.parametrize("D", [40, 57, 136, 1024])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_loop_injection(D, dtype):
    """Before a pass: every form gives the f32 product of the f32 stream (a stream rounded to bf16 would be off by 1e-3)."""
    P, S, M = _pkg()
    g = torch.Generator().manual_seed(D)
    W = {"loop.in": (torch.randn(D, 2 * D, generator=g) / math.sqrt(D)).bfloat16().float(), "loop.step": torch.randn(3, D, generator=g).bfloat16().float()}
    norm, bias = (1 + 0.1 * torch.randn(D, generator=g)).bfloat16().float(), torch.randn(D, generator=g).bfloat16().float()
    inj = M.LoopInjection(W["loop.in"].to(DEV, dtype), W["loop.step"].to(DEV, dtype))
    Wd = {k: v.double() for k, v in W.items()}
    for T in (1, 2, 4, 5, 40):
        x, x0 = torch.randn(T, D, generator=g), torch.randn(T, D, generator=g).bfloat16().float()
        ctx = M.StepContext(T, torch.zeros(2, dtype=torch.int32, device=DEV), {}, dtype)
        base = inj.start(x0.to(DEV), x0.to(DEV, dtype), ctx)
        xd = x.to(DEV)
        split = M.residual_step(xd, None, ctx, split=True) if inj.wants_split(ctx) else None
        for t in range(3):
            new, h = inj.forward(xd, split, base, t, ctx, norm=norm.to(DEV, dtype), bias=bias.to(DEV, dtype), kind="layer", eps=1e-5)
            want = O.inject(x.double(), x0.double(), Wd, t)
            assert rel(new, want) < (2e-6 if dtype == torch.float32 or T <= M.FEW_TOKENS else 2e-5), (T, t, rel(new, want))
            assert rel(h, O.layer_norm(want, norm.double(), bias.double(), 1e-5)) < (TOL if dtype == torch.float32 else 4e-3)
