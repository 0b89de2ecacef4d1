"""GPU: the Lukupel model family and its mechanisms against the plain restatement in tests/lukupel_oracle.py (float64),
on small random models of several shapes: each mechanism alone, whole prompts against token-by-token decoding and
portions of many sizes, interleaved requests, reused slots, keys that dominate just inside and just outside a chunk (in
prompts, across portions and in decoding), memories that last for hundreds of tokens, the first tokens of a sequence,
long decoding through the captured step, layers that share weights, greedy generation through the engine's scheduler."""
import ctypes as C
import json
import math

import pytest
import torch

import lukupel_oracle as O

pytestmark = pytest.mark.gpu

DEV = "cuda"
TOL = 3e-5


def _pkg():
    import lit_llama_b200 as P
    from lit_llama_b200 import _seqlib as S
    from lit_llama_b200 import mixers as M
    return P, S, M


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).norm() / (want.norm() + 1e-30))


# ----------------------------------------------------------------------------- configurations (none is a served model's)
def attn(heads, kv_heads, dim, vdim, scale, size=None, rot=None, factor=None, mlp=None, of=None):
    c = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        c["mask"] = {"size": size}
    if rot:
        c["rot"] = {"base": rot[0], "dims": rot[1]}
        if factor:
            c["rot"]["scaling"] = {"factor": factor}
    return layer("attention", c, mlp, of)


def memory(heads, dim, vdim, cap, mlp=None, of=None):
    return layer("mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, mlp, of)


def layer(kind, mixer, ff, of):
    out = {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}
    if of is not None:
        out["weights_of"] = of
    return out


def config(vocab, width, layers, eps=1e-5, scale=1.0, mult=1.0, cap=None):
    out = {"architecture": "Lukupel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale}, "residual_mult": mult, "layers": layers}
    if cap:
        out["logit_softcap"] = cap
    return out


def cfg_a():
    """Odd sizes, chunks of 7 and 19, partial rotation, three query heads per kv head, weights used three times over (once
    through another shared layer), a recurrence with a feed-forward, attention without one."""
    a, m, b = (3, 1, 10, 12, 0.7, 7, (500.0, 6), 3.0, 50), (3, 10, 14, 6.0, 40), (4, 2, 6, 8, 1.1, 19, (90.0, 4), 1.5)
    return config(131, 72, [memory(*m), attn(*a), attn(*b), memory(2, 7, 9, 9.0), attn(*a, of=1), memory(*m, of=0), attn(*b, of=2), attn(*a, of=4)],
                  eps=1e-5, scale=5.0, mult=0.6, cap=12.0)


def cfg_b():
    """Shapes that take the tiled attention kernel and the chunked recurrence in prompts: 16-byte rows, portions of hundreds of
    tokens; chunks of 96 and 150."""
    return config(200, 128, [memory(4, 32, 64, 11.0), attn(8, 2, 32, 48, 0.2, 96, (7e4, 16), 2.0, 160), attn(4, 4, 24, 32, 0.25, 150, (3e5, 24), 8.0),
                             memory(2, 64, 96, 15.0, 96), attn(8, 2, 32, 48, 0.2, 96, (7e4, 16), 2.0, 160, of=1), memory(4, 32, 64, 11.0, of=0)],
                  eps=1e-6, scale=9.0, mult=0.45, cap=20.0)


def cfg_c():
    """What a served model may happen to make equal or one: one head, kv heads = heads, key size = value size = rotated
    dims, no scaling, a factor of one, no rotation, chunks of one position, chunks longer than any prompt, no chunks, no
    residual multiplier, no embedding scale, no soft cap on the logits, a small gate cap."""
    return config(90, 64, [attn(1, 1, 16, 16, 0.3, 1, (100.0, 16)), memory(1, 16, 16, 1.5, 24), attn(4, 4, 8, 8, 0.9, 100000, (100.0, 8), 1.0, 32),
                           attn(2, 1, 8, 16, 0.8, None, None, None, 16), memory(1, 1, 33, 4.0), memory(5, 8, 4, 15.0), attn(2, 2, 16, 8, 0.5, 2, (1e4, 2), 40.0)],
                  eps=1e-6)


CONFIGS = {"a": cfg_a, "b": cfg_b, "c": cfg_c}


def random_weights(cfg, seed=1):
    """bf16-representable float32 tensors on the CPU under the family's tensor names.  Forget gates from long to short
    memory, input gates around one."""
    g = torch.Generator().manual_seed(seed)
    D, W = cfg["width"], {}

    def rnd(*shape, std=1.0, mean=0.0):
        return (mean + std * torch.randn(*shape, generator=g)).bfloat16().float()

    def lin(o, i, gain=1.0):
        return rnd(o, i, std=gain / math.sqrt(i))

    W["embed"], W["final.norm"] = rnd(cfg["vocab"], D, std=1.5 / cfg["embedding"]["scale"]), rnd(D, std=0.2, mean=1.0)
    for i, l in enumerate(cfg["layers"]):
        if l.get("weights_of") is not None:
            continue
        p, m, c = f"l{i}.", f"l{i}.mix.", l["mixer"]
        H, K, V = c["heads"], c["dim"], c["vdim"]
        W[p + "norm1"] = rnd(D, std=0.2, mean=1.0)
        if l["type"] == "attention":
            G = c["kv_heads"]
            W[m + "q"], W[m + "k"], W[m + "v"], W[m + "o"] = lin(H * K, D), lin(G * K, D), lin(G * V, D), lin(D, H * V)
        else:
            W[m + "q"], W[m + "k"], W[m + "v"], W[m + "g"], W[m + "o"] = lin(H * K, D), lin(H * K, D), lin(H * V, D), lin(H * V, D), lin(D, H * V)
            W[m + "norm"] = rnd(H * V, std=0.3, mean=1.0)
            W[m + "i"], W[m + "i.b"], W[m + "f"], W[m + "f.b"] = lin(H, D, 2.0), rnd(H, std=1.5), lin(H, D, 1.5), rnd(H, std=2.5, mean=3.0)
        if l.get("mlp"):
            W[p + "norm2"], W[p + "mlp.up"], W[p + "mlp.down"] = rnd(D, std=0.2, mean=1.0), lin(l["mlp"]["ff"], D, 1.5), lin(D, l["mlp"]["ff"])
    return W


def build(cfg, dtype, seed=1, n_slots=3, max_positions=512):
    P, S, M = _pkg()
    W = random_weights(cfg, seed)
    model = P.Lukupel(P.LukupelConfig.from_dict(cfg), {k: v.to(DEV, dtype) for k, v in W.items()}, max_positions=max_positions)
    return model, P.Engine(model, n_slots=n_slots), W


def oracle(toks, cfg, W, capture=None):
    """The plain model; without a soft cap in the configuration, one far above every logit."""
    return O.model(toks, dict(cfg, logit_softcap=cfg.get("logit_softcap", 1e9)), W, capture=capture)


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
@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_model_matches_the_oracle_layer_by_layer_f32(name):
    cfg = CONFIGS[name]()
    model, engine, W = build(cfg, torch.float32)
    toks = tokens_of(cfg, 200 if name == "b" else 45)
    cap = []
    want = oracle(toks, cfg, W, capture=cap)
    model.capture_layers = []
    got = run_whole(engine, toks)
    assert len(model.capture_layers) == len(cap) == len(cfg["layers"])
    for i, (g, w) in enumerate(zip(model.capture_layers, cap)):
        assert rel(g, w) < TOL, (name, "layer", i, rel(g, w))
    assert rel(got, want) < TOL


@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_model_bf16_is_close_to_the_oracle(name):
    cfg = CONFIGS[name]()
    model, engine, W = build(cfg, torch.bfloat16)
    toks = tokens_of(cfg, 60)
    got = run_whole(engine, toks)
    assert rel(got, oracle(toks, cfg, W)) < 0.05
    assert rel(run_pieces(engine, toks, [7, 1, 2, 13]), got) < 0.03


@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_portions_and_single_tokens_equal_the_whole_prompt(name):
    cfg = CONFIGS[name]()
    n = 420 if name == "b" else 80          # b: several query tiles, chunks of the recurrence, several chunk borders
    model, engine, W = build(cfg, torch.float32)
    toks = tokens_of(cfg, n)
    whole = run_whole(engine, toks)
    if name != "b":
        assert rel(whole, oracle(toks, cfg, W)) < TOL
    for sizes in ([1], [2], [3, 2, 17, 1, 5], [33, 64], [n - 9, 1, 1, 2]):
        if name == "b" and sizes == [1]:
            sizes = [n - 170, 1]            # a long first portion, then 170 tokens one by one: both chunk sizes are passed while decoding
        got = run_pieces(engine, toks, sizes)
        assert rel(got, whole) < TOL, (name, sizes, rel(got, whole))


def test_long_prompt_matches_the_oracle():
    cfg = cfg_b()
    model, engine, W = build(cfg, torch.float32)
    toks = tokens_of(cfg, 310, seed=9)
    want = oracle(toks, cfg, W)
    assert rel(run_whole(engine, toks), want) < TOL
    assert rel(run_pieces(engine, toks, [261, 1, 2, 1, 1]), want) < TOL


def test_interleaved_requests_and_reused_slots():
    cfg = cfg_a()
    model, engine, W = build(cfg, torch.float32, n_slots=2)
    prompts = [tokens_of(cfg, n, seed=s) for n, s in ((23, 1), (5, 2), (41, 3), (1, 4), (12, 5))]
    alone = [run_whole(engine, p, rid=("alone", i)) for i, p in enumerate(prompts)]
    for i, p in enumerate(prompts):
        assert rel(alone[i], oracle(p, cfg, W)) < TOL
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
    cfg = cfg_a()                            # the chunks of 7 and 19 are passed many times; the recurrences run 230 steps
    model, engine, W = build(cfg, torch.float32)
    toks = tokens_of(cfg, 230)
    want = oracle(toks, cfg, W)
    first = engine.step([{"id": "d", "tokens": toks[:20], "want": [19]}])[0]
    outs = [first] + [engine.step([{"id": "d", "tokens": [t], "want": [0]}])[0] for t in toks[20:]]
    assert engine._graph is not None
    assert rel(torch.cat(outs), want[19:]) < TOL
    # the same captured step serves another request in another slot from its first token on
    outs2 = [engine.step([{"id": "e", "tokens": [t], "want": [0]}])[0] for t in toks[:40]]
    assert rel(torch.cat(outs2), want[:40]) < TOL


def test_first_tokens_of_a_sequence():
    """One-token and two-token sequences in a slot that another request used before: matrix, normaliser and running maximum
    start from zero, the first tokens see no key before position 0."""
    cfg = cfg_a()
    model, engine, W = build(cfg, torch.float32, n_slots=1)
    run_whole(engine, tokens_of(cfg, 30, seed=2))
    for toks in ([7], [7, 7], [130, 0], tokens_of(cfg, 3), tokens_of(cfg, 8)):
        want = oracle(toks, cfg, W)
        assert rel(run_whole(engine, toks), want) < TOL
        assert rel(run_pieces(engine, toks, [1]), want) < TOL
        assert rel(run_pieces(engine, toks, [2, 1]), want) < TOL
    assert engine.pool.reused >= 10


def test_shared_layers_share_weights_and_nothing_else():
    cfg = cfg_a()
    model, engine, W = build(cfg, torch.float32)
    L = model.layers
    for i, j in ((4, 1), (7, 1), (5, 0), (6, 2)):
        assert L[i].mixer.w_in is L[j].mixer.w_in and L[i].norm1 is L[j].norm1 and L[i].mlp is L[j].mlp
        assert L[i].mixer.name == f"l{i}" and not set(L[i].mixer.state_specs()) & set(L[j].mixer.state_specs())
    assert len(model.state_specs()) == 5 * 2 + 3 * 3
    separate = cfg_a()
    for l in separate["layers"]:
        l.pop("weights_of", None)
    other = random_weights(separate, 1)
    for i in (4, 5, 6, 7):                   # the same model written out with copies of the shared tensors
        src = f"l{O.owner(cfg['layers'], i)}."
        other.update({f"l{i}." + k[len(src):]: v for k, v in W.items() if k.startswith(src)})
    other = {k: W.get(k, v) for k, v in other.items()}
    P, S, M = _pkg()
    twin = P.Lukupel(P.LukupelConfig.from_dict(separate), {k: v.to(DEV) for k, v in other.items()})
    assert twin.n_parameters() > model.n_parameters()
    toks = tokens_of(cfg, 40)
    assert rel(run_whole(P.Engine(twin, n_slots=1), toks), run_whole(engine, toks)) < 1e-6


def test_position_limit_only_without_chunks():
    P, S, M = _pkg()
    model, engine, W = build(cfg_c(), torch.float32, max_positions=16)
    toks = tokens_of(cfg_c(), 20)
    engine.step([{"id": "x", "tokens": toks[:16], "want": []}])
    with pytest.raises(P.state.PoolFull):
        engine.step([{"id": "x", "tokens": toks[16:], "want": [0]}])
    model, engine, W = build(cfg_a(), torch.float32, max_positions=16)
    assert model.max_positions == 0
    engine.step([{"id": "x", "tokens": tokens_of(cfg_a(), 50), "want": []}])


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
            lg = oracle(seq, cfg, W)[-1]
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


def test_registry_loads_a_saved_model(tmp_path):
    P, S, M = _pkg()
    from lit_llama_b200.checkpoint_io import write_safetensors

    cfg = cfg_a()
    W = random_weights(cfg, seed=3)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(str(tmp_path / "model.safetensors"), {k: v.bfloat16() for k, v in W.items()})
    toks = tokens_of(cfg, 12)
    want = oracle(toks, cfg, W)
    for dtype, tol in ((torch.float32, TOL), (torch.bfloat16, 0.05)):
        model = P.load_model(str(tmp_path), dtype=dtype, device=DEV, max_positions=64)
        assert type(model).__name__ == "Lukupel" and model.dtype == dtype
        assert rel(run_whole(P.Engine(model, n_slots=1), toks), want) < tol


# ----------------------------------------------------------------------------- mechanisms alone
def _run_mixer(M, P, mixer, h, sizes, dtype=torch.float32, slot=1):
    """A mixer over h [T, width] in portions of the given sizes (cycled) in one slot of a fresh pool."""
    pool = P.SequenceStatePool(mixer.state_specs(), 2, torch.device(DEV))
    pool.acquire("other")
    pool.acquire("it")
    assert pool.slot("it") == slot
    outs, at, i = [], 0, 0
    while at < h.shape[0]:
        n = min(sizes[i % len(sizes)], h.shape[0] - at)
        meta = torch.tensor([slot, at], dtype=torch.int32, device=DEV)
        ctx = M.StepContext(n, meta, pool.tensors, dtype, pos_hint=at, slot_hint=slot)
        outs.append(mixer.forward(h[at:at + n].to(DEV, dtype).contiguous(), ctx))
        at, i = at + n, i + 1
    for name, t in pool.tensors.items():
        assert float(t[1 - slot].abs().max()) == 0.0, name              # the other slot is untouched
    return torch.cat(outs).float().cpu()


def _mixer_weights(l, D, seed):
    W = random_weights(config(8, D, [l], eps=1e-6), seed)
    return {k[len("l0.mix."):]: v for k, v in W.items() if k.startswith("l0.mix.")}


@pytest.mark.parametrize("shape", [(3, 1, 10, 12, 7, 4), (8, 2, 32, 48, 96, 8), (4, 4, 24, 32, 150, 0), (2, 1, 64, 128, 64, 16), (6, 3, 40, 72, 33, 20), (2, 2, 128, 64, 130, 32)])
def test_chunk_attention_alone_with_standout_keys_at_the_borders(shape):
    P, S, M = _pkg()
    H, G, K, V, size, rd = shape
    D, T = 48, 330
    # heads of unit root mean square: a score is scale * K * cosine, so 14 for equal directions and within a few units of 0 otherwise
    l = attn(H, G, K, V, 14.0 / K, size, (700.0, rd) if rd else None, 5.0 if rd else None)
    c = l["mixer"]
    W = _mixer_weights(l, D, 3)
    for g in range(G):                       # the first query head of every group looks for keys like itself
        W["k"][g * K:(g + 1) * K] = W["q"][g * (H // G) * K:(g * (H // G) + 1) * K]
    h = torch.randn(T, D, generator=torch.Generator().manual_seed(1))
    # pairs (query, key): the key at the first position of the query's chunk and the one just before it, for the last queries of
    # chunks, for a portion's last token and for decoded tokens
    queries = [q for q in (2 * size - 1, 200, 297, 329, size - 2) if 0 < q < T and q % size]
    taken = set(queries)
    for q in queries:
        lo = (q // size) * size
        for k, gain in ((lo, 2.0), (lo - 1, 6.0)):      # the query's direction for q and k, a value of its own
            if k >= 0 and k not in taken:
                h[k] = h[q] * gain
                taken.add(k)
    assert len(taken) > len(queries) + 2
    h = h.bfloat16().float()
    want = O.chunk_attention(h.double(), W, "", c, 1e-6)
    for off in (-1, 1):                      # a border one token off shows in these inputs: some token is another one
        wrong = O.chunk_attention(h.double(), W, "", dict(c, mask={"size": size + off}), 1e-6)
        assert float(((wrong - want).norm(dim=1) / want.norm(dim=1)).max()) > 0.2
    kw = dict(heads=H, kv_heads=G, dim=K, vdim=V, scale=c["scale"], eps=1e-6, block=size, rot=c.get("rot"), norm_over="unit", gate=False)
    mixer = M.LocalAttention("m", {k: v.to(DEV) for k, v in W.items()}, "", **kw)
    assert mixer.state_specs()["m.k"].shape == (size, G, K)
    for sizes in ([T], [1], [201, 1], [64, 1, 2, 37], [2], [297, 1]):
        got = _run_mixer(M, P, mixer, h, sizes)
        assert rel(got, want) < TOL, (shape, sizes, rel(got, want))
    mixer = M.LocalAttention("m", {k: v.to(DEV, torch.bfloat16) for k, v in W.items()}, "", **kw)
    assert rel(_run_mixer(M, P, mixer, h, [100, 1, 29], dtype=torch.bfloat16), want) < 0.06


def test_local_attention_refuses_what_it_cannot_mean():
    P, S, M = _pkg()
    W = {k: v.to(DEV) for k, v in _mixer_weights(attn(2, 1, 8, 8, 1.0, 4), 16, 1).items()}
    kw = dict(heads=2, kv_heads=1, dim=8, vdim=8, scale=1.0, eps=1e-6, gate=False)
    for bad in (dict(window=4, block=4), dict(), dict(block=4, norm_over="column")):
        with pytest.raises(ValueError):
            M.LocalAttention("m", W, "", **dict(kw, **bad))
    # a window in place of chunks, with the same weightless norm after the rotation
    mixer = M.LocalAttention("m", W, "", window=5, norm_over="unit", **kw)
    h = torch.randn(30, 16, generator=torch.Generator().manual_seed(2))
    q, k = O.heads_rotated_then_normed(h.double() @ W["q"].double().cpu().T, 2, 8, None, 1e-6), O.heads_rotated_then_normed(h.double() @ W["k"].double().cpu().T, 1, 8, None, 1e-6)
    v = (h.double() @ W["v"].double().cpu().T).view(30, 1, 8)
    want = torch.zeros(30, 2, 8, dtype=torch.float64)
    for i in range(30):
        lo = max(0, i - 4)
        for hd in range(2):
            want[i, hd] = torch.softmax(k[lo:i + 1, 0] @ q[i, hd], 0) @ v[lo:i + 1, 0]
    want = want.reshape(30, 16) @ W["o"].double().cpu().T
    for sizes in ([30], [1], [7, 2]):
        assert rel(_run_mixer(M, P, mixer, h, sizes), want) < TOL


def _memory_case(shape, D, T, seed, long_memory):
    """Weights and inputs of one recurrence: one loud input gate early on (a far token that dominates), or gates that open and
    close at random."""
    H, K, V, cap = shape
    l = memory(H, K, V, cap)
    W = _mixer_weights(l, D, seed)
    h = torch.randn(T, D, generator=torch.Generator().manual_seed(seed + 1))
    if long_memory:
        W["f.b"] = torch.linspace(6.0, 9.0, H).bfloat16().float()                 # forget gates of 0.9975 ... 0.9999
        W["f"] = (W["f"] * 0.1).bfloat16().float()
        W["i"][0] = 0.0
        W["i"][:, 0] = 3.0
        h[:, 0] = -1.0
        for t in (3, 127, 128, 255, 256, 300):                                    # far tokens written a hundred times louder
            if t < T:
                h[t, 0] = 1.5
    return l, W, h.bfloat16().float()


@pytest.mark.parametrize("long_memory", [False, True])
@pytest.mark.parametrize("shape", [(3, 10, 14, 6.0), (4, 32, 64, 11.0), (2, 64, 100, 15.0), (1, 1, 33, 4.0), (2, 128, 256, 8.0), (1, 200, 40, 20.0)])
def test_matrix_memory_alone(shape, long_memory):
    P, S, M = _pkg()
    D, T = 48, 420
    H, K, V, cap = shape
    l, W, h = _memory_case(shape, D, T, 7, long_memory)
    c = l["mixer"]
    # the unit-RMS read-out hides a head's denominator: a large eps under its root brings the normaliser's scale out
    eps = 0.3 if long_memory else 1e-6
    want = O.mlstm(h.double(), W, "", c, eps)
    mixer = M.MatrixMemoryMixer("m", {k: v.to(DEV) for k, v in W.items()}, "", heads=H, dim=K, vdim=V, gate_cap=cap, eps=eps)
    assert S.lib().b2l_seq_scan_chunks(T, 0) > 1 and S.lib().b2l_seq_scan_chunks(100, 0) == 1
    for sizes in ([T], [1], [100, 1, 2, 63], [T - 1, 1], [257, 163], [2]):
        got = _run_mixer(M, P, mixer, h, sizes)
        assert rel(got, want) < TOL, (shape, sizes, rel(got, want))
    mixer = M.MatrixMemoryMixer("m", {k: v.to(DEV, torch.bfloat16) for k, v in W.items()}, "", heads=H, dim=K, vdim=V, gate_cap=cap, eps=eps)
    assert rel(_run_mixer(M, P, mixer, h, [300, 1, 60], dtype=torch.bfloat16), want) < 0.06


def test_matrix_memory_takes_both_sides_of_its_denominator():
    """Both max(|n . q|, exp(-m)) sides occur, and a state that lost its normaliser or its running maximum would show (with an eps
    that keeps the unit-RMS read-out from hiding the denominator)."""
    l, W, h = _memory_case((3, 10, 14, 6.0), 48, 200, 3, False)
    c = l["mixer"]
    hd = h.double()
    li, lf = O.log_gates(hd, W, "", c["gate_cap"])
    q, k = (hd @ O.w64(W, "q").T).view(200, 3, 10) * 10 ** -0.5, (hd @ O.w64(W, "k").T).view(200, 3, 10)
    sides = set()
    for a in range(3):
        n, m = torch.zeros(10, dtype=torch.float64), 0.0
        for t in range(200):
            new = max(float(lf[t, a]) + m, float(li[t, a]))
            n = math.exp(float(lf[t, a]) + m - new) * n + math.exp(float(li[t, a]) - new) * k[t, a]
            m = new
            sides.add(abs(float(n @ q[t, a])) > math.exp(-m))
    assert sides == {True, False}
    P, S, M = _pkg()
    mixer = M.MatrixMemoryMixer("m", {k_: v.to(DEV) for k_, v in W.items()}, "", heads=3, dim=10, vdim=14, gate_cap=6.0, eps=0.3)
    want = O.mlstm(hd, W, "", c, 0.3)
    assert rel(_run_mixer(M, P, mixer, h, [57, 1]), want) < TOL
    # a long memory over a cut: a restatement that loses S, n or m there gives something else
    l, W, h = _memory_case((3, 10, 14, 6.0), 48, 200, 3, True)
    mixer = M.MatrixMemoryMixer("m", {k_: v.to(DEV) for k_, v in W.items()}, "", heads=3, dim=10, vdim=14, gate_cap=6.0, eps=0.3)
    want = O.mlstm(h.double(), W, "", l["mixer"], 0.3)
    for t in (5, 57, 120):
        assert rel(_run_mixer(M, P, mixer, h, [t, 200 - t]), want) < TOL
        assert rel(_run_mixer(M, P, mixer, h, [t, 1, 199 - t]), want) < TOL
        for part in "Snm":
            assert rel(O.mlstm(h.double(), W, "", l["mixer"], 0.3, lose=(t, part)), want) > 0.03, (t, part)


def test_gate_kernel_over_several_tiles():
    P, S, M = _pkg()
    H, T = 3, 2600                            # the gate kernel scans 1024 tokens at a time
    g = torch.Generator().manual_seed(5)
    z = 4.0 * torch.randn(T, 2 * H, generator=g)
    z[1030:1060, :H] += 9.0                   # a run of large input gates right behind a tile's edge
    b = torch.randn(2, H, generator=g)
    cap = 7.0
    li, f = O.soft_cap((z[:, :H] + b[0]).double(), cap), O.soft_cap((z[:, H:] + b[1]).double(), cap)
    lf = -torch.log1p(torch.exp(-f))
    want = torch.zeros(3, T, H, dtype=torch.float64)
    end = []
    for a in range(H):
        m = 0.0
        for t in range(T):
            new = max(float(lf[t, a]) + m, float(li[t, a]))
            want[0, t, a], want[1, t, a], want[2, t, a] = math.exp(float(lf[t, a]) + m - new), math.exp(float(li[t, a]) - new), math.exp(-new)
            m = new
        end.append(m)
    zd, bd, state = z.to(DEV), b.to(DEV), torch.zeros(2, H, device=DEV)
    outs = []
    at = 0
    for n in (2, 1500, 1, 3, T - 1506):
        out = torch.empty(3, n, H, device=DEV)
        meta = torch.tensor([1, at], dtype=torch.int32, device=DEV)
        a = S.MlstmArgs(proj=zd[at:].data_ptr(), ld=2 * H, g_off=0, i_off=0, f_off=H, b_i=bd[0].data_ptr(), b_f=bd[1].data_ptr(), gate_cap=cap, state_m=state.data_ptr(),
                        meta=meta.data_ptr(), keep=out[0].data_ptr(), put=out[1].data_ptr(), floor=out[2].data_ptr(), T=n, heads=H, K=4, V=1, act_dtype=S.B2L_F32)
        S.check(S.lib().b2l_seq_mlstm_gates(C.byref(a), None), "gates")
        outs.append(out.cpu())
        at += n
    got = torch.cat(outs, dim=1)
    for i in range(3):
        assert rel(got[i], want[i]) < 3e-6, (i, rel(got[i], want[i]))
    assert rel(state[1], torch.tensor(end)) < 1e-6 and float(state[0].abs().max()) == 0.0
    a.T = 2
    assert S.lib().b2l_seq_mlstm_step(C.byref(a), None) != 0 and b"one token" in S.lib().b2l_seq_last_error()


def test_scan_keeps_a_column_of_ones():
    """The normaliser of the scan equals a value column that holds 1 everywhere, sequential and chunked."""
    P, S, M = _pkg()
    g = torch.Generator().manual_seed(6)
    for H, K, V, T in ((2, 16, 64, 40), (3, 10, 7, 30), (2, 32, 128, 400), (1, 100, 65, 300)):
        q, k = torch.randn(T, H * K, generator=g).to(DEV), torch.randn(T, H * K, generator=g).to(DEV)
        v = torch.randn(T, H * V, generator=g).to(DEV)
        d, s = torch.rand(T, H, generator=g).to(DEV) * 0.2 + 0.8, torch.rand(T, H, generator=g).to(DEV)
        v1 = torch.cat([v.view(T, H, V), torch.ones(T, H, 1, device=DEV)], dim=2).reshape(T, H * (V + 1)).contiguous()
        meta = torch.tensor([0, 0], dtype=torch.int32, device=DEV)
        ctx = M.StepContext(T, meta, {}, torch.float32)
        kw = dict(q=M._p(q), ldq=H * K, k=M._p(k), ldk=H * K, q_mult=0.3, decay=M._p(d), ldd=H, per_channel=False, vscale=M._p(s), ldvs=H, heads=H, qk_heads=H, K=K)
        st0 = torch.randn(1, H, V + 1, K, generator=g).to(DEV)
        st, wide = st0.clone(), torch.empty(T, H * (V + 1), device=DEV)
        M._scan(ctx, v=M._p(v1), ldv=H * (V + 1), state=st, out=M._p(wide), ldo=H * (V + 1), V=V + 1, **kw)
        stS, stn = st0[:, :, :V].contiguous(), st0[:, :, V].contiguous()
        o, nq = torch.empty(T, H * V, device=DEV), torch.empty(T, H, device=DEV)
        M._scan(ctx, v=M._p(v), ldv=H * V, state=stS, out=M._p(o), ldo=H * V, V=V, state_ones=stn, out_ones=M._p(nq), **kw)
        wide = wide.view(T, H, V + 1)
        assert rel(o.view(T, H, V), wide[..., :V]) < 1e-6 and rel(nq, wide[..., V]) < 1e-6, (H, K, V, T)
        assert rel(stS, st[:, :, :V]) < 1e-6 and rel(stn, st[:, :, V]) < 1e-6


def test_post_norm_residual_step_and_embedding_kernels_alone():
    P, S, M = _pkg()
    lib = S.lib()
    g = torch.Generator().manual_seed(8)
    for dtype, tol in ((torch.float32, 1e-6), (torch.bfloat16, 4e-3)):
        for D in (72, 328, 1500, 3000, 4500):
            T = 5
            y = torch.randn(T, D, generator=g).bfloat16().float()
            x, w, wn = torch.randn(T, D, generator=g), torch.randn(D, generator=g).bfloat16().float(), torch.randn(D, generator=g).bfloat16().float()
            x_want = x.double() + 0.35 * O.rms_norm(y.double(), w.double(), 1e-5)
            yd, wd, wnd = y.to(DEV, dtype), w.to(DEV, dtype), wn.to(DEV, dtype)
            for w_next, h_want in ((None, x_want), (wnd, O.rms_norm(x_want, wn.double(), 1e-5))):
                xd, h = x.to(DEV), torch.zeros(T, D, dtype=dtype, device=DEV)
                S.check(lib.b2l_seq_norm_add_norm(M._p(yd), M._p(wd), 1e-5, 0.35, M._p(xd), M._p(w_next), M._p(h), T, D, S.act_code(dtype), None), "step")
                assert rel(xd, x_want) < 1e-6 and rel(h, h_want) < tol, (dtype, D)
            xd = x.to(DEV)
            S.check(lib.b2l_seq_norm_add_norm(M._p(yd), M._p(wd), 1e-5, 0.35, M._p(xd), None, None, T, D, S.act_code(dtype), None), "step")
            assert rel(xd, x_want) < 1e-6
        tab, tok = torch.randn(11, 50, generator=g).bfloat16().float(), torch.tensor([3, 10, 0, 3])
        tabd, tokd = tab.to(DEV, dtype), tok.to(DEV)
        xe, he = torch.empty(4, 50, device=DEV), torch.empty(4, 50, dtype=dtype, device=DEV)
        S.check(lib.b2l_seq_embed(M._p(tokd), 1, M._p(tabd), S.act_code(dtype), 1.7, M._p(xe), M._p(he), 4, 50, 11, None), "embed")
        assert rel(xe, tab[tok] * 1.7) < 1e-6 and rel(he, tab[tok] * 1.7) < tol


def test_attention_operands_normed_after_the_rotation():
    P, S, M = _pkg()
    g = torch.Generator().manual_seed(9)
    for H, G, K, V, rd, mult in ((3, 1, 10, 12, 6, 1.0), (4, 2, 40, 8, 40, 1.0), (2, 2, 64, 16, 0, 1.0), (5, 5, 128, 8, 32, 1.3)):
        T, pos0 = 9, 1234
        proj = torch.randn(T, (H + G) * K + G * V, generator=g)
        proj[2] *= 1e-3                       # small rows: eps counts
        f = [50.0 ** (-2.0 * i / max(rd, 1)) / 3.0 for i in range(rd // 2)]
        want = []
        for x, n in ((proj[:, :H * K], H), (proj[:, H * K:(H + G) * K], G)):
            x = x.double().reshape(T, n, K).clone()
            for t in range(T):
                for a in range(n):
                    x[t, a] = O.rotate(x[t, a], pos0 + t, f)
                    x[t, a, :rd] *= mult
            want.append(O.unit_rms(x, 1e-6).reshape(T, n * K))
        pd, freq, meta = proj.to(DEV), torch.tensor(f, dtype=torch.float32, device=DEV) if rd else None, torch.tensor([0, pos0], dtype=torch.int32, device=DEV)
        q, k = torch.empty(T, H * K, device=DEV), torch.empty(T, G * K, device=DEV)
        a = S.QkvPrepArgs(proj=M._p(pd), ld=pd.shape[1], q_off=0, k_off=H * K, v_off=(H + G) * K, eps=1e-6, freq=M._p(freq), rot_dims=rd, rot_mult=mult, meta=M._p(meta),
                          q_out=M._p(q), k_out=M._p(k), T=T, heads=H, kv_heads=G, K=K, V=V, act_dtype=S.B2L_F32, unit_rms=1)
        S.check(S.lib().b2l_seq_qkv_prep(C.byref(a), None), "prep")
        assert rel(q, want[0]) < 1e-4 and rel(k, want[1]) < 1e-4, (H, K)          # angles of 1234 rad in f32
        small = [rel(o[2], w[2]) for o, w in zip((q, k), want)]
        assert max(small) < 1e-4
        w1 = torch.ones(K, device=DEV)
        a.q_norm = M._p(w1)
        assert S.lib().b2l_seq_qkv_prep(C.byref(a), None) != 0


def test_feed_forward_alone():
    P, S, M = _pkg()
    D, T = 40, 21
    for ff in (50, 392):
        W = {k[len("l0.mlp."):]: v for k, v in random_weights(config(8, D, [memory(1, 4, 4, 5.0, ff)]), 11).items() if k.startswith("l0.mlp.")}
        h = torch.randn(T, D, generator=torch.Generator().manual_seed(10)).bfloat16().float()
        want = O.dense_ff(h.double(), W, "")
        for dtype, tol in ((torch.float32, TOL), (torch.bfloat16, 0.02)):
            mlp = M.DenseMLP(W["up"].to(DEV, dtype), W["down"].to(DEV, dtype), act="relu2")
            for n in (T, 1):
                ctx = M.StepContext(n, torch.zeros(2, dtype=torch.int32, device=DEV), {}, dtype)
                hd = h[:n].to(DEV, dtype)
                keep = hd.clone()
                assert rel(mlp.forward(hd, ctx), want[:n]) < tol and torch.equal(hd, keep)
