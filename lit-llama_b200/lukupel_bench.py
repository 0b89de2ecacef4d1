"""Throughput of the Lukupel family beside the package's Lugovik family at equal width and depth
(`bench.py --family lukupel`).

Random weights, bf16, one sequence: prefill of a `prompt`-token prompt in one portion, then single-token decoding
through the engine (CUDA-graph replay).  The Lugovik arm is the closest served model: matrix-state recurrences beside
block-local attention, post-norms on an f32 residual stream, dense feed-forwards, the same engine, state pool and library
products.  A second table times the family's mechanisms alone at the model's shapes with their algorithmic bytes and flops,
each next to the like kernel of the closest model run on operands of the same size.  CUDA events, warm-up, L2 flushed
between iterations."""
import ctypes as C
import json
import os
import time
from typing import List

import torch

from . import seq_bench, zenasun_bench

SIZES = {
    # the layer pattern repeats: mlstm without feed-forward, then three attention layers with one.  ff is 3/2 of the closest
    # model's: its feed-forwards have three matrices
    "1k": dict(width=1024, layers=8, heads=8, kv_heads=2, dim=128, chunk=1024, m_heads=4, m_dim=128, m_vdim=256, ff=6144, vocab=32000),
    "2k": dict(width=2048, layers=8, heads=16, kv_heads=4, dim=128, chunk=2048, m_heads=4, m_dim=256, m_vdim=512, ff=12288, vocab=32000),
}


def lukupel_config(width, layers, heads, kv_heads, dim, chunk, m_heads, m_dim, m_vdim, ff, vocab, shared=False) -> dict:
    """shared: every layer after the first four runs the weights of the layer four before it once more."""
    att = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "mask": {"size": chunk},
           "rot": {"base": 1e6, "dims": dim // 2, "scaling": {"factor": 8.0}}}
    mem = {"heads": m_heads, "dim": m_dim, "vdim": m_vdim, "gate_cap": 12.0}
    out = []
    for i in range(layers):
        l = {"type": "mlstm", "mixer": mem, "mlp": None} if i % 4 == 0 else {"type": "attention", "mixer": att, "mlp": {"kind": "dense", "ff": ff}}
        out.append(dict(l, weights_of=i - 4) if shared and i >= 4 else l)
    return {"architecture": "Lukupel", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "embedding": {"scale": width ** 0.5}, "residual_mult": 0.8,
            "logit_softcap": 25.0, "layers": out}


def kernel_table(model, engine, T: int, device, timer, peaks: dict) -> List[dict]:
    """The family's mechanisms alone at this model's shapes, each followed by the like kernel of the closest model: a
    T-token portion from position 0 and one token deep inside its chunk."""
    from . import _seqlib as S
    from . import mixers as M

    rows, hbm, es = [], peaks["hbm_gbs"] * 1e9, 2
    slot = engine.pool.acquire("kernels")
    D, dt, lib, eps = model.width, model.dtype, S.lib(), model.eps
    att = next(l.mixer for l in model.layers if isinstance(l.mixer, M.LocalAttention))
    mem = next(l.mixer for l in model.layers if isinstance(l.mixer, M.MatrixMemoryMixer))
    mlp = next(l.mlp for l in model.layers if l.mlp is not None)
    H, G, K, V, ring = att.H, att.G, att.K, att.V, att.ring

    def add(name, tt, t, nbytes, flops=0.0, note=""):
        rows.append({"kernel": name, "tokens": int(tt), "us": t * 1e6, "GB_s": nbytes / t / 1e9, "frac_of_measured_hbm": nbytes / t / hbm,
                     "GFLOP_s": flops / t / 1e9, "note": note})

    full = M.StepContext(T, torch.tensor([slot, 0], dtype=torch.int32, device=device), engine.pool.tensors, dt, pos_hint=0, slot_hint=slot)
    att.forward(torch.randn(T, D, device=device).to(dt), full)          # a filled ring
    for tt, pos0 in ((T, 0), (1, min(T, ring) - 1)):
        meta = torch.tensor([slot, pos0], dtype=torch.int32, device=device)
        ctx = M.StepContext(tt, meta, engine.pool.tensors, dt)
        act, st = ctx.act, ctx.stream
        hh = torch.randn(tt, D, device=device).to(dt)
        y, x, h, w = torch.randn(tt, D, device=device).to(dt), torch.randn(tt, D, device=device), torch.empty(tt, D, dtype=dt, device=device), torch.ones(D, dtype=dt, device=device)
        # ---- residual step
        nb = tt * D * (es + 4 + 4 + es)
        for name, nxt in (("seq_norm_add_norm_kernel (post-norm, multiplied sum, the stream cast for the next sublayer)", None),
                          ("  like: seq_norm_add_norm_kernel (post-norm, sum, next pre-norm)", w)):
            t = timer(lambda: S.check(lib.b2l_seq_norm_add_norm(M._p(y), M._p(w), eps, 0.8, M._p(x), M._p(nxt), M._p(h), tt, D, act, st), "k"))
            add(name, tt, t, nb)
        # ---- attention operands
        ld = att.w_in.shape[0]
        proj = torch.randn(tt, ld, device=device).to(dt)
        q, kn, wk = torch.empty(tt, H * K, device=device), torch.empty(tt, G * K, dtype=dt, device=device), torch.ones(K, dtype=dt, device=device)
        a = S.QkvPrepArgs(proj=M._p(proj), ld=ld, q_off=att.o_q, k_off=att.o_k, v_off=att.o_v, eps=eps, freq=M._p(att.freq), rot_dims=att.rot_dims, rot_mult=1.0,
                          meta=M._p(meta), q_out=M._p(q), k_out=M._p(kn), T=tt, heads=H, kv_heads=G, K=K, V=V, act_dtype=act, unit_rms=1)
        nb = tt * ((H + G) * K * es + H * K * 4 + G * K * es)
        t = timer(lambda: S.check(lib.b2l_seq_qkv_prep(C.byref(a), st), "k"))
        add("seq_qkv_prep_kernel (rotation, unit RMS per head, q and k)", tt, t, nb)

        def two_norms():
            for off, out, f32, n in ((att.o_q, q, 1, H), (att.o_k, kn, 0, G)):
                S.check(lib.b2l_seq_headnorm_rope(M._p(proj, off), ld, M._p(wk), eps, M._p(att.freq), att.rot_dims, 1.0, M._p(meta), M._p(out), f32, tt, n, K, act, st), "k")

        add("  like: 2 x seq_headnorm_rope_kernel (weighted norm per head, rotation)", tt, timer(two_norms), nb)
        # ---- attention inside chunks
        keys = (sum(n * (n + 1) / 2 for n in (min(ring, tt - lo) for lo in range(0, tt, ring))) / tt) if tt > 1 else pos0 % ring + 1
        out = torch.empty(tt, H * V, dtype=dt, device=device)
        gate = torch.randn(tt, H, device=device).to(dt)
        nb = tt * (H * K * 4 + G * (K + V) * es * 2 + H * V * es) + (keys * G * (K + V) * es if tt == 1 else 0)
        for name, kw in (("seq_block_attention (chunks, ordinary softmax) + append", dict(gate=None, ldg=0, softcap=0.0, has_sink=0)),
                         ("  like: seq_block_attention (blocks, sink, soft-capped scores, gate per head) + append", dict(gate=M._p(gate), ldg=H, softcap=50.0, has_sink=1))):
            b = S.AttnArgs(q=M._p(q), k_new=M._p(kn), v_new=M._p(proj, att.o_v), ldv=ld, cache_k=M._p(ctx.state[att.name + ".k"]),
                           cache_v=M._p(ctx.state[att.name + ".v"]), meta=M._p(meta), out=M._p(out), ldo=H * V, scale=att.scale, out_mult=1.0, block=ring, T=tt,
                           heads=H, kv_heads=G, K=K, V=V, act_dtype=act, **kw)
            t = timer(lambda: M.local_attention(b, ctx))
            add(name, tt, t, nb, 2.0 * tt * H * keys * (K + V), f"f32 scores on CUDA cores, {keys:.0f} keys per query")
        t = timer(lambda: att.forward(hh, ctx))
        wb = (att.w_in.numel() + att.w_o.numel()) * es
        add("LocalAttention whole (2 products + operands + attention)", tt, t, wb + 2 * tt * D * es, 2.0 * tt * H * keys * (K + V) + 2.0 * tt * wb / es)
        rows += memory_rows(model, mem, ctx, tt, timer, hbm)
        # ---- feed-forward
        u, gu = torch.randn(tt, mlp.ff, device=device).to(dt), torch.randn(tt, 2 * mlp.ff, device=device).to(dt)
        t = timer(lambda: S.check(lib.b2l_seq_unary_act(M._p(u), mlp.ff, M._p(u), mlp.ff, tt, mlp.ff, mlp.act, None, act, st), "k"))
        add("seq_unary_act_kernel (square of relu, in place)", tt, t, tt * mlp.ff * 2 * es)
        t = timer(lambda: S.check(lib.b2l_seq_gated_act(M._p(gu), 2 * mlp.ff, M._p(u), tt, mlp.ff, S.ACT_GELU_TANH, 0.0, act, st), "k"))
        add("  like: seq_gated_act_kernel (gelu gate)", tt, t, tt * mlp.ff * 3 * es)
        t = timer(lambda: mlp.forward(hh, ctx))
        wb = (mlp.w_up.numel() + mlp.w_down.numel()) * es
        add("DenseMLP whole (2 products + square of relu)", tt, t, wb + 2 * tt * D * es, 2.0 * tt * wb / es)
        # ---- ends of the model
        tok = torch.randint(0, model.vocab, (tt,), device=device)
        for name, ho in (("seq_embed_kernel (f32 stream and its cast)", h), ("  like: seq_embed_kernel (f32 stream)", None)):
            t = timer(lambda: S.check(lib.b2l_seq_embed(M._p(tok), 1, M._p(model.embed), act, 2.0, M._p(x), M._p(ho), tt, D, model.vocab, st), "k"))
            add(name, tt, t, tt * D * (es + 4 + (es if ho is not None else 0)))
        z = torch.randn(1, model.vocab, device=device)
        if tt == 1:
            t = timer(lambda: S.check(lib.b2l_seq_softcap(M._p(z), model.vocab, 25.0, st), "k"))
            add("seq_softcap_kernel (one row of logits)", 1, t, model.vocab * 8)
            t = timer(lambda: S.check(lib.b2l_seq_scale(M._p(z), model.vocab, 1.0, st), "k"))
            add("  like: seq_scale_kernel (one row of logits)", 1, t, model.vocab * 8)
    engine.pool.release("kernels")
    return rows


def memory_rows(model, mem, ctx, tt: int, timer, hbm: float) -> List[dict]:
    """The matrix memory between its two products, whole and kernel by kernel, beside the closest model's scalar-decay
    recurrence with the same state (cast, decay, scan, grouped norm with its gate)."""
    from . import _seqlib as S
    from . import mixers as M

    rows, lib, es, device, dt, eps = [], S.lib(), 2, model.device, model.dtype, model.eps
    H, K, V, act, st = mem.H, mem.K, mem.V, ctx.act, ctx.stream
    ld = mem.w_in.shape[0]

    def add(name, t, nbytes, flops=0.0, note=""):
        rows.append({"kernel": name, "tokens": int(tt), "us": t * 1e6, "GB_s": nbytes / t / 1e9, "frac_of_measured_hbm": nbytes / t / hbm,
                     "GFLOP_s": flops / t / 1e9, "note": note})

    proj, projb = torch.randn(tt, ld, device=device), torch.randn(tt, ld, device=device).to(dt)
    out = torch.empty(tt, H * V, dtype=dt, device=device)
    o, nq, gates = torch.empty(tt, H * V, device=device), torch.empty(tt, H, device=device), torch.empty(3, tt, H, device=device)
    state = 2 * H * K * (V + 1) * 4
    fl = 6.0 * tt * H * K * V
    t = timer(lambda: mem.recur(proj, out, ctx))
    add("matrix memory between its products (" + ("seq_mlstm_step_kernel" if tt == 1 else "gates + scan + read-out") + ")", t,
        tt * (2 * H * K + 2 * H * V) * 4 + tt * H * V * es + state, fl)
    qkv = torch.empty(tt, mem.o_g, device=device)
    w_a, w_n = torch.zeros(H, dtype=dt, device=device), torch.ones(H * V, dtype=dt, device=device)

    def scan(**kw):
        M._scan(ctx, q=M._p(qkv, mem.o_q), ldq=mem.o_g, k=M._p(qkv, mem.o_k), ldk=mem.o_g, v=M._p(qkv, mem.o_v), ldv=mem.o_g, q_mult=K ** -0.5, decay=M._p(gates[0]),
                ldd=H, per_channel=False, vscale=M._p(gates[1]), ldvs=H, state=ctx.state[mem.name + ".S"], out=M._p(o), ldo=H * V, heads=H, qk_heads=H, K=K, V=V, **kw)

    def cast():
        S.check(lib.b2l_seq_cast_f32(M._p(projb), ld, M._p(qkv), mem.o_g, tt, mem.o_g, act, st), "k")

    def decay():
        S.check(lib.b2l_seq_decay(M._p(projb, mem.o_i), ld, M._p(w_a), M._p(w_a), S.DECAY_EXP_SOFTPLUS, 0.0, M._p(gates[0]), M._p(gates[1]), tt, H, 1, act, st), "k")

    def norm():
        S.check(lib.b2l_seq_group_norm_gate(M._p(o), H * V, M._p(w_n), 0, M._p(projb, mem.o_g), ld, S.ACT_SIGMOID, 0, eps, 1.0, M._p(out), H * V, tt, H * V, V, act, st), "k")

    def like():
        cast()
        decay()
        scan()
        norm()

    add("  like: scalar-decay recurrence with the same state (cast + decay + seq_scan + grouped norm and gate)", timer(like),
        tt * (2 * H * K + 2 * H * V) * es + tt * H * V * es + state - 2 * H * K * 4, fl)
    if tt > 1:
        a = mem.args(proj, out, ctx)
        a.keep, a.put, a.floor, a.o, a.ldr, a.nq = M._p(gates[0]), M._p(gates[1]), M._p(gates[2]), M._p(o), H * V, M._p(nq)
        t = timer(lambda: S.check(lib.b2l_seq_mlstm_gates(C.byref(a), st), "k"))
        add("  seq_mlstm_gates_kernel", t, tt * H * (8 + 12))
        add("    like: seq_decay_kernel", timer(decay), tt * H * (es + 8))
        sb = tt * (2 * H * K + 2 * H * V) * 4 + state
        t = timer(lambda: scan(state_ones=ctx.state[mem.name + ".n"], out_ones=M._p(nq)))
        add("  seq_scan with the column of ones", t, sb, fl)
        add("    like: seq_scan", timer(scan), sb, fl)
        t = timer(lambda: S.check(lib.b2l_seq_mlstm_readout(C.byref(a), st), "k"))
        add("  seq_mlstm_readout_kernel", t, tt * H * V * (4 + 4 + es))
        add("    like: seq_group_norm_gate_kernel", timer(norm), tt * H * V * (4 + es + es))
    hh = torch.randn(tt, model.width, device=device).to(dt)
    wb = (mem.w_in.numel() + mem.w_o.numel()) * es
    add("MatrixMemoryMixer whole (2 products + recurrence)", timer(lambda: mem.forward(hh, ctx)), wb + 2 * tt * model.width * es + state, fl + 2.0 * tt * wb / es)
    return rows


def run_size(name: str, prompt: int, decode_steps: int, device, timer, peaks: dict) -> dict:
    import lit_llama_b200 as P
    from .lukupel import random_weights

    sz = SIZES[name]
    cfg = lukupel_config(**sz)
    model = P.Lukupel(P.LukupelConfig.from_dict(cfg), random_weights(cfg, device))
    engine = P.Engine(model, n_slots=2, prefill_chunk=prompt)
    toks = torch.randint(0, sz["vocab"], (prompt + decode_steps,), generator=torch.Generator().manual_seed(1)).tolist()

    def arm(params, t_pre, t_dec, weights, state):
        return {"params": params, "state_bytes_per_sequence": state, "prefill_tok_s": prompt / t_pre, "prefill_ms": t_pre * 1e3, "decode_tok_s": 1.0 / t_dec,
                "decode_us": t_dec * 1e6, "decode_frac_of_measured_hbm": (2 * weights + state) / t_dec / (peaks["hbm_gbs"] * 1e9)}

    t_pre, t_dec = zenasun_bench._throughput(engine, toks, prompt, decode_steps, device, timer)
    params, state = model.n_parameters(), engine.pool.bytes() // engine.pool.n_slots
    out = {"lukupel": arm(params, t_pre, t_dec, params, state)}          # the embedding table is the head: a token reads all of it
    out["kernels"] = kernel_table(model, engine, prompt, device, timer, peaks)
    del engine, model
    torch.cuda.empty_cache()

    # ---- the closest served family at the same width and depth
    lcfg = seq_bench.lugovik_config(**seq_bench.SIZES[name])
    lug = P.Lugovik(P.LugovikConfig.from_dict(lcfg), seq_bench.random_weights(lcfg, device), max_positions=prompt + decode_steps + 8)
    lengine = P.Engine(lug, n_slots=2, prefill_chunk=prompt)
    t_pre2, t_dec2 = zenasun_bench._throughput(lengine, toks, prompt, decode_steps, device, timer)
    lp = lug.n_parameters()
    out["lugovik"] = arm(lp, t_pre2, t_dec2, lp - lug.embed.numel(), lengine.pool.bytes() // 2)
    del lengine, lug
    torch.cuda.empty_cache()
    return out


def run(args, sizes: List[str]) -> dict:
    device = torch.device("cuda", 0)
    torch.cuda.set_device(device)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as f:
            peaks = json.load(f)
        peaks["source"] = "measured"
    except OSError:
        peaks = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0, "source": "fallback"}
    timer = seq_bench._Timer(device)
    out = {"metric": "lukupel_vs_lugovik_throughput", "unit": "tokens/s", "dtype": "bf16", "data": "synthetic (random weights)", "prompt": args.prompt,
           "decode_steps": args.decode_steps, "peaks": {k: peaks[k] for k in ("hbm_gbs", "bf16_tflops", "source")}, "l2": "flushed between timed iterations",
           "sizes": {}}
    t0 = time.time()
    for name in sizes:
        out["sizes"][name] = run_size(name, args.prompt, args.decode_steps, device, timer, peaks)
    out["seconds"] = round(time.time() - t0, 1)
    return out
