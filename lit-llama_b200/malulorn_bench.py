"""Throughput of the Malulorn family beside the package's Zenasun family at equal width and number of layer runs
(`bench.py --family malulorn`).

Random weights, bf16, one sequence: prefill of a `prompt`-token prompt in one portion, then single-token decoding
through the engine (CUDA-graph replay).  The Zenasun arm is the closest served model: latent attention and routed experts on
an f32 residual stream, the same engine, state pool and library products.  A second table times the family's mechanisms
alone at the model's shapes with their algorithmic bytes and flops, each next to the like kernel of the framework's other
families run on operands of the same size.  CUDA events, warm-up, L2 flushed between iterations."""
import ctypes as C
import json
import os
import time
from typing import List

import torch

from . import seq_bench, zenasun_bench

SIZES = {
    # six layers, two of which run twice: eight layer runs, three of them latent attention
    "1k": dict(width=1024, heads=8, kv_heads=2, dim=128, l_heads=8, l_dim=128, l_rot=64, l_vdim=128, kv_rank=256, experts=20, top=4, ff=512, shared=512, vocab=32000),
    "2k": dict(width=2048, heads=16, kv_heads=4, dim=128, l_heads=16, l_dim=128, l_rot=64, l_vdim=128, kv_rank=512, experts=28, top=6, ff=1024, shared=1024, vocab=32000),
}


def malulorn_config(width, heads, kv_heads, dim, l_heads, l_dim, l_rot, l_vdim, kv_rank, experts, top, ff, shared, vocab, kinds="AALAAL", loop=(1, 3, 2)) -> dict:
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared}}
    att = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5, "q_temp": {"coef": 0.1, "every": 512}}
    lat = {"heads": l_heads, "dim": l_dim, "rot_dim": l_rot, "vdim": l_vdim, "kv_rank": kv_rank, "scale": (l_dim + l_rot) ** -0.5, "rot": {"base": 1e5, "dims": l_rot}}
    layers = [{"type": "attention", "mixer": att, "mlp": mlp} if k == "A" else {"type": "latent_attention", "mixer": lat, "mlp": mlp} for k in kinds]
    return {"architecture": "Malulorn", "vocab": vocab, "width": width, "norm": {"eps": 1e-6}, "loop": dict(zip(("start", "stop", "times"), loop)), "layers": layers}


def kernel_table(model, engine, T: int, device, timer, peaks: dict) -> List[dict]:
    """The family's mechanisms alone at this model's shapes, each followed by the like kernel: a T-token portion from
    position 0 and one token at position T - 1."""
    from . import _seqlib as S
    from . import mixers as M

    rows, hbm, es = [], peaks["hbm_gbs"] * 1e9, 2
    slot = engine.pool.acquire("kernels")
    D, dt, lib, eps, p = model.width, model.dtype, S.lib(), model.eps, M._p
    att = next(l.mixers[0] for l in model.layers if isinstance(l.mixers[0], M.LocalAttention))
    lat = next(l.mixers[0] for l in model.layers if isinstance(l.mixers[0], M.LatentAttention))
    moe = next(l.mlp for l in model.layers if l.mlp is not None)

    def add(name, tt, t, nbytes, flops=0.0, note=""):
        rows.append({"kernel": name, "tokens": int(tt), "us": t * 1e6, "GB_s": nbytes / t / 1e9, "frac_of_measured_hbm": nbytes / t / hbm,
                     "GFLOP_s": flops / t / 1e9, "note": note})

    full = M.StepContext(T, torch.tensor([slot, 0], dtype=torch.int32, device=device), engine.pool.tensors, dt, pos_hint=0, slot_hint=slot)
    for m in (att, lat):                                     # filled caches
        m.forward(torch.randn(T, D, device=device).to(dt), full)
    for tt, pos0 in ((T, 0), (1, T - 1)):
        meta = torch.tensor([slot, pos0], dtype=torch.int32, device=device)
        ctx = M.StepContext(tt, meta, engine.pool.tensors, dt, pos_hint=pos0 if tt > 1 else None, slot_hint=slot if tt > 1 else None)
        act, st = ctx.act, ctx.stream
        keys = (tt + 1) / 2 if tt > 1 else pos0 + 1
        hh, y = torch.randn(tt, D, device=device).to(dt), torch.randn(tt, D, device=device).to(dt)
        x, x2 = torch.randn(tt, D, device=device), torch.randn(tt, D, device=device)
        w, b, h = torch.ones(D, dtype=dt, device=device), torch.zeros(D, dtype=dt, device=device), torch.empty(tt, D, dtype=dt, device=device)
        # ---- residual step
        nb = tt * D * (es + 4 + 4 + es)

        def residual(**kw):
            a = S.ResidualArgs(x_in=p(x), x_out=p(x), eps=eps, norm_kind=S.NORM_LAYER, T=tt, D=D, act_dtype=act, **kw)
            return timer(lambda: S.check(lib.b2l_seq_residual_step(C.byref(a), st), "k"))

        add("seq_residual_step_kernel (sum, layer norm)", tt, residual(y1=p(y), w=p(w), b=p(b), h=p(h)), nb)
        t = timer(lambda: S.check(lib.b2l_seq_depth_step(p(y), None, p(x), p(x2), 1, None, p(x), p(w), p(b), S.NORM_LAYER, eps, p(h), tt, D, act, st), "k"))
        add("  like: seq_depth_step_kernel (sum, history entry, layer norm)", tt, t, nb + tt * D * 4)
        # ---- injection before a pass
        inj = model.inject
        base = inj.start(x, hh, ctx)
        if tt > M.FEW_TOKENS:
            pair = torch.empty(tt, 2 * D, dtype=dt, device=device)
            add("seq_residual_step_kernel (sum, split pair)", tt, residual(y1=p(y), split=p(pair)), tt * D * (es + 4 + 4 + 2 * es))
            add("seq_residual_step_kernel (product + base + step vector, layer norm)", tt,
                residual(base=p(base), vec=p(inj.step[0]), w=p(w), b=p(b), h=p(h)), tt * D * (4 + 4 + 4 + es))
            t = timer(lambda: inj.forward(x, pair, base, 0, ctx, norm=w, bias=b, kind="layer", eps=eps))
            add("LoopInjection whole (product of the pair + step)", tt, t, 2 * D * D * es + tt * D * (2 * es + 4 * 4 + es), 4.0 * tt * D * D)
        else:
            new = torch.empty(tt, D, device=device)
            t = timer(lambda: S.check(lib.b2l_seq_linear_few(p(inj.w_x), p(x), p(base), p(inj.step[0]), p(new), tt, D, D, act, st), "k"))
            add("seq_linear_few_kernel (W x + base + step vector, f32 rows)", tt, t, D * D * es)
            add("  like: library product of the same size (bf16 row)", tt, timer(lambda: M.linear(hh, inj.w_x)), D * D * es)
        # ---- attention
        H, G, K, V, ring, ld = att.H, att.G, att.K, att.V, att.ring, att.w_in.shape[0]
        proj = torch.randn(tt, ld, device=device).to(dt)
        q, kn = torch.empty(tt, H * K, device=device), torch.empty(tt, G * K, dtype=dt, device=device)
        wq, wk = torch.ones(H * K, dtype=dt, device=device), torch.ones(G * K, dtype=dt, device=device)
        freq = M.rope_frequencies(K, 1e4, None)[0].to(device)
        nb = tt * ((H + G) * K * es + H * K * 4 + G * K * es)
        for name, kw in (("seq_qkv_prep_kernel (query temperature)", dict(temp_coef=att.temp_coef, temp_every=att.temp_every)),
                         ("  like: seq_qkv_prep_kernel (norm over the row, rotation)", dict(q_norm=p(wq), k_norm=p(wk), whole_row=1, freq=p(freq), rot_dims=K))):
            a = S.QkvPrepArgs(proj=p(proj), ld=ld, q_off=att.o_q, k_off=att.o_k, v_off=att.o_v, eps=eps, rot_mult=1.0, meta=p(meta), q_out=p(q), k_out=p(kn), T=tt,
                              heads=H, kv_heads=G, K=K, V=V, act_dtype=act, **kw)
            add(name, tt, timer(lambda: S.check(lib.b2l_seq_qkv_prep(C.byref(a), st), "k")), nb)
        out = torch.empty(tt, H * V, dtype=dt, device=device)
        nb = tt * (H * K * 4 + G * (K + V) * es * 2 + H * V * es) + (keys * G * (K + V) * es if tt == 1 else 0)
        for name, kw in (("seq_block_attention (whole sequence, one in the denominator, gate per head) + append", dict(softcap=0.0)),
                         ("  like: the same with soft-capped scores", dict(softcap=50.0))):
            a2 = S.AttnArgs(q=p(q), k_new=p(kn), v_new=p(proj, att.o_v), ldv=ld, cache_k=p(ctx.state[att.name + ".k"]), cache_v=p(ctx.state[att.name + ".v"]),
                            meta=p(meta), gate=p(proj, att.o_g), ldg=ld, out=p(out), ldo=H * V, scale=att.scale, out_mult=1.0, has_sink=1, block=ring, T=tt, heads=H,
                            kv_heads=G, K=K, V=V, act_dtype=act, **kw)
            add(name, tt, timer(lambda: M.local_attention(a2, ctx)), nb, 2.0 * tt * H * keys * (K + V), f"f32 scores on CUDA cores, {keys:.0f} keys per query")
        wb = (att.w_in.numel() + att.w_o.numel()) * es
        add("LocalAttention whole (2 products + operands + attention)", tt, timer(lambda: att.forward(hh, ctx)), wb + 2 * tt * D * es,
            2.0 * tt * H * keys * (K + V) + 2.0 * tt * wb / es)
        rows += latent_rows(model, lat, ctx, tt, pos0, keys, timer, hbm)
        # ---- experts
        idx, wgt = torch.empty(tt, moe.top, dtype=torch.int32, device=device), torch.empty(tt, moe.top, device=device)
        z = torch.randn(tt, moe.n, device=device)
        for name, fn in (("seq_moe_route_kernel (softmax over the chosen logits)", S.SCORE_CHOSEN_SOFTMAX), ("  like: seq_moe_route_kernel (softmax over all)", S.SCORE_SOFTMAX)):
            t = timer(lambda: S.check(lib.b2l_seq_moe_route(p(z), moe.n, p(moe.correction), moe.n, 1, 1, moe.top, fn, 1, 1, 1.0, p(idx), p(wgt), tt, st), "k"))
            add(name, tt, t, tt * (moe.n * 4 + moe.top * 8))
        form = "device-indexed expert products" if tt <= moe.SMALL else "sort + gather + grouped library products + combine"
        per = 3 * moe.ff * D
        shared = moe.shared
        for name, sh in (("MoEFeedForward whole (router + experts + shared expert)", shared), ("  like: MoEFeedForward whole (router + experts)", None)):
            moe.shared = sh
            more = 3 * sh.ff * D if sh is not None else 0
            t = timer(lambda: moe.forward(hh, ctx))
            add(name, tt, t, (min(moe.E, tt * moe.top) * per + more) * es + 2 * tt * D * es, 2.0 * tt * (moe.top * per + more), form)
        moe.shared = shared
    engine.pool.release("kernels")
    return rows


def latent_rows(model, lat, ctx, tt: int, pos0: int, keys: float, timer, hbm: float) -> List[dict]:
    """Latent attention kernel by kernel, beside the kernels that low-rank queries and an ungated output take."""
    from . import _seqlib as S
    from . import mixers as M

    rows, lib, es, device, dt, eps, p = [], S.lib(), 2, model.device, model.dtype, model.eps, M._p
    H, rk, dr, dn, dv, dq, Kd = lat.H, lat.rk, lat.dr, lat.dn, lat.dv, lat.dn + lat.dr, lat.rk + lat.dr
    D, act, st, ld, n_keys = model.width, ctx.act, ctx.stream, lat.w_in.shape[0], pos0 + tt
    cache = ctx.state[lat.name + ".kv"]

    def add(name, t, nbytes, flops=0.0, note=""):
        rows.append({"kernel": name, "tokens": int(tt), "us": t * 1e6, "GB_s": nbytes / t / 1e9, "frac_of_measured_hbm": nbytes / t / hbm,
                     "GFLOP_s": flops / t / 1e9, "note": note})

    proj, hh = torch.randn(tt, ld, device=device), torch.randn(tt, D, device=device).to(dt)
    qb = torch.randn(tt, H * dq, device=device).to(dt)
    cq, wc = torch.empty(tt, dq, dtype=dt, device=device), torch.ones(dq, dtype=dt, device=device)
    q32, q_rot, q_lat = torch.empty(tt, H * dq, device=device), torch.empty(tt, H, dr, device=device), torch.empty(H, tt, rk, device=device)
    expanded = tt >= lat.expand_from
    shared_b = dict(key_b=p(cache, rk), ldkb=Kd, slot_stride_b=lat.max_positions * Kd, n_b=dr)

    def operands():
        a = S.LatentOperandsArgs(proj=p(proj), ld=ld, q_off=lat.o_q, kv_off=lat.o_kv, heads=H, dn=dn, dr=dr, rank=rk, w_kv=p(lat.kv_norm), freq=p(lat.freq),
                                 rot_dims=lat.rot_dims, interleaved=1, rot_mult=1.0, eps=eps, meta=p(ctx.meta), cache=p(cache), max_pos=lat.max_positions,
                                 q_full=p(q32) if expanded else None, q_rot=None if expanded else p(q_rot), w_uk=None if expanded else p(lat.w_uk),
                                 q_lat=None if expanded else p(q_lat), T=tt, act_dtype=act)
        S.check(lib.b2l_seq_latent_operands(C.byref(a), st), "k")

    def prep():
        S.check(lib.b2l_seq_latent_prep(p(proj), ld, lat.o_q, dq, p(wc), p(cq), lat.o_kv, rk, p(lat.kv_norm), dr, p(lat.freq), lat.rot_dims, 1, 1.0, eps,
                                        p(ctx.meta), p(cache), lat.max_positions, tt, act, st), "k")
        if expanded:
            lat._rope(qb, 0, dn, dq, q32, ctx)
        else:
            lat._rope(qb, dn, 0, dr, q_rot, ctx)
            torch.bmm(qb.view(tt, H, dq)[:, :, :dn].transpose(0, 1), lat.w_uk, out_dtype=torch.float32)

    wuk = 0 if expanded else lat.w_uk.numel() * es
    nb = tt * (rk + dr) * (4 + es) + wuk
    add("seq_latent_operands_kernel" + ("" if expanded else " (with W_uk)"), timer(operands), nb + tt * H * (dq * 4 + (dq if expanded else rk + dr) * 4),
        2.0 * tt * H * dn * rk if not expanded else 0.0)
    add("  like: seq_latent_prep + seq_rope" + ("" if expanded else " + batched library product"), timer(prep), nb + tt * (dq * 6 + H * (dq * es + (dq if expanded else rk + dr) * 4)))
    gate = dict(gate=p(proj, lat.o_g), ldg=ld)
    sink = torch.zeros(H, device=device)
    if expanded:
        kv = torch.randn(n_keys, H * (dv + dn), device=device).to(dt)
        out = torch.empty(tt, H * dv, dtype=dt, device=device)
        splits = lat._splits(ctx, 1)
        kw = dict(q_a=p(q32), ldqa_t=H * dq, ldqa_h=dq, q_b=p(q32, dn), ldqb_t=H * dq, ldqb_h=dq, key_a=p(kv), ldka=H * (dv + dn), hska=dv + dn, slot_stride_a=0,
                  n_a=dv + dn, score_off=dv, heads_per_group=1, **shared_b)
        fl, nb = 2.0 * tt * H * keys * (dq + dv), n_keys * (H * (dv + dn) + dr) * es + tt * H * (dq * 4 + dv * es)
        t = timer(lambda: lat._attend(ctx, out, dv, splits, **gate, **kw))
        add("seq_latent_attention_kernel (expanded form, gate per channel)", t, nb + tt * H * dv * 4, fl, f"f32 scores on CUDA cores, {splits} key split(s)")
        lat.sink = sink
        t = timer(lambda: lat._attend(ctx, out, dv, splits, **kw))
        lat.sink = None
        add("  like: the same with a sink per head, no gate", t, nb, fl)
    else:
        out = torch.empty(tt, H * dv, dtype=dt, device=device)
        o_lat = torch.empty(tt, H * rk, dtype=dt, device=device)
        splits = lat._splits(ctx, H)
        kw = dict(q_a=p(q_lat), ldqa_t=rk, ldqa_h=tt * rk, q_b=p(q_rot), ldqb_t=H * dr, ldqb_h=dr, key_a=p(cache), ldka=Kd, hska=0,
                  slot_stride_a=lat.max_positions * Kd, n_a=rk, score_off=0, heads_per_group=H, **shared_b)

        def tail():
            work = lat._attend(ctx, None, rk, splits, **kw)
            S.check(lib.b2l_seq_latent_up(p(work), None, p(lat.w_uv), gate["gate"], ld, p(out), H * dv, tt, H, rk, dv, splits, act, st), "k")

        def like():
            lat._attend(ctx, o_lat, rk, splits, **kw)
            torch.bmm(o_lat.view(tt, H, rk).transpose(0, 1), lat.w_uv.transpose(1, 2))

        fl, nb = 2.0 * tt * H * keys * (2 * rk + dr) + 2.0 * tt * H * rk * dv, n_keys * Kd * es + tt * H * (Kd * 4 + dv * es) + lat.w_uv.numel() * es
        add("seq_latent_attention_kernel + seq_latent_up_kernel (merge, W_uv, gate)", timer(tail), nb, fl, f"{splits} key split(s)")
        add("  like: seq_latent_attention_kernel + seq_latent_combine_kernel + batched library product, no gate", timer(like), nb, fl)
    wb = (lat.w_in.numel() + lat.w_uk.numel() + lat.w_uv.numel() + lat.w_o.numel()) * es
    add("LatentAttention whole", timer(lambda: lat.forward(hh, ctx)), wb + n_keys * Kd * es + 2 * tt * D * es, fl + 2.0 * tt * wb / es)
    return rows


def run_size(name: str, prompt: int, decode_steps: int, device, timer, peaks: dict) -> dict:
    import lit_llama_b200 as P
    from . import zenasun
    from .malulorn import random_weights

    sz = SIZES[name]
    cfg = malulorn_config(**sz)
    model = P.Malulorn(P.MalulornConfig.from_dict(cfg), random_weights(cfg, device), max_positions=prompt + decode_steps + 8)
    engine = P.Engine(model, n_slots=2, prefill_chunk=prompt)
    toks = torch.randint(0, sz["vocab"], (prompt + decode_steps,), generator=torch.Generator().manual_seed(1)).tolist()
    hbm = peaks["hbm_gbs"] * 1e9

    def arm(total, active, cache, t_pre, t_dec):
        return {"params": total, "active_params_per_token": active, "cache_bytes_at_prompt": cache, "prefill_tok_s": prompt / t_pre, "prefill_ms": t_pre * 1e3,
                "decode_tok_s": 1.0 / t_dec, "decode_us": t_dec * 1e6, "decode_frac_of_measured_hbm": (2 * active + cache) / t_dec / hbm}

    t_pre, t_dec = zenasun_bench._throughput(engine, toks, prompt, decode_steps, device, timer)
    total, active = model.n_parameters()
    out = {"malulorn": arm(total, active, engine.pool.bytes() / engine.pool.n_slots * prompt / model.max_positions, t_pre, t_dec)}
    out["malulorn"]["layer_runs"] = len(model.runs)
    out["kernels"] = kernel_table(model, engine, prompt, device, timer, peaks)
    del engine, model
    torch.cuda.empty_cache()

    # ---- the closest served family at the same width and number of layer runs
    zsz = zenasun_bench.SIZES[name]
    zcfg = zenasun_bench.zenasun_config(**zsz)
    zen = P.Zenasun(P.ZenasunConfig.from_dict(zcfg), zenasun.random_weights(zcfg, device), max_positions=prompt + decode_steps + 8)
    zengine = P.Engine(zen, n_slots=2, prefill_chunk=prompt)
    t_pre2, t_dec2 = zenasun_bench._throughput(zengine, toks, prompt, decode_steps, device, timer)
    moe, params = zen.layers[0].mlp, zen.n_parameters()
    zactive = params - sum(1 for l in zen.layers if l.mlp is not None) * (moe.E - moe.top) * 3 * moe.ff * zsz["width"]
    cache = sum(t[0].numel() * t.element_size() * (prompt / zen.max_positions if k.endswith(".kv") else 1.0) for k, t in zengine.pool.tensors.items())
    out["zenasun"] = arm(params, zactive, cache, t_pre2, t_dec2)
    del zengine, zen
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
    out = {"metric": "malulorn_vs_zenasun_throughput", "unit": "tokens/s", "dtype": "bf16", "data": "synthetic (random weights)", "prompt": args.prompt,
           "decode_steps": args.decode_steps, "peaks": {k: peaks[k] for k in ("hbm_gbs", "bf16_tflops", "source")}, "l2": "flushed between timed iterations",
           "sizes": {}}
    t0 = time.time()
    for name in sizes:
        out["sizes"][name] = run_size(name, args.prompt, args.decode_steps, device, timer, peaks)
    out["seconds"] = round(time.time() - t0, 1)
    return out
