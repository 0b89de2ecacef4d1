"""Malulorn: a decoder-only language model that runs a stretch of its layers several times.

    x = x0 = embed[token]
    x <- x + mixer(norm1(x));   x <- x + experts(norm2(x))         per layer run (a layer may have no feed-forward)
    x <- W_in [x; x0] + step[t]                                    before pass t = 0, 1, ... of layers loop.start .. loop.stop - 1,
                                                                   which run loop.times times with the same weights
    logits = head(norm(x))

Norms are layer norms with a weight and a bias.  The mixer of a layer is one of
    attention         `LocalAttention` over the whole sequence: no norms, no rotation, a query temperature that grows with
                      the position, grouped kv heads, a one in the softmax denominator, a sigmoid gate per head
    latent_attention  `LatentAttention`: direct queries, keys and values from a cached latent, interleaved rotation of the shared
                      key part, ordinary softmax, a sigmoid gate per channel
and its feed-forward `MoEFeedForward`: the `top` largest router logits (with a bias), softmax over them, a shared expert.
Every pass of a looped layer has a cache of its own (`share_weights`); what stands before a pass is `LoopInjection`.

Everything about a model comes from its config.json (`MalulornConfig`) and from the shapes of its tensors.  Tensor names:
`embed`, `loop.in|step`, `l<i>.norm1|norm2[.b]`, `l<i>.mix.*`, `l<i>.mlp.router[.b]|shared.*|e<k>.gate|up|down`,
`final.norm[.b]`, `head`; linear weights are [out, in].  The residual stream, norms, positions and angles, attention scores
and weights and the router are f32 in both number formats.  What a sequence carries between steps is declared through
`state_specs()` and lives in a `SequenceStatePool`, so the `Engine` serves this model like any other."""
import json
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

from . import _seqlib as S
from .mixers import (FEW_TOKENS, LatentAttention, LocalAttention, LoopInjection, MoEFeedForward, StepContext, _p, linear_f32, norm_rows, residual_step,
                     share_weights)
from .state import StateSpec

MIXERS = ("attention", "latent_attention")
DEFAULT_MAX_POSITIONS = 4096


@dataclass
class MalulornConfig:
    vocab: int
    width: int
    eps: float
    layers: List[dict] = field(default_factory=list)
    loop: Optional[dict] = None        # {"start", "stop", "times"}

    @classmethod
    def from_dict(cls, d: dict) -> "MalulornConfig":
        if d.get("architecture") not in (None, "Malulorn"):
            raise ValueError(f"not a Malulorn configuration: architecture = {d.get('architecture')!r}")
        layers, loop = list(d["layers"]), d.get("loop")
        for i, layer in enumerate(layers):
            if layer["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown layer type {layer['type']!r}")
            mlp = layer.get("mlp")
            if mlp and mlp.get("kind", "moe") != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            rot = layer["mixer"].get("rot")
            if layer["type"] == "latent_attention" and rot and int(rot.get("dims", layer["mixer"]["rot_dim"])) != int(layer["mixer"]["rot_dim"]):
                raise ValueError(f"layer {i}: the whole rotated part of {layer['mixer']['rot_dim']} entries turns, not {rot['dims']} of it")
        if loop:
            loop = {k: int(loop[k]) for k in ("start", "stop", "times")}
            if not (0 <= loop["start"] < loop["stop"] <= len(layers) and loop["times"] >= 1):
                raise ValueError(f"loop {loop} does not name a stretch of the {len(layers)} layers")
        return cls(vocab=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]), layers=layers, loop=loop or None)

    @classmethod
    def from_json(cls, path: str) -> "MalulornConfig":
        with open(path) as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> dict:
        return {"architecture": "Malulorn", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": self.layers, "loop": self.loop}

    def runs(self) -> List[Tuple[int, int, bool]]:
        """The layer runs of a token in order: (layer, pass, whether the injection of that pass stands before it)."""
        if not self.loop:
            return [(i, 0, False) for i in range(len(self.layers))]
        a, b, n = self.loop["start"], self.loop["stop"], self.loop["times"]
        return [(i, 0, False) for i in range(a)] + [(i, t, i == a) for t in range(n) for i in range(a, b)] + [(i, 0, False) for i in range(b, len(self.layers))]


def build_mixer(name: str, kind: str, c: dict, W: Dict[str, torch.Tensor], p: str, eps: float, max_positions: int):
    if kind == "attention":
        return LocalAttention(name, W, p, heads=c["heads"], kv_heads=c.get("kv_heads", c["heads"]), dim=c["dim"], vdim=c.get("vdim", c["dim"]),
                              scale=c["scale"], eps=eps, max_positions=max_positions, rot=None, norm_over="head", gate="head", sink=True,
                              q_temp=c.get("q_temp"))
    if kind == "latent_attention":
        rot = c.get("rot") or {}
        return LatentAttention(name, W, p, heads=c["heads"], dim=c["dim"], rot_dim=c.get("rot_dim", 0), vdim=c["vdim"], q_rank=None, kv_rank=c["kv_rank"],
                               scale=c["scale"], eps=eps, rot=dict(rot, dims=c.get("rot_dim", 0)) if rot else None, max_positions=max_positions,
                               interleaved=True, gate=True)
    raise ValueError(kind)


def build_experts(m: dict, W: Dict[str, torch.Tensor], p: str) -> MoEFeedForward:
    r = m["router"]
    return MoEFeedForward(W, p, experts=r["experts"], identity=0, top=r["top"], groups=1, keep=1, ff=m["expert"]["ff"], act="silu",
                          score="chosen_softmax", shared_ff=(m.get("shared") or {}).get("ff", 0))


class _Layer:
    """A layer's weights; `mixers[t]` is its mixer with the cache of pass t."""

    def __init__(self, i: int, spec: dict, W: Dict[str, torch.Tensor], eps: float, max_positions: int, times: int) -> None:
        p = f"l{i}."
        first = build_mixer(f"l{i}", spec["type"], spec["mixer"], W, p + "mix.", eps, max_positions)
        self.mixers = [first] + [share_weights(first, f"l{i}.pass{t}") for t in range(1, times)]
        self.norm1 = (W[p + "norm1"].contiguous(), W[p + "norm1.b"].contiguous())
        self.mlp: Optional[MoEFeedForward] = None
        self.norm2 = None
        if spec.get("mlp"):
            self.mlp = build_experts(spec["mlp"], W, p + "mlp.")
            self.norm2 = (W[p + "norm2"].contiguous(), W[p + "norm2.b"].contiguous())


class Malulorn:
    """The model over a dict of device tensors in the activation dtype (torch.bfloat16, or torch.float32 for true
    32-bit arithmetic throughout).  `max_positions`: the most positions a sequence may reach (the attention layers cache
    every position)."""

    graph_safe = True

    def __init__(self, config: MalulornConfig, weights: Dict[str, torch.Tensor], max_positions: int = 0) -> None:
        self.config = config
        self.embed = weights["embed"].contiguous()
        self.dtype, self.device = self.embed.dtype, self.embed.device
        if not self.embed.is_cuda:
            raise RuntimeError("Malulorn runs on CUDA only (no CPU fallback)")
        S.act_code(self.dtype)
        if tuple(self.embed.shape) != (config.vocab, config.width):
            raise ValueError(f"embed is {tuple(self.embed.shape)}, the configuration says {(config.vocab, config.width)}")
        self.vocab, self.width, self.eps = config.vocab, config.width, config.eps
        self.max_positions = int(max_positions) if max_positions and max_positions > 0 else DEFAULT_MAX_POSITIONS
        self.runs = config.runs()
        times = [1 + max((t for j, t, _ in self.runs if j == i), default=0) for i in range(len(config.layers))]
        self.layers = [_Layer(i, spec, weights, config.eps, self.max_positions, times[i]) for i, spec in enumerate(config.layers)]
        self.inject = LoopInjection(weights["loop.in"], weights["loop.step"]) if config.loop else None
        if self.inject is not None and (self.inject.width, self.inject.times) != (config.width, config.loop["times"]):
            raise ValueError(f"loop tensors for width {self.inject.width} and {self.inject.times} passes, the configuration says {config.width} and {config.loop}")
        self.final_norm = (weights["final.norm"].contiguous(), weights["final.norm.b"].contiguous())
        self.head = weights["head"].contiguous()
        self.capture_layers: Optional[List[torch.Tensor]] = None     # set to [] to record the residual stream after every layer run

    # ------------------------------------------------------------------ framework interface
    def state_specs(self) -> Dict[str, StateSpec]:
        out: Dict[str, StateSpec] = {}
        for layer in self.layers:
            for m in layer.mixers:
                out.update(m.state_specs())
        return out

    def n_parameters(self) -> Tuple[int, int]:
        """(all parameters, parameters that a token reads, those of looped layers once per pass): matrices only."""
        total = active = self.embed.numel() + self.head.numel()
        active -= self.embed.numel()                                 # one row of it
        for layer in self.layers:
            m, f = layer.mixers[0], layer.mlp
            n = sum(v.numel() for k, v in vars(m).items() if isinstance(v, torch.Tensor) and v.dim() >= 2 and k != "w_expand")
            used = n
            if f is not None:
                per = (f.w_gu.numel() + f.w_down.numel()) // max(f.E, 1)
                rest = f.w_router.numel() + (f.shared.w_in.numel() + f.shared.w_down.numel() if f.shared is not None else 0)
                n, used = n + per * f.E + rest, used + per * f.top + rest
            total, active = total + n, active + used * len(layer.mixers)
        if self.inject is not None:
            total, active = total + 2 * self.width ** 2, active + (1 + self.inject.times) * self.width ** 2
        return total, active

    @torch.no_grad()
    def forward_portion(self, tokens: torch.Tensor, ctx: StepContext, want: Optional[torch.Tensor] = None) -> torch.Tensor:
        """tokens: device int32/int64 [T], the next T tokens of the sequence in ctx's slot.  want: device int32 indices
        into the portion (None = every token).  Returns f32 logits [len(want), vocab]."""
        T, D, dev = ctx.T, self.width, self.device
        if torch.backends.cuda.matmul.allow_tf32:
            raise RuntimeError("32-bit products of this model (router, float32 mode) must be true f32: torch.backends.cuda.matmul.allow_tf32 is on")
        n = T if want is None else int(want.numel())
        x0 = torch.empty((T, D), dtype=torch.float32, device=dev)
        h0 = torch.empty((T, D), dtype=self.dtype, device=dev) if self.inject is not None and T > FEW_TOKENS else None
        S.check(S.lib().b2l_seq_embed(_p(tokens), int(tokens.dtype == torch.int64), _p(self.embed), ctx.act, 1.0, _p(x0), _p(h0), T, D, self.vocab, ctx.stream),
                "b2l_seq_embed")
        base = self.inject.start(x0, h0, ctx) if self.inject is not None else None
        norm = dict(kind="layer", eps=self.eps)
        x, split, h = x0, None, None                # the stream, its split form before a pass, the next sublayer's normed input
        buf = torch.empty((T, D), dtype=torch.float32, device=dev)    # x0 stays as it is while the stream moves on
        if self.inject is not None and self.runs[0][2] and self.inject.wants_split(ctx):
            split = residual_step(x, None, ctx, split=True)
        elif self.runs and not self.runs[0][2]:
            h = norm_rows(x, *self.layers[self.runs[0][0]].norm1, ctx=ctx, **norm)
        hn = None
        for r, (i, t, injected) in enumerate(self.runs):
            layer = self.layers[i]
            if injected:
                x, h = self.inject.forward(x, split, base, t, ctx, norm=layer.norm1[0], bias=layer.norm1[1], **norm)
                split = None
            y = layer.mixers[t].forward(h, ctx)
            out = buf if x is x0 else x
            if layer.mlp is not None:
                h = residual_step(x, out, ctx, y1=y, norm=layer.norm2[0], bias=layer.norm2[1], **norm)
                x = out
                y = layer.mlp.forward(h, ctx)
            if r + 1 < len(self.runs):              # the layer's last sum, with what reads the stream next
                j, _, inj = self.runs[r + 1]
                if not inj:
                    h = residual_step(x, out, ctx, y1=y, norm=self.layers[j].norm1[0], bias=self.layers[j].norm1[1], **norm)
                else:
                    split = residual_step(x, out, ctx, y1=y, split=self.inject.wants_split(ctx))
            elif T == 1 and n == 1:                 # a single token: the last sum and the final norm in one launch
                hn = residual_step(x, out, ctx, y1=y, norm=self.final_norm[0], bias=self.final_norm[1], **norm)
            else:
                residual_step(x, out, ctx, y1=y)
            x = out
            if self.capture_layers is not None:
                self.capture_layers.append(x.clone())
        if n == 0:
            return torch.empty((0, self.vocab), dtype=torch.float32, device=dev)
        if hn is None:
            hn = norm_rows(x, *self.final_norm, ctx=ctx, rows=want, n_rows=n, **norm)
        return linear_f32(hn, self.head)


def load(model_dir: str, dtype: torch.dtype = torch.bfloat16, device: Optional[torch.device] = None, max_positions: int = 0) -> Malulorn:
    """config.json + model.safetensors of `model_dir` -> a model on `device`."""
    from .checkpoint_io import read_safetensors

    device = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
    config = MalulornConfig.from_json(os.path.join(model_dir, "config.json"))
    weights = read_safetensors(os.path.join(model_dir, "model.safetensors"), device=device, float_dtype=dtype)
    return Malulorn(config, weights, max_positions=max_positions)


def random_weights(cfg: dict, device, dtype: torch.dtype = torch.bfloat16, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random tensors with the family's names and shapes (projections ~ N(0, 1/in), norm weights around one), for
    benchmarks, tests and smoke runs."""
    import math

    g = torch.Generator(device="cpu").manual_seed(seed)
    D, W = cfg["width"], {}

    def lin(o, i, gain=1.0):
        return (gain * torch.randn(o, i, generator=g) / math.sqrt(i)).to(device, dtype)

    def vec(n, mean=0.0, std=0.1):
        return (mean + std * torch.randn(n, generator=g)).to(device, dtype)

    W["embed"], W["head"] = torch.randn(cfg["vocab"], D, generator=g).to(device, dtype), lin(cfg["vocab"], D)
    W["final.norm"], W["final.norm.b"] = vec(D, 1.0), vec(D)
    if cfg.get("loop"):
        W["loop.in"], W["loop.step"] = lin(D, 2 * D), (0.3 * torch.randn(cfg["loop"]["times"], D, generator=g)).to(device, dtype)
    for i, layer in enumerate(cfg["layers"]):
        p, m, c = f"l{i}.", f"l{i}.mix.", layer["mixer"]
        W[p + "norm1"], W[p + "norm1.b"] = vec(D, 1.0), vec(D)
        if layer["type"] == "attention":
            H, G, K, V = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
            W[m + "q"], W[m + "k"], W[m + "v"], W[m + "g"], W[m + "o"] = lin(H * K, D), lin(G * K, D), lin(G * V, D), lin(H, D), lin(D, H * V)
        else:
            H, dn, dr, dv, rk = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
            W[m + "q"], W[m + "dkv"], W[m + "dkv.norm"] = lin(H * (dn + dr), D), lin(rk + dr, D), vec(rk, 1.0)
            W[m + "uk"], W[m + "uv"], W[m + "g"], W[m + "o"] = lin(H * dn, rk), lin(H * dv, rk), lin(H * dv, D), lin(D, H * dv)
        f = layer.get("mlp")
        if f:
            W[p + "norm2"], W[p + "norm2.b"] = vec(D, 1.0), vec(D)
            W[p + "mlp.router"], W[p + "mlp.router.b"] = lin(f["router"]["experts"], D, 2.0), vec(f["router"]["experts"], 0.0, 0.3)
            kinds = [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])] + ([("shared", f["shared"]["ff"])] if f.get("shared") else [])
            for name, ff in kinds:
                q = f"{p}mlp.{name}."
                W[q + "gate"], W[q + "up"], W[q + "down"] = lin(ff, D), lin(ff, D), lin(D, ff)
    return W
