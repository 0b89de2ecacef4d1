"""Lukupel: a decoder-only language model whose sublayers read the residual stream itself and are normed on their way out:

    x = embed[token] * embedding.scale
    x <- x + residual_mult * norm1(mixer(x));   x <- x + residual_mult * norm2(ff(x))        per layer
    logits = logit_softcap * tanh(embed . norm(x) / logit_softcap)                            the table is the head, too

Norms are RMS norms with a weight.  The mixer of a layer is one of
    attention   `LocalAttention` inside chunks of mask.size positions counted from position 0: rotate-half rotation with
                linearly scaled frequencies, then every head of q and k divided by its root mean square; grouped kv heads
    mlstm       `MatrixMemoryMixer`: a matrix state per head with exponential gates
and its feed-forward, if it has one, is dense (`DenseMLP` with the square of relu).  A layer with "weights_of": j runs layer
j's weights (mixer, feed-forward and norms) once more with a cache or state of its own (`share_weights`).

Everything about a model comes from its config.json (`LukupelConfig`) and from the shapes of its tensors.  Tensor names:
`embed`, `l<i>.norm1|norm2`, `l<i>.mix.*`, `l<i>.mlp.up|down`, `final.norm`; linear weights are [out, in].  The residual
stream, norms, angles, attention scores and weights and everything of the recurrence are f32 in both number formats; what
a sublayer reads is the stream in the activation type.  What a sequence carries between steps is declared through
`state_specs()` and lives in a `SequenceStatePool`, so the `Engine` serves this model like any other."""
import json
import os
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

from . import _seqlib as S
from .mixers import DenseMLP, LocalAttention, MatrixMemoryMixer, StepContext, _p, linear_f32, share_weights
from .state import StateSpec

MIXERS = ("attention", "mlstm")
DEFAULT_MAX_POSITIONS = 4096       # of attention layers without chunks, when the caller names no limit


@dataclass
class LukupelConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    logit_softcap: float = 0.0     # 0: none
    layers: List[dict] = field(default_factory=list)

    @classmethod
    def from_dict(cls, d: dict) -> "LukupelConfig":
        if d.get("architecture") not in (None, "Lukupel"):
            raise ValueError(f"not a Lukupel configuration: architecture = {d.get('architecture')!r}")
        c = cls(vocab=int(d["vocab"]), width=int(d["width"]), eps=float(d["norm"]["eps"]),
                embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)), residual_mult=float(d.get("residual_mult", 1.0)),
                logit_softcap=float(d.get("logit_softcap") or 0.0), layers=list(d["layers"]))
        for i, layer in enumerate(c.layers):
            if layer["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown layer type {layer['type']!r}")
            mlp = layer.get("mlp")
            if mlp and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            own = c.layers[c.owner(i)]
            if any(k in layer and layer[k] != own.get(k) for k in ("type", "mixer", "mlp")):
                raise ValueError(f"layer {i} uses the weights of layer {c.owner(i)} but describes another layer")
        return c

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses: itself, or where its "weights_of" leads."""
        seen = set()
        while self.layers[i].get("weights_of") is not None:
            j = int(self.layers[i]["weights_of"])
            if i in seen or not 0 <= j < len(self.layers):
                raise ValueError(f"layer {i}: weights_of = {j} leads to no layer with weights of its own")
            seen.add(i)
            i = j
        return i

    @classmethod
    def from_json(cls, path: str) -> "LukupelConfig":
        with open(path) as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> dict:
        return {"architecture": "Lukupel", "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult, "logit_softcap": self.logit_softcap,
                "layers": self.layers}


def build_mixer(name: str, kind: str, c: dict, W: Dict[str, torch.Tensor], p: str, eps: float, max_positions: int):
    if kind == "attention":
        block = (c.get("mask") or {}).get("size")
        return LocalAttention(name, W, p, heads=c["heads"], kv_heads=c.get("kv_heads", c["heads"]), dim=c["dim"], vdim=c.get("vdim", c["dim"]),
                              scale=c["scale"], eps=eps, block=block, max_positions=max_positions, rot=c.get("rot"), norm_over="unit", gate=False)
    if kind == "mlstm":
        return MatrixMemoryMixer(name, W, p, heads=c["heads"], dim=c["dim"], vdim=c.get("vdim", c["dim"]), gate_cap=c["gate_cap"], eps=eps)
    raise ValueError(kind)


class _Layer:
    def __init__(self, i: int, spec: dict, W: Dict[str, torch.Tensor], eps: float, max_positions: int) -> None:
        p = f"l{i}."
        self.mixer = build_mixer(f"l{i}", spec["type"], spec["mixer"], W, p + "mix.", eps, max_positions)
        self.norm1 = W[p + "norm1"].contiguous()
        self.mlp: Optional[DenseMLP] = None
        self.norm2: Optional[torch.Tensor] = None
        if spec.get("mlp"):
            self.mlp = DenseMLP(W[p + "mlp.up"], W[p + "mlp.down"], act="relu2")
            self.norm2 = W[p + "norm2"].contiguous()

    def again(self, i: int) -> "_Layer":
        """Layer i with this layer's weights and a state of its own."""
        twin = _Layer.__new__(_Layer)
        twin.mixer, twin.norm1, twin.mlp, twin.norm2 = share_weights(self.mixer, f"l{i}"), self.norm1, self.mlp, self.norm2
        return twin


class Lukupel:
    """The model over a dict of device tensors in the activation dtype (torch.bfloat16, or torch.float32 for true
    32-bit arithmetic throughout).  `max_positions` bounds a sequence only when a layer attends without chunks."""

    graph_safe = True

    def __init__(self, config: LukupelConfig, weights: Dict[str, torch.Tensor], max_positions: int = 0) -> None:
        self.config = config
        self.embed = weights["embed"].contiguous()
        self.dtype, self.device = self.embed.dtype, self.embed.device
        if not self.embed.is_cuda:
            raise RuntimeError("Lukupel runs on CUDA only (no CPU fallback)")
        S.act_code(self.dtype)
        if tuple(self.embed.shape) != (config.vocab, config.width):
            raise ValueError(f"embed is {tuple(self.embed.shape)}, the configuration says {(config.vocab, config.width)}")
        self.vocab, self.width, self.eps = config.vocab, config.width, config.eps
        unbounded = any(l["type"] == "attention" and not (l["mixer"].get("mask") or {}).get("size") for l in config.layers)
        limit = int(max_positions) if max_positions and max_positions > 0 else DEFAULT_MAX_POSITIONS
        self.max_positions = limit if unbounded else 0
        own = {j: _Layer(j, config.layers[j], weights, config.eps, limit) for j in sorted({config.owner(i) for i in range(len(config.layers))})}
        self.layers: List[_Layer] = [own[i] if i in own else own[config.owner(i)].again(i) for i in range(len(config.layers))]
        self.final_norm = weights["final.norm"].contiguous()
        self.capture_layers: Optional[List[torch.Tensor]] = None     # set to [] to record the residual stream after every layer

    # ------------------------------------------------------------------ framework interface
    def state_specs(self) -> Dict[str, StateSpec]:
        out: Dict[str, StateSpec] = {}
        for layer in self.layers:
            out.update(layer.mixer.state_specs())
        return out

    def n_parameters(self) -> int:
        """Matrices, shared ones once."""
        seen = {t.data_ptr(): t.numel() for layer in self.layers for obj in (layer.mixer, layer.mlp) if obj is not None
                for t in vars(obj).values() if isinstance(t, torch.Tensor) and t.dim() >= 2}
        return self.embed.numel() + sum(seen.values())

    @torch.no_grad()
    def forward_portion(self, tokens: torch.Tensor, ctx: StepContext, want: Optional[torch.Tensor] = None) -> torch.Tensor:
        """tokens: device int32/int64 [T], the next T tokens of the sequence in ctx's slot.  want: device int32 indices
        into the portion (None = every token).  Returns f32 logits [len(want), vocab]."""
        lib, T, D, dev = S.lib(), ctx.T, self.width, self.device
        if self.dtype == torch.float32 and torch.backends.cuda.matmul.allow_tf32:
            raise RuntimeError("float32 models need true 32-bit products: torch.backends.cuda.matmul.allow_tf32 is on")
        x = torch.empty((T, D), dtype=torch.float32, device=dev)
        cast = self.dtype != torch.float32                        # what the sublayers read: the stream itself when it has their type
        h = torch.empty((T, D), dtype=self.dtype, device=dev) if cast else x
        S.check(lib.b2l_seq_embed(_p(tokens), int(tokens.dtype == torch.int64), _p(self.embed), ctx.act, self.config.embedding_scale, _p(x),
                                  _p(h) if cast else None, T, D, self.vocab, ctx.stream), "b2l_seq_embed")
        n = T if want is None else int(want.numel())
        hn = torch.empty((n, D), dtype=self.dtype, device=dev)
        steps = [(layer, sub) for layer in self.layers for sub in ((layer.mixer, layer.norm1), (layer.mlp, layer.norm2)) if sub[0] is not None]
        fuse_last = T == 1 and n == 1 and len(steps) > 0          # a single token: the last residual step and the final norm in one launch
        for k, (layer, (run, norm)) in enumerate(steps):
            y = run.forward(h, ctx)
            last = k + 1 == len(steps)
            w_next = self.final_norm if last and fuse_last else None
            h_out = hn if w_next is not None else (h if cast and not last else None)
            S.check(lib.b2l_seq_norm_add_norm(_p(y), _p(norm), self.eps, self.config.residual_mult, _p(x), _p(w_next), _p(h_out), T, D, ctx.act,
                                              ctx.stream), "b2l_seq_norm_add_norm")
            if self.capture_layers is not None and (last or steps[k + 1][0] is not layer):
                self.capture_layers.append(x.clone())
        if n == 0:
            return torch.empty((0, self.vocab), dtype=torch.float32, device=dev)
        if not fuse_last:
            S.check(lib.b2l_seq_rmsnorm(_p(x), _p(self.final_norm), self.eps, _p(hn), _p(want), n, D, ctx.act, ctx.stream), "b2l_seq_rmsnorm")
        logits = linear_f32(hn, self.embed)
        if self.config.logit_softcap > 0.0:
            S.check(lib.b2l_seq_softcap(_p(logits), logits.numel(), self.config.logit_softcap, ctx.stream), "b2l_seq_softcap")
        return logits


def load(model_dir: str, dtype: torch.dtype = torch.bfloat16, device: Optional[torch.device] = None, max_positions: int = 0) -> Lukupel:
    """config.json + model.safetensors of `model_dir` -> a model on `device`."""
    from .checkpoint_io import read_safetensors

    device = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
    config = LukupelConfig.from_json(os.path.join(model_dir, "config.json"))
    weights = read_safetensors(os.path.join(model_dir, "model.safetensors"), device=device, float_dtype=dtype)
    return Lukupel(config, weights, max_positions=max_positions)


def random_weights(cfg: dict, device, dtype: torch.dtype = torch.bfloat16, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random tensors with the family's names and shapes (projections ~ N(0, 1/in), norm weights around one, forget gates
    mostly open), for benchmarks, tests and smoke runs."""
    import math

    g = torch.Generator(device="cpu").manual_seed(seed)
    D, W = cfg["width"], {}

    def lin(o, i):
        return (torch.randn(o, i, generator=g) / math.sqrt(i)).to(device, dtype)

    def vec(n, mean=1.0, std=0.1):
        return (mean + std * torch.randn(n, generator=g)).to(device, dtype)

    W["embed"], W["final.norm"] = (torch.randn(cfg["vocab"], D, generator=g) / math.sqrt(D)).to(device, dtype), vec(D)
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m, c = f"l{i}.", f"l{i}.mix.", layer["mixer"]
        W[p + "norm1"] = vec(D)
        H, K = c["heads"], c["dim"]
        V = c.get("vdim", K)
        if layer["type"] == "attention":
            G = c.get("kv_heads", H)
            W[m + "q"], W[m + "k"], W[m + "v"], W[m + "o"] = lin(H * K, D), lin(G * K, D), lin(G * V, D), lin(D, H * V)
        else:
            W[m + "q"], W[m + "k"], W[m + "v"], W[m + "g"], W[m + "o"] = lin(H * K, D), lin(H * K, D), lin(H * V, D), lin(H * V, D), lin(D, H * V)
            W[m + "norm"], W[m + "i"], W[m + "i.b"], W[m + "f"], W[m + "f.b"] = vec(H * V), lin(H, D), vec(H, -1.0, 1.0), lin(H, D), vec(H, 4.0, 1.5)
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            W[p + "norm2"], W[p + "mlp.up"], W[p + "mlp.down"] = vec(D), lin(ff, D), lin(D, ff)
    return W
