"""Sequence-mixer mechanisms over libb200seq (include/b2l_seq.h), each usable by any model: its sizes and
constants are constructor parameters.

    GatedMLP             act(W_gate h) * (W_up h) -> W_down, both halves from one product
    ChannelDeltaMixer    gated delta rule with one decay per key channel, short convolutions on q / k / v
    BlockSinkAttention   block-local causal softmax attention: q/k norm, partial rotation (YaRN-scaled), soft-capped
                         scores, a sink in the denominator, grouped kv heads, per-head sigmoid output gate, ring cache
    GatedLinearAttention S_t = diag(alpha_t) S_(t-1) + k_t v_t^T with a low-rank decay projection
    ParallelMixer        two mixers on the same input, one output product over their concatenated read-outs
    Mamba2Mixer          state-space duality layer: scalar decay per head, convolution on x | B | C, gated grouped norm
    LatentAttention      causal softmax attention whose keys and values are linear images of one cached latent per position
                         (+ one rotated key part shared by the heads), low-rank or direct queries, a learned sink per head,
                         an optional sigmoid gate per output channel
    RetentionMixer       linear attention with a fixed decay per head, rotated q / k, per-head unit-RMS read-out, silu gate
    MoEFeedForward       routed gated experts: softmax or sigmoid scores or a softmax over the chosen logits, selection or logit
                         bias, expert groups, top-k, identity experts, a shared expert, weights renormalised or not, on an
                         expert's output or on its input, clamped gated unit
    LocalAttention       causal softmax attention over the last `window` positions (SlidingWindowAttention) or inside blocks:
                         q/k norm over the whole projection or per head before the rotation, or weightless per head after it,
                         partial rotation, a query temperature by position, grouped kv heads, values mixed with an earlier
                         layer's, an optional one in the softmax denominator, an optional sigmoid gate per head or per output
                         channel, ring cache of one window or block
    PairHashEmbedding    token embedding plus a hashed (previous token, token) embedding, into several residual streams
    HyperConnection      one sublayer's read weights, stream-mixing matrix and write weights over several residual streams
    DenseMLP             W_down act(W_up h) without a gate: gelu_tanh, silu, relu2, or xIELU with its two learned numbers
    DifferentialAttention  causal softmax attention with two score maps per head over the same values, combined as
                         a0 - lambda a1 and divided by its root mean square; biases and short convolutions on q / k / v,
                         interleaved rotation, grouped kv heads, keys and values of its own or of an earlier layer
    MinGRUMixer          S_t = (1 - z_t) S_(t-1) + z_t c_t per channel with gates that read only the current token, silu gate
    DepthAverage         the residual step of layers whose input is a learned average over all earlier layers' results
    residual_step        x + results (+ a vector, + an f32 row), fused with the next norm or with the operand of a product on x
    LoopInjection        what a looped stretch of layers reads: x <- W [x; embedding output] + a vector of the pass
    MatrixMemoryMixer    mLSTM: a matrix state per head with exponential input gates, sigmoid forget gates, a normaliser and a
                         running maximum; per-head unit-RMS read-out, one weight, a sigmoid gate per channel
    share_weights        the same mixer over the same weights with a state of its own (a layer that runs again)

A mixer is built from a dict of weight tensors (`from_weights`) and runs one portion of one sequence:
`forward(h, ctx)` with h [T, width] in the model's activation dtype.  Products go through torch (cuBLAS), as the
dense linears of the package's LLaMA do; everything else is a kernel of libb200seq.  What a mixer carries between
tokens is declared by `state_specs()` and lives in a `SequenceStatePool`.  CUDA only; no CPU fallback."""
import copy
import ctypes as C
import math
from typing import Dict, List, Optional, Tuple

import torch
import torch.nn.functional as F

from . import _seqlib as S
from .state import StateSpec


class StepContext:
    """One portion of one sequence: T tokens, the device pair {slot, first position} and the slot pool's tensors.
    `pos_hint` / `slot_hint` are the first position and the slot as the host knows them (None inside a captured step,
    which must not depend on them): kernels never read them, they size grids and pick between equivalent forms."""

    def __init__(self, T: int, meta: torch.Tensor, state: Dict[str, torch.Tensor], dtype: torch.dtype, pos_hint: Optional[int] = None,
                 slot_hint: Optional[int] = None) -> None:
        self.T, self.meta, self.state, self.dtype, self.pos_hint, self.slot_hint = T, meta, state, dtype, pos_hint, slot_hint
        self.act = S.act_code(dtype)
        self.shared: Dict[str, object] = {}      # what one layer of this step hands to later ones (values of an earlier layer, ...)

    @property
    def stream(self) -> int:
        """The current CUDA stream at the time of each launch (the capturing stream while a graph is recorded)."""
        return S.stream_ptr()


def _p(t: Optional[torch.Tensor], offset: int = 0) -> Optional[int]:
    """Device address of element `offset` of a tensor's storage view."""
    if t is None:
        return None
    return S.ptr(t) + offset * t.element_size()


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def stack_rows(parts: List[torch.Tensor]) -> Tuple[torch.Tensor, List[int]]:
    """Linear weights that read the same input, stacked into one [sum, in] matrix.  Every part starts at a multiple
    of 8 rows (zero rows between), so each part's columns of the product start 16-byte aligned.  Returns the matrix
    and the first row of every part."""
    offs, rows, at = [], [], 0
    for w in parts:
        offs.append(at)
        rows.append(w)
        gap = pad8(w.shape[0]) - w.shape[0]
        if gap:
            rows.append(w.new_zeros((gap,) + tuple(w.shape[1:])))
        at += pad8(w.shape[0])
    return torch.cat(rows, dim=0).contiguous(), offs


def share_weights(mixer, name: str):
    """`mixer` over the same weight tensors with a state of its own under `name`, for a layer that uses another layer's
    weights.  Mixers find their state by their name and hold everything else in tensors they never write."""
    if hasattr(mixer, "branches"):
        raise ValueError("a mixer of several branches has several states: share its branches one by one")
    twin = copy.copy(mixer)
    twin.name = name
    return twin


FEW_TOKENS = 4          # up to this many tokens a mechanism may run its products in its own kernels, without the library


def linear(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return F.linear(x, w)


def linear_f32(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x W^T with the f32 accumulator kept (bf16 operands), or the plain f32 product."""
    if x.dtype == torch.float32:
        return F.linear(x, w)
    return torch.mm(x, w.t(), out_dtype=torch.float32)


# ------------------------------------------------------------------------------------------------ feed-forward
class GatedMLP:
    ACTS = {"gelu_tanh": S.ACT_GELU_TANH, "silu": S.ACT_SILU, "clamped_swish": S.ACT_CLAMPED_SWISH}

    def __init__(self, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor, act: str = "gelu_tanh", limit: float = 0.0) -> None:
        self.ff = gate.shape[0]
        self.w_in = torch.cat([gate, up], dim=0).contiguous()
        self.w_down = down.contiguous()
        self.act, self.limit = self.ACTS[act], float(limit)

    def state_specs(self) -> Dict[str, StateSpec]:
        return {}

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        gu = linear(h, self.w_in)
        mid = torch.empty((ctx.T, self.ff), dtype=h.dtype, device=h.device)
        S.check(S.lib().b2l_seq_gated_act(_p(gu), 2 * self.ff, _p(mid), ctx.T, self.ff, self.act, self.limit, ctx.act, ctx.stream),
                "b2l_seq_gated_act")
        return linear(mid, self.w_down)


class DenseMLP:
    """W_down act(W_up h), no gate.  act: gelu_tanh, silu, sigmoid, relu2 (max(z, 0)^2), or xIELU with its two learned numbers `params` = (p, q):
    softplus(p) z^2 + z/2 for z > 0, (1/2 + softplus(q)) (exp(z) - 1 - z) + z/2 otherwise."""

    ACTS = {"gelu_tanh": S.ACT_GELU_TANH, "silu": S.ACT_SILU, "sigmoid": S.ACT_SIGMOID, "relu2": S.ACT_RELU2, "xielu": S.ACT_XIELU}

    def __init__(self, up: torch.Tensor, down: torch.Tensor, act: str = "gelu_tanh", params: Optional[torch.Tensor] = None) -> None:
        if act not in self.ACTS:
            raise ValueError(f"dense feed-forward: unknown activation {act!r}")
        self.ff = up.shape[0]
        self.w_up, self.w_down = up.contiguous(), down.contiguous()
        self.act = self.ACTS[act]
        self.coef = None
        if self.act == S.ACT_XIELU:
            if params is None or params.numel() != 2:
                raise ValueError("dense feed-forward: xIELU needs its two numbers")
            pq = params.detach().reshape(-1).double().cpu()
            sp = torch.nn.functional.softplus(pq)                       # the two coefficients, once, in 64-bit; kept as f32
            self.coef = torch.stack([sp[0], 0.5 + sp[1]]).to(torch.float32).to(up.device)

    def state_specs(self) -> Dict[str, StateSpec]:
        return {}

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        u = linear(h, self.w_up)
        S.check(S.lib().b2l_seq_unary_act(_p(u), self.ff, _p(u), self.ff, ctx.T, self.ff, self.act, _p(self.coef), ctx.act, ctx.stream),
                "b2l_seq_unary_act")                      # in place: every element is read and written by the same thread
        return linear(u, self.w_down)


# ------------------------------------------------------------------------------------------------ recurrences
def _scan(ctx: StepContext, *, q, ldq, k, ldk, v, ldv, q_mult, decay, ldd, per_channel, state, out, ldo, heads, qk_heads,
          K, V, beta=None, ldb=0, vscale=None, ldvs=0, skip=None, state_ones=None, out_ones=None) -> None:
    lib = S.lib()
    n_chunks = lib.b2l_seq_scan_chunks(ctx.T, int(beta is not None))
    ws = wd = None
    if n_chunks > 1:      # long portion, no delta rule: chunks in parallel (local states, combine, outputs)
        ws = torch.empty((n_chunks, heads, V + int(state_ones is not None), K), dtype=torch.float32, device=state.device)
        wd = torch.empty((n_chunks, heads, K if per_channel else 1), dtype=torch.float32, device=state.device)
    a = S.ScanArgs(q=q, ldq=ldq, k=k, ldk=ldk, v=v, ldv=ldv, q_mult=float(q_mult), decay=decay, ldd=ldd,
                   decay_per_channel=int(per_channel), beta=beta, ldb=ldb, delta=int(beta is not None), vscale=vscale, ldvs=ldvs,
                   skip=skip, state=_p(state), meta=_p(ctx.meta), out=out, ldo=ldo, T=ctx.T, heads=heads, qk_heads=qk_heads, K=K, V=V,
                   act_dtype=ctx.act, work_state=_p(ws), work_decay=_p(wd), n_chunks=n_chunks, ones=int(state_ones is not None), state_ones=_p(state_ones),
                   out_ones=out_ones)
    S.check(lib.b2l_seq_scan(C.byref(a), ctx.stream), "b2l_seq_scan")


class ChannelDeltaMixer:
    """Gated delta rule, one decay per head and key channel.

        q, k, v = silu(conv(W h)); q, k unit vectors per head (q times dim^-1/2); beta = sigmoid(W_b h)
        g = exp(-exp(A_log) softplus(W_a2 W_a1 h + dt_bias))              [heads x dim]
        S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
        y = W_o (o / rms(o) * w_norm * sigmoid(W_g2 W_g1 h))
    State per sequence: S (f32, heads x vdim x dim) and the last taps-1 inputs of the convolutions."""

    def __init__(self, name: str, W: Dict[str, torch.Tensor], p: str, *, heads: int, kv_heads: int, dim: int, vdim: int, conv: int,
                 eps: float, unit_eps: float = 1e-6) -> None:
        self.name, self.H, self.G, self.K, self.V, self.taps, self.eps, self.unit_eps = name, heads, kv_heads, dim, vdim, conv, eps, unit_eps
        parts = [W[p + "q"], W[p + "k"], W[p + "v"], W[p + "b"], W[p + "a1"], W[p + "g1"]]
        self.w_in, (self.o_q, self.o_k, self.o_v, self.o_b, self.o_a1, self.o_g1) = stack_rows(parts)
        self.n_in = self.w_in.shape[0]
        self.rank_a, self.rank_g = W[p + "a1"].shape[0], W[p + "g1"].shape[0]
        self.C = self.o_b                                  # conv channels: q | k | v with their alignment gaps
        self.w_conv, _ = stack_rows([W[p + "q.conv"], W[p + "k.conv"], W[p + "v.conv"]])
        assert self.w_conv.shape == (self.C, conv)
        self.w_a2, self.w_g2 = W[p + "a2"].contiguous(), W[p + "g2"].contiguous()
        self.dt_bias, self.A_log, self.w_norm = W[p + "dt_bias"].contiguous(), W[p + "A_log"].contiguous(), W[p + "norm"].contiguous()
        self.w_o = W[p + "o"].contiguous()

    def state_specs(self) -> Dict[str, StateSpec]:
        return {self.name + ".S": StateSpec((self.H, self.V, self.K), torch.float32),
                self.name + ".conv": StateSpec((self.taps - 1, self.C), self.w_in.dtype)}

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        lib, T, dev = S.lib(), ctx.T, h.device
        proj = linear(h, self.w_in)                                         # [T, n_in]
        a = linear(proj[:, self.o_a1:self.o_a1 + self.rank_a], self.w_a2)    # [T, H*K]
        gate = linear(proj[:, self.o_g1:self.o_g1 + self.rank_g], self.w_g2)  # [T, H*V]
        qkv = torch.empty((T, self.C), dtype=torch.float32, device=dev)
        S.check(lib.b2l_seq_conv_silu(_p(proj), self.n_in, _p(self.w_conv), None, _p(ctx.state[self.name + ".conv"]), _p(ctx.meta),
                                      _p(qkv), self.C, T, self.C, self.taps, ctx.act, ctx.stream), "b2l_seq_conv_silu")
        S.check(lib.b2l_seq_unit_norm(_p(qkv, self.o_q), self.C, T, self.G, self.K, self.unit_eps, self.K ** -0.5, ctx.stream), "b2l_seq_unit_norm")
        S.check(lib.b2l_seq_unit_norm(_p(qkv, self.o_k), self.C, T, self.G, self.K, self.unit_eps, 1.0, ctx.stream), "b2l_seq_unit_norm")
        g = torch.empty((T, self.H * self.K), dtype=torch.float32, device=dev)
        S.check(lib.b2l_seq_decay(_p(a), self.H * self.K, _p(self.dt_bias), _p(self.A_log), S.DECAY_EXP_SOFTPLUS, 0.0, _p(g), None, T,
                                  self.H, self.K, ctx.act, ctx.stream), "b2l_seq_decay")
        o = torch.empty((T, self.H * self.V), dtype=torch.float32, device=dev)
        _scan(ctx, q=_p(qkv, self.o_q), ldq=self.C, k=_p(qkv, self.o_k), ldk=self.C, v=_p(qkv, self.o_v), ldv=self.C,
              q_mult=1.0, decay=_p(g), ldd=self.H * self.K, per_channel=True, beta=_p(proj, self.o_b), ldb=self.n_in,
              state=ctx.state[self.name + ".S"], out=_p(o), ldo=self.H * self.V, heads=self.H, qk_heads=self.G, K=self.K, V=self.V)
        y = torch.empty((T, self.H * self.V), dtype=h.dtype, device=dev)
        S.check(lib.b2l_seq_group_norm_gate(_p(o), self.H * self.V, _p(self.w_norm), 1, _p(gate), self.H * self.V, S.ACT_SIGMOID, 0, self.eps,
                                            1.0, _p(y), self.H * self.V, T, self.H * self.V, self.V, ctx.act, ctx.stream), "b2l_seq_group_norm_gate")
        return linear(y, self.w_o)


class Mamba2Mixer:
    """State-space duality layer.  W_in h = [z | x | B | C | dt]; x | B | C pass a causal convolution (+ bias) and silu;
    dt = softplus(dt + dt_bias); per head S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x; then y silu(z),
    RMS norm in `norm_groups` equal parts, W_o.  State: S (f32, heads x vdim x state) and the convolution's inputs."""

    def __init__(self, name: str, W: Dict[str, torch.Tensor], p: str, *, heads: int, vdim: int, state: int, groups: int, norm_groups: int,
                 conv: int, eps: float) -> None:
        self.name, self.H, self.P, self.N, self.G, self.parts, self.taps, self.eps = name, heads, vdim, state, groups, norm_groups, conv, eps
        self.inner = heads * vdim
        self.C = self.inner + 2 * groups * state
        self.w_in = W[p + "in"].contiguous()
        self.n_in = self.w_in.shape[0]
        assert self.n_in == 2 * self.inner + 2 * groups * state + heads, "mamba2: the input projection does not fit z|x|B|C|dt"
        self.w_conv, self.b_conv = W[p + "conv"].contiguous(), W[p + "conv.b"].contiguous()
        self.dt_bias, self.A_log, self.D = W[p + "dt_bias"].contiguous(), W[p + "A_log"].contiguous(), W[p + "D"].contiguous()
        self.w_norm, self.w_o = W[p + "norm"].contiguous(), W[p + "o"].contiguous()

    def state_specs(self) -> Dict[str, StateSpec]:
        return {self.name + ".S": StateSpec((self.H, self.P, self.N), torch.float32),
                self.name + ".conv": StateSpec((self.taps - 1, self.C), self.w_in.dtype)}

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        lib, T, dev = S.lib(), ctx.T, h.device
        u = linear(h, self.w_in)
        xbc = torch.empty((T, self.C), dtype=torch.float32, device=dev)
        S.check(lib.b2l_seq_conv_silu(_p(u, self.inner), self.n_in, _p(self.w_conv), _p(self.b_conv), _p(ctx.state[self.name + ".conv"]),
                                      _p(ctx.meta), _p(xbc), self.C, T, self.C, self.taps, ctx.act, ctx.stream), "b2l_seq_conv_silu")
        decay = torch.empty((T, self.H), dtype=torch.float32, device=dev)
        dt = torch.empty((T, self.H), dtype=torch.float32, device=dev)
        S.check(lib.b2l_seq_decay(_p(u, self.inner + self.C), self.n_in, _p(self.dt_bias), _p(self.A_log), S.DECAY_EXP_SOFTPLUS, 0.0, _p(decay),
                                  _p(dt), T, self.H, 1, ctx.act, ctx.stream), "b2l_seq_decay")
        y = torch.empty((T, self.inner), dtype=torch.float32, device=dev)
        GN = self.G * self.N
        _scan(ctx, q=_p(xbc, self.inner + GN), ldq=self.C, k=_p(xbc, self.inner), ldk=self.C, v=_p(xbc), ldv=self.C, q_mult=1.0,
              decay=_p(decay), ldd=self.H, per_channel=False, vscale=_p(dt), ldvs=self.H, skip=_p(self.D), state=ctx.state[self.name + ".S"],
              out=_p(y), ldo=self.inner, heads=self.H, qk_heads=self.G, K=self.N, V=self.P)
        out = torch.empty((T, self.inner), dtype=h.dtype, device=dev)
        S.check(lib.b2l_seq_group_norm_gate(_p(y), self.inner, _p(self.w_norm), 0, _p(u), self.n_in, S.ACT_SILU, 1, self.eps, 1.0, _p(out),
                                            self.inner, T, self.inner, self.inner // self.parts, ctx.act, ctx.stream), "b2l_seq_group_norm_gate")
        return linear(out, self.w_o)


class MatrixMemoryMixer:
    """Matrix memory with exponential gates (mLSTM), per head, cap(z) = gate_cap tanh(z / gate_cap):

        q = W_q h dim^-1/2;  k = W_k h;  v = W_v h;  log_i = cap(W_i h + b_i);  log_f = log sigmoid(cap(W_f h + b_f))
        m <- max(log_f + m, log_i), starting at 0;  keep = exp(log_f + m_before - m);  put = exp(log_i - m)
        S <- keep S + put k v^T;  n <- keep n + put k;  o = S^T q / (max(|n . q|, exp(-m)) + DEN_ADD)
        y = W_o (o / rms(o) * w_norm * sigmoid(W_g h))
    The projections are one product whose f32 accumulator is kept; everything up to the read-out is f32.  A single token is
    one launch; a portion runs gates, scan (n is a column of ones beside the values) and read-out.  State per sequence:
    S (heads x vdim x dim), n (heads x dim), m (heads), all f32, zero at the start."""

    DEN_ADD = 1e-6

    def __init__(self, name: str, W: Dict[str, torch.Tensor], p: str, *, heads: int, dim: int, vdim: int, gate_cap: float, eps: float) -> None:
        self.name, self.H, self.K, self.V, self.gate_cap, self.eps = name, int(heads), int(dim), int(vdim), float(gate_cap), float(eps)
        parts = [W[p + n] for n in ("q", "k", "v", "g", "i", "f")]
        want = [self.H * self.K] * 2 + [self.H * self.V] * 2 + [self.H] * 2
        assert [w.shape[0] for w in parts] == want and W[p + "o"].shape[1] == self.H * self.V, "matrix memory: projections do not fit the head sizes"
        self.w_in, (self.o_q, self.o_k, self.o_v, self.o_g, self.o_i, self.o_f) = stack_rows(parts)
        self.b_i, self.b_f = W[p + "i.b"].contiguous(), W[p + "f.b"].contiguous()
        self.w_norm, self.w_o = W[p + "norm"].contiguous(), W[p + "o"].contiguous()

    def state_specs(self) -> Dict[str, StateSpec]:
        return {self.name + ".S": StateSpec((self.H, self.V, self.K), torch.float32),
                self.name + ".n": StateSpec((self.H, self.K), torch.float32),
                self.name + ".m": StateSpec((self.H,), torch.float32)}

    def args(self, proj: torch.Tensor, out: torch.Tensor, ctx: StepContext) -> "S.MlstmArgs":
        st, n = ctx.state, self.name
        return S.MlstmArgs(proj=_p(proj), ld=proj.shape[1], q_off=self.o_q, k_off=self.o_k, v_off=self.o_v, g_off=self.o_g, i_off=self.o_i,
                           f_off=self.o_f, b_i=_p(self.b_i), b_f=_p(self.b_f), w_norm=_p(self.w_norm), gate_cap=self.gate_cap, q_mult=self.K ** -0.5,
                           den_add=self.DEN_ADD, eps=self.eps, state_S=_p(st[n + ".S"]), state_n=_p(st[n + ".n"]), state_m=_p(st[n + ".m"]),
                           meta=_p(ctx.meta), out=_p(out), ldo=out.shape[1], T=ctx.T, heads=self.H, K=self.K, V=self.V, act_dtype=ctx.act)

    def recur(self, proj: torch.Tensor, out: torch.Tensor, ctx: StepContext) -> None:
        """Everything between the input product and the output product."""
        lib, T, dev, H, ld = S.lib(), ctx.T, out.device, self.H, proj.shape[1]
        a = self.args(proj, out, ctx)
        if T == 1:
            S.check(lib.b2l_seq_mlstm_step(C.byref(a), ctx.stream), "b2l_seq_mlstm_step")
            return
        gates = torch.empty((4, T, H), dtype=torch.float32, device=dev)               # keep, put, exp(-m), n . q
        o = torch.empty((T, H * self.V), dtype=torch.float32, device=dev)
        a.keep, a.put, a.floor, a.nq, a.o, a.ldr = _p(gates[0]), _p(gates[1]), _p(gates[2]), _p(gates[3]), _p(o), H * self.V
        S.check(lib.b2l_seq_mlstm_gates(C.byref(a), ctx.stream), "b2l_seq_mlstm_gates")
        _scan(ctx, q=_p(proj, self.o_q), ldq=ld, k=_p(proj, self.o_k), ldk=ld, v=_p(proj, self.o_v), ldv=ld, q_mult=self.K ** -0.5, decay=a.keep, ldd=H,
              per_channel=False, vscale=a.put, ldvs=H, state=ctx.state[self.name + ".S"], out=a.o, ldo=H * self.V, heads=H, qk_heads=H, K=self.K,
              V=self.V, state_ones=ctx.state[self.name + ".n"], out_ones=a.nq)
        S.check(lib.b2l_seq_mlstm_readout(C.byref(a), ctx.stream), "b2l_seq_mlstm_readout")

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        proj = linear_f32(h, self.w_in)
        out = torch.empty((ctx.T, self.H * self.V), dtype=h.dtype, device=h.device)
        self.recur(proj, out, ctx)
        return linear(out, self.w_o)


class MinGRUMixer:
    """A gated recurrence whose gates read only the current token, channel by channel:

        z = sigmoid(W_z h + b_z);  u = W_x h + b_x;  c = u + 1/2 where u >= 0, sigmoid(u) where u < 0
        S_t = (1 - z) S_(t-1) + z c;   y = W_o (S_t * silu(W_g h))

    The three projections are one product; everything after it is f32.  State per sequence: S (f32, width), zero at the
    start.  Long portions run as chunks in parallel (the recurrence is linear in S)."""

    def __init__(self, name: str, W: Dict[str, torch.Tensor], p: str, *, width: int) -> None:
        self.name, self.width = name, int(width)
        parts = [W[p + "z"], W[p + "x"], W[p + "g"]]
        assert all(w.shape[0] == self.width for w in parts) and W[p + "o"].shape[1] == self.width, "minGRU: projections do not fit the width"
        self.w_in, (self.o_z, self.o_x, self.o_g) = stack_rows(parts)
        zero = torch.zeros_like(W[p + "z.b"])
        self.b_in, _ = stack_rows([W[p + "z.b"] if (p + "z.b") in W else zero, W[p + "x.b"] if (p + "x.b") in W else zero, zero])
        self.w_o = W[p + "o"].contiguous()

    def state_specs(self) -> Dict[str, StateSpec]:
        return {self.name + ".S": StateSpec((self.width,), torch.float32)}

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        lib, T = S.lib(), ctx.T
        proj = F.linear(h, self.w_in, self.b_in)
        out = torch.empty((T, self.width), dtype=h.dtype, device=h.device)
        n_chunks = lib.b2l_seq_mingru_chunks(T)
        work = torch.empty((n_chunks, 2, self.width), dtype=torch.float32, device=h.device) if n_chunks > 1 else None
        S.check(lib.b2l_seq_mingru(_p(proj), proj.shape[1], self.o_z, self.o_x, self.o_g, _p(ctx.state[self.name + ".S"]), _p(ctx.meta), _p(out),
                                   self.width, _p(work), n_chunks, T, self.width, ctx.act, ctx.stream), "b2l_seq_mingru")
        return linear(out, self.w_o)


# ------------------------------------------------------------------------------------------------ rotation
def rope_frequencies(dims: int, base: float, scaling: Optional[dict]) -> Tuple[torch.Tensor, float]:
    """Per-pair rotation frequencies f_i = base^(-2i/dims), i < dims/2, optionally scaled.  Linear (scaling has a `factor`
    alone): f_i / factor.  YaRN (it also has `original`, `fast` and `slow`): with
    d(t) = dims ln(original / (2 pi t)) / (2 ln base), lo = max(floor(d(fast)), 0), hi = min(ceil(d(slow)), dims - 1) and
    ramp_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1) the frequency becomes f_i / factor * ramp_i + f_i (1 - ramp_i),
    and cos / sin are multiplied by 0.1 ln(factor) + 1.  Returns (f32 frequencies on the CPU, multiplier)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = float(base) ** (-2.0 * i / dims)
    mult = 1.0
    if scaling and "original" not in scaling:
        f = f / float(scaling["factor"])
    elif scaling:
        factor, orig = float(scaling["factor"]), float(scaling["original"])

        def d(t: float) -> float:
            return dims * math.log(orig / (2 * math.pi * t)) / (2 * math.log(float(base)))

        lo = max(math.floor(d(float(scaling["fast"]))), 0)
        hi = min(math.ceil(d(float(scaling["slow"]))), dims - 1)
        ramp = torch.clamp((i - lo) / max(hi - lo, 0.001), 0, 1)
        f = f / factor * ramp + f * (1 - ramp)
        mult = 0.1 * math.log(factor) + 1.0
    return f.to(torch.float32), mult


# ------------------------------------------------------------------------------------------------ attention
def local_attention(a: "S.AttnArgs", ctx: StepContext) -> None:
    """b2l_seq_block_attention with the work space its few-query form asks for."""
    lib = S.lib()
    n = lib.b2l_seq_block_attention_work_floats(C.byref(a))
    work = None
    if n:
        work = torch.empty((n,), dtype=torch.float32, device=ctx.meta.device)
        a.work, a.work_floats = _p(work), n
    S.check(lib.b2l_seq_block_attention(C.byref(a), ctx.stream), "b2l_seq_block_attention")


class BlockSinkAttention:
    """Softmax attention inside blocks of `block` positions (query p sees j <= p with j // block == p // block; block
    None: the whole sequence up to `max_positions`), weights exp(s_j) / (1 + sum exp(s_j)) when `sink`.  As a branch of
    a ParallelMixer it shares the input product: `parts()` lists its projection weights, `run()` consumes columns of
    the shared product and writes its gated heads into a slice of the shared read-out buffer."""

    def __init__(self, name: str, W: Dict[str, torch.Tensor], p: str, *, heads: int, kv_heads: int, dim: int, vdim: int, scale: float,
                 eps: float, softcap: Optional[float] = None, block: Optional[int] = None, rot: Optional[dict] = None, sink: bool = True,
                 max_positions: int = 0) -> None:
        self.name, self.H, self.G, self.K, self.V, self.scale, self.eps = name, heads, kv_heads, dim, vdim, float(scale), eps
        self.softcap = float(softcap) if softcap else 0.0
        self.block = int(block) if block else int(max_positions)
        if self.block <= 0:
            raise ValueError("attention without a block size needs max_positions")
        self.sink = bool(sink)
        self.w = [W[p + "q"], W[p + "k"], W[p + "v"], W[p + "g"]]
        self.q_norm, self.k_norm = W[p + "q.norm"].contiguous(), W[p + "k.norm"].contiguous()
        self.w_o = W[p + "o"]
        self.rot_dims, self.rot_mult, self.freq = 0, 1.0, None
        if rot:
            self.rot_dims = int(rot["dims"])
            f, self.rot_mult = rope_frequencies(self.rot_dims, float(rot["base"]), rot.get("scaling"))
            self.freq = f.to(self.w_o.device)

    def parts(self) -> List[torch.Tensor]:
        return self.w

    def out_width(self) -> int:
        return self.H * self.V

    def state_specs(self) -> Dict[str, StateSpec]:
        dt = self.w_o.dtype
        return {self.name + ".k": StateSpec((self.block, self.G, self.K), dt, zero_on_acquire=False),
                self.name + ".v": StateSpec((self.block, self.G, self.V), dt, zero_on_acquire=False)}

    def run(self, proj: torch.Tensor, offs: List[int], ctx: StepContext, out: torch.Tensor, out_off: int, out_mult: float) -> None:
        lib, T, dev, ld = S.lib(), ctx.T, proj.device, proj.shape[1]
        o_q, o_k, o_v, o_g = offs
        q = torch.empty((T, self.H * self.K), dtype=torch.float32, device=dev)
        kn = torch.empty((T, self.G * self.K), dtype=proj.dtype, device=dev)
        S.check(lib.b2l_seq_headnorm_rope(_p(proj, o_q), ld, _p(self.q_norm), self.eps, _p(self.freq), self.rot_dims, self.rot_mult, _p(ctx.meta),
                                          _p(q), 1, T, self.H, self.K, ctx.act, ctx.stream), "b2l_seq_headnorm_rope")
        S.check(lib.b2l_seq_headnorm_rope(_p(proj, o_k), ld, _p(self.k_norm), self.eps, _p(self.freq), self.rot_dims, self.rot_mult, _p(ctx.meta),
                                          _p(kn), 0, T, self.G, self.K, ctx.act, ctx.stream), "b2l_seq_headnorm_rope")
        a = S.AttnArgs(q=_p(q), k_new=_p(kn), v_new=_p(proj, o_v), ldv=ld, cache_k=_p(ctx.state[self.name + ".k"]),
                       cache_v=_p(ctx.state[self.name + ".v"]), meta=_p(ctx.meta), gate=_p(proj, o_g), ldg=ld, out=_p(out, out_off),
                       ldo=out.shape[1], scale=self.scale, softcap=self.softcap, out_mult=float(out_mult), has_sink=int(self.sink),
                       block=self.block, T=T, heads=self.H, kv_heads=self.G, K=self.K, V=self.V, act_dtype=ctx.act)
        local_attention(a, ctx)


class GatedLinearAttention:
    """S_t = diag(alpha_t) S_(t-1) + k_t v_t^T, o_t = S_t^T (q_t dim^-1/2), alpha = sigmoid(W_a2 W_a1 h + b)^(1/tau);
    read-out: per-head RMS norm (shared weight), times silu(W_g h).  A branch like BlockSinkAttention."""

    def __init__(self, name: str, W: Dict[str, torch.Tensor], p: str, *, heads: int, dim: int, vdim: int, tau: float, eps: float) -> None:
        self.name, self.H, self.K, self.V, self.tau, self.eps = name, heads, dim, vdim, float(tau), eps
        self.w = [W[p + "q"], W[p + "k"], W[p + "v"], W[p + "g"], W[p + "a1"]]
        self.rank = W[p + "a1"].shape[0]
        self.w_a2, self.b_a2 = W[p + "a2"].contiguous(), W[p + "a2.b"].contiguous()
        self.w_norm, self.w_o = W[p + "norm"].contiguous(), W[p + "o"]

    def parts(self) -> List[torch.Tensor]:
        return self.w

    def out_width(self) -> int:
        return self.H * self.V

    def state_specs(self) -> Dict[str, StateSpec]:
        return {self.name + ".S": StateSpec((self.H, self.V, self.K), torch.float32)}

    def run(self, proj: torch.Tensor, offs: List[int], ctx: StepContext, out: torch.Tensor, out_off: int, out_mult: float) -> None:
        lib, T, dev, ld = S.lib(), ctx.T, proj.device, proj.shape[1]
        o_q, o_k, o_v, o_g, o_a1 = offs
        a = linear(proj[:, o_a1:o_a1 + self.rank], self.w_a2)
        n = self.H * self.K
        alpha = torch.empty((T, n), dtype=torch.float32, device=dev)
        S.check(lib.b2l_seq_decay(_p(a), n, _p(self.b_a2), None, S.DECAY_SIGMOID_ROOT, self.tau, _p(alpha), None, T, self.H, self.K, ctx.act,
                                  ctx.stream), "b2l_seq_decay")
        o = torch.empty((T, self.H * self.V), dtype=torch.float32, device=dev)
        nq = o_g - o_q                                   # q | k | v are consecutive columns of the product
        qkv = torch.empty((T, nq), dtype=torch.float32, device=dev)
        S.check(lib.b2l_seq_cast_f32(_p(proj, o_q), ld, _p(qkv), nq, T, nq, ctx.act, ctx.stream), "b2l_seq_cast_f32")
        _scan(ctx, q=_p(qkv), ldq=nq, k=_p(qkv, o_k - o_q), ldk=nq, v=_p(qkv, o_v - o_q), ldv=nq, q_mult=self.K ** -0.5, decay=_p(alpha),
              ldd=n, per_channel=True, state=ctx.state[self.name + ".S"], out=_p(o), ldo=self.H * self.V, heads=self.H, qk_heads=self.H,
              K=self.K, V=self.V)
        S.check(lib.b2l_seq_group_norm_gate(_p(o), self.H * self.V, _p(self.w_norm), 1, _p(proj, o_g), ld, S.ACT_SILU, 0, self.eps, float(out_mult),
                                            _p(out, out_off), out.shape[1], T, self.H * self.V, self.V, ctx.act, ctx.stream),
                "b2l_seq_group_norm_gate")


class ParallelMixer:
    """y = sum_b scale_b * W_o,b branch_b(h): the branches' input projections are one product, and so are their
    output projections (the branches write scale_b * read-out into one buffer that meets [W_o,1 | W_o,2 | ...])."""

    def __init__(self, branches: List[Tuple[object, float]]) -> None:
        self.branches = [b for b, _ in branches]
        self.scales = [float(s) for _, s in branches]
        parts, self.counts = [], []
        for b in self.branches:
            parts += b.parts()
            self.counts.append(len(b.parts()))
        self.w_in, self.offs = stack_rows(parts)
        self.widths = [b.out_width() for b in self.branches]
        self.w_o = torch.cat([b.w_o for b in self.branches], dim=1).contiguous()

    def state_specs(self) -> Dict[str, StateSpec]:
        out: Dict[str, StateSpec] = {}
        for b in self.branches:
            out.update(b.state_specs())
        return out

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        proj = linear(h, self.w_in)
        out = torch.empty((ctx.T, sum(self.widths)), dtype=h.dtype, device=h.device)
        at, col = 0, 0
        for b, n, s, w in zip(self.branches, self.counts, self.scales, self.widths):
            b.run(proj, self.offs[at:at + n], ctx, out, col, s)
            at += n
            col += w
        return linear(out, self.w_o)


class LocalAttention:
    """Causal softmax attention over the last `window` positions (the query's own and the window - 1 before it), over the
    query's block of `block` positions (query p sees j <= p with j // block == p // block), or, with neither, over the whole
    sequence up to `max_positions`.

        q, k, v = W_q h, W_k h, W_v h (one stacked product, with the gate);  q, k: RMS norm, over the whole projection
        with a weight of its size (`norm_over` = "row") or per head with one weight of `dim` entries ("head"), then
        rotation of the first rot.dims entries of every head (entry i with entry i + dims/2); or ("unit") the rotation first,
        then every head divided by its root mean square, without a weight
        v <- (1 - lambda) v + lambda v_first in every layer with `v_mix` but the first of them, whose v is v_first
        with `q_temp` = {"coef", "every"} q at position p is multiplied by 1 + coef ln(floor((p + 1) / every) + 1)
        weights = softmax(q . k * scale) over the visible keys, with `sink` exp(s_j) / (1 + sum_j exp(s_j)); query head h
        reads key / value head h // (heads / kv_heads)
        y = W_o (concat_h(sum_j weight_j v_j) * sigmoid(W_g h))            a gate per output channel (`gate` = "channel" or
        True), one number per head (`gate` = "head"), or no gate (False)

    State per sequence: a ring of `window` (or `block`) positions of rotated keys and (mixed) values, entry position %
    size.  The first value-mixing layer of a step leaves its values in `ctx.shared` for the later ones."""

    NORMS = ("row", "head", "unit")

    def __init__(self, name: str, W: Dict[str, torch.Tensor], p: str, *, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float,
                 window: Optional[int] = None, block: Optional[int] = None, max_positions: int = 0, rot: Optional[dict] = None,
                 norm_over: str = "row", gate=True, v_mix: bool = False, mix_key: str = "v_first", sink: bool = False,
                 q_temp: Optional[dict] = None) -> None:
        self.name, self.H, self.G, self.K, self.V, self.scale, self.eps = name, int(heads), int(kv_heads), int(dim), int(vdim), float(scale), eps
        if window is not None and block is not None:
            raise ValueError("local attention: a window or blocks, not both")
        self.window = 0 if window is None else int(window)                     # 0: inside blocks
        self.ring = int(window if window is not None else (block or max_positions))
        if self.ring < 1 or self.H % self.G:
            raise ValueError("local attention: the window or block must hold at least the query's own position, heads a multiple of kv_heads")
        if norm_over not in self.NORMS:
            raise ValueError(f"local attention: norm over {norm_over!r}")
        self.whole_row, self.unit_rms, self.v_mix, self.mix_key = int(norm_over == "row"), int(norm_over == "unit"), bool(v_mix), mix_key
        assert W[p + "q"].shape[0] == heads * dim and W[p + "k"].shape[0] == kv_heads * dim and W[p + "v"].shape[0] == kv_heads * vdim, \
            "local attention: projections do not fit the head sizes"
        if gate not in (True, False, "channel", "head"):
            raise ValueError(f"local attention: gate per {gate!r}")
        self.gate_per_channel, self.sink = int(gate in (True, "channel")), int(bool(sink))
        assert W[p + "o"].shape[1] == heads * vdim and (not gate or W[p + "g"].shape[0] == (heads * vdim if self.gate_per_channel else heads)), \
            "local attention: gate / output do not fit"
        self.temp_coef, self.temp_every = (float(q_temp["coef"]), int(q_temp["every"])) if q_temp else (0.0, 0)
        if q_temp and (self.temp_every < 1 or self.temp_every != q_temp["every"]):
            raise ValueError(f"local attention: the query temperature steps every {q_temp['every']!r} positions")
        self.w_in, offs = stack_rows([W[p + "q"], W[p + "k"], W[p + "v"]] + ([W[p + "g"]] if gate else []))
        self.o_q, self.o_k, self.o_v = offs[:3]
        self.o_g = offs[3] if gate else None
        self.q_norm = W[p + "q.norm"].contiguous() if (p + "q.norm") in W else None
        self.k_norm = W[p + "k.norm"].contiguous() if (p + "k.norm") in W else None
        self.lam = W[p + "vmix"].reshape(1).contiguous() if self.v_mix else None
        self.w_o = W[p + "o"].contiguous()
        self.rot_dims, self.rot_mult, self.freq = 0, 1.0, None
        if rot and int(rot.get("dims", 0)):
            self.rot_dims = int(rot["dims"])
            f, self.rot_mult = rope_frequencies(self.rot_dims, float(rot["base"]), rot.get("scaling"))
            self.freq = f.to(self.w_o.device)

    def state_specs(self) -> Dict[str, StateSpec]:
        dt = self.w_o.dtype
        return {self.name + ".k": StateSpec((self.ring, self.G, self.K), dt, zero_on_acquire=False),
                self.name + ".v": StateSpec((self.ring, self.G, self.V), dt, zero_on_acquire=False)}

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        lib, T, dev = S.lib(), ctx.T, h.device
        proj = linear(h, self.w_in)
        ld = proj.shape[1]
        q = torch.empty((T, self.H * self.K), dtype=torch.float32, device=dev)
        kn = torch.empty((T, self.G * self.K), dtype=proj.dtype, device=dev)
        first = ctx.shared.get(self.mix_key) if self.v_mix else None          # (tensor, column, leading dimension, width) of the first layer's values
        if first is not None and first[3] != self.G * self.V:
            raise ValueError(f"{self.name}: values of {self.G * self.V} entries cannot be mixed with the first layer's {first[3]}")
        v, v_off, ldv = proj, self.o_v, ld
        vm = None
        if first is not None:
            vm = torch.empty((T, self.G * self.V), dtype=proj.dtype, device=dev)
            v, v_off, ldv = vm, 0, self.G * self.V
        elif self.v_mix:
            ctx.shared[self.mix_key] = (proj, self.o_v, ld, self.G * self.V)
        a = S.QkvPrepArgs(proj=_p(proj), ld=ld, q_off=self.o_q, k_off=self.o_k, v_off=self.o_v, q_norm=_p(self.q_norm), k_norm=_p(self.k_norm),
                          whole_row=self.whole_row, eps=self.eps, freq=_p(self.freq), rot_dims=self.rot_dims, rot_mult=self.rot_mult,
                          meta=_p(ctx.meta), q_out=_p(q), k_out=_p(kn), v_first=_p(first[0], first[1]) if first is not None else None,
                          ldvf=first[2] if first is not None else 0, lambda_=_p(self.lam) if first is not None else None, v_out=_p(vm), T=T,
                          heads=self.H, kv_heads=self.G, K=self.K, V=self.V, act_dtype=ctx.act, unit_rms=self.unit_rms, temp_coef=self.temp_coef,
                          temp_every=self.temp_every)
        S.check(lib.b2l_seq_qkv_prep(C.byref(a), ctx.stream), "b2l_seq_qkv_prep")
        att = torch.empty((T, self.H * self.V), dtype=h.dtype, device=dev)
        gated = self.o_g is not None
        b = S.AttnArgs(q=_p(q), k_new=_p(kn), v_new=_p(v, v_off), ldv=ldv, cache_k=_p(ctx.state[self.name + ".k"]),
                       cache_v=_p(ctx.state[self.name + ".v"]), meta=_p(ctx.meta), gate=_p(proj, self.o_g) if gated else None, ldg=ld if gated else 0,
                       out=_p(att), ldo=self.H * self.V, scale=self.scale, softcap=0.0, out_mult=1.0, has_sink=self.sink, block=self.ring, T=T, heads=self.H,
                       kv_heads=self.G, K=self.K, V=self.V, act_dtype=ctx.act, window=self.window, gate_per_channel=self.gate_per_channel)
        local_attention(b, ctx)
        return linear(att, self.w_o)


class SlidingWindowAttention(LocalAttention):
    """`LocalAttention` over a sliding window, q / k norms with weights, the output gated per channel."""

    def __init__(self, name: str, W: Dict[str, torch.Tensor], p: str, *, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, window: int,
                 eps: float, rot: Optional[dict] = None, v_mix: bool = False, norm_over: str = "row", mix_key: str = "v_first") -> None:
        if norm_over not in ("row", "head"):
            raise ValueError(f"sliding-window attention: norm over {norm_over!r}")
        super().__init__(name, W, p, heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, eps=eps, window=window, rot=rot,
                         norm_over=norm_over, gate=True, v_mix=v_mix, mix_key=mix_key)


class DifferentialAttention:
    """Causal softmax attention with two score maps per head over the same values.

        q = conv(W_q h + b_q) [heads x 2 x dim], k = conv(W_k h + b_k) [kv_heads x 2 x dim], v = conv(W_v h + b_v) [kv_heads x vdim]
        conv: a causal convolution of `conv` taps over time on every channel (no bias, no activation)
        q, k: the first rot.dims entries of every map of every head turn by position, pairs (2i, 2i+1) when `interleaved`
        a_m = softmax_j(q_m . k_m,j * scale) v_j over all j <= i, for the maps m = 0, 1;  query head h reads key/value head
        h // (heads / kv_heads)
        o = a_0 - lambda a_1,  lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff  (one number per layer)
        y = W_o concat_h(o / sqrt(mean(o^2) + eps) * (1 - diff))

    The three projections are one product.  State per sequence: the last conv - 1 projected rows, and every position's
    rotated keys and convolved values (`max_positions` of them).  With `kv_from` (an earlier DifferentialAttention with the
    same head counts and rotation) the layer has only queries of its own: it attends over that layer's keys and values, read
    from that layer's cache and, for the portion's own tokens, from what that layer left in `ctx.shared` in this step."""

    def __init__(self, name: str, W: Dict[str, torch.Tensor], p: str, *, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, diff: float,
                 eps: float, conv: int = 0, rot: Optional[dict] = None, max_positions: int = 0, kv_from: Optional["DifferentialAttention"] = None,
                 interleaved: bool = True) -> None:
        if max_positions <= 0:
            raise ValueError("differential attention caches every position: it needs max_positions")
        self.name, self.H, self.G, self.K, self.V = name, int(heads), int(kv_heads), int(dim), int(vdim)
        self.scale, self.diff, self.eps, self.max_positions, self.interleaved = float(scale), float(diff), eps, int(max_positions), bool(interleaved)
        if self.H % self.G or self.K % 2:
            raise ValueError("differential attention: heads must be a multiple of kv_heads, the map size even")
        self.src = kv_from
        if kv_from is not None and (kv_from.src is not None or (kv_from.H, kv_from.G, kv_from.K, kv_from.V) != (self.H, self.G, self.K, self.V)):
            raise ValueError(f"{name}: keys and values must come from a layer with projections of its own and the same head sizes")
        names = ["q"] if kv_from is not None else ["q", "k", "v"]
        rows = {"q": self.H * 2 * self.K, "k": self.G * 2 * self.K, "v": self.G * self.V}
        for n in names:
            assert W[p + n].shape[0] == rows[n], f"differential attention: projection {n} does not fit the head sizes"
        assert W[p + "o"].shape[1] == self.H * self.V, "differential attention: output projection does not fit"
        self.w_in, offs = stack_rows([W[p + n] for n in names])
        self.b_in, _ = stack_rows([W[p + n + ".b"] if (p + n + ".b") in W else torch.zeros_like(W[p + n][:, 0]) for n in names])
        self.o_q, self.o_k, self.o_v = offs[0], (offs[1] if len(offs) > 1 else -1), (offs[2] if len(offs) > 2 else -1)
        self.C = self.w_in.shape[0]
        self.taps = int(conv) if conv else 1
        if conv:
            self.w_conv, _ = stack_rows([W[p + n + ".conv"] for n in names])
            assert self.w_conv.shape == (self.C, self.taps), "differential attention: convolution weights do not fit"
        else:                                   # no convolution: one tap of weight one
            self.w_conv = torch.ones((self.C, 1), dtype=self.w_in.dtype, device=self.w_in.device)
        lam = [float((W[p + f"lq{m}"].double() * W[p + f"lk{m}"].double()).sum()) for m in (1, 2)]
        self.lam = math.exp(lam[0]) - math.exp(lam[1]) + self.diff
        self.w_o = W[p + "o"].contiguous()
        self.rot_dims, self.rot_mult, self.freq = 0, 1.0, None
        if rot and int(rot.get("dims", 0)):
            self.rot_dims = int(rot["dims"])
            f, self.rot_mult = rope_frequencies(self.rot_dims, float(rot["base"]), rot.get("scaling"))
            self.freq = f.to(self.w_o.device)

    def state_specs(self) -> Dict[str, StateSpec]:
        dt = self.w_o.dtype
        out = {self.name + ".conv": StateSpec((self.taps - 1, self.C), dt)} if self.taps > 1 else {}
        if self.src is None:
            out[self.name + ".k"] = StateSpec((self.max_positions, self.G * 2 * self.K), dt, zero_on_acquire=False)
            out[self.name + ".v"] = StateSpec((self.max_positions, self.G * self.V), dt, zero_on_acquire=False)
        return out

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        lib, T, dev, H, G, K, V = S.lib(), ctx.T, h.device, self.H, self.G, self.K, self.V
        proj = F.linear(h, self.w_in, self.b_in)
        q = torch.empty((T, H * 2 * K), dtype=torch.float32, device=dev)
        own = self.src is None
        kn = torch.empty((T, G * 2 * K), dtype=proj.dtype, device=dev) if own else None
        vn = torch.empty((T, G * V), dtype=proj.dtype, device=dev) if own else None
        a = S.ConvRopeArgs(proj=_p(proj), ld=proj.shape[1], c_off=0, C=self.C, taps=self.taps, w=_p(self.w_conv),
                           state=_p(ctx.state[self.name + ".conv"]) if self.taps > 1 else None, meta=_p(ctx.meta), q_off=self.o_q, q_heads=2 * H,
                           k_off=self.o_k, k_heads=2 * G, K=K, v_off=self.o_v, n_v=G * V, freq=_p(self.freq), rot_dims=self.rot_dims,
                           interleaved=int(self.interleaved), rot_mult=self.rot_mult, q_out=_p(q), k_out=_p(kn), v_out=_p(vn), T=T, act_dtype=ctx.act)
        S.check(lib.b2l_seq_conv_rope(C.byref(a), ctx.stream), "b2l_seq_conv_rope")
        if own:
            ctx.shared["kv:" + self.name] = (kn, vn)
            holder = self.name
        else:
            if ("kv:" + self.src.name) not in ctx.shared:
                raise RuntimeError(f"{self.name}: layer {self.src.name} has not run in this step")
            kn, vn = ctx.shared["kv:" + self.src.name]
            holder = self.src.name
        maps = torch.empty((T, H * 2 * V), dtype=torch.float32, device=dev)      # scratch of the forms that do not merge the maps themselves
        y = torch.empty((T, H * V), dtype=h.dtype, device=dev)
        b = S.AttnArgs(q=_p(q), k_new=_p(kn), v_new=_p(vn), ldv=G * V, cache_k=_p(ctx.state[holder + ".k"]), cache_v=_p(ctx.state[holder + ".v"]),
                       meta=_p(ctx.meta), gate=None, ldg=0, out=_p(maps), ldo=H * 2 * V, scale=self.scale, softcap=0.0, out_mult=1.0, has_sink=0,
                       block=self.max_positions, T=T, heads=2 * H, kv_heads=G, K=K, V=V, act_dtype=ctx.act, window=0, gate_per_channel=0, maps=2,
                       out_f32=1, no_append=int(not own), diff_out=_p(y), ldd=H * V, diff_lambda=self.lam, diff_eps=self.eps,
                       diff_mult=1.0 - self.diff)
        local_attention(b, ctx)                 # attention of both maps and the differential read-out
        return linear(y, self.w_o)


# ------------------------------------------------------------------------------------------------ residual streams
def norm_rows(x: torch.Tensor, w: torch.Tensor, b: Optional[torch.Tensor], kind: str, eps: float, ctx: StepContext,
              rows: Optional[torch.Tensor] = None, n_rows: Optional[int] = None) -> torch.Tensor:
    """RMS norm ("rms") or layer norm with a bias ("layer") of rows of the f32 stream x [T, width] -> act [n_rows, width]."""
    n = x.shape[0] if n_rows is None else n_rows
    out = torch.empty((n, x.shape[1]), dtype=ctx.dtype, device=x.device)
    S.check(S.lib().b2l_seq_norm(_p(x), _p(w), _p(b), NORM_KINDS[kind], eps, _p(out), _p(rows), n, x.shape[1], ctx.act, ctx.stream), "b2l_seq_norm")
    return out


NORM_KINDS = {"rms": S.NORM_RMS, "layer": S.NORM_LAYER}


def residual_step(x_in: torch.Tensor, x_out: Optional[torch.Tensor], ctx: StepContext, *, y1: Optional[torch.Tensor] = None, y2: Optional[torch.Tensor] = None,
                  vec: Optional[torch.Tensor] = None, base: Optional[torch.Tensor] = None, norm: Optional[torch.Tensor] = None,
                  bias: Optional[torch.Tensor] = None, kind: str = "rms", eps: float = 0.0, split: bool = False) -> Optional[torch.Tensor]:
    """x_out = x_in + y1 + y2 (act rows) + vec (act, the same for every token) + base (f32 rows), f32 [T, width]; x_out may be
    x_in.  Returns norm(x_out) (act) when `norm` is given, or with `split` the row as two act numbers per entry [T, 2 width]
    (see LoopInjection), or None: one launch in every case."""
    T, D = x_in.shape
    h = torch.empty((T, D), dtype=ctx.dtype, device=x_in.device) if norm is not None else None
    s = torch.empty((T, 2 * D), dtype=ctx.dtype, device=x_in.device) if split else None
    a = S.ResidualArgs(x_in=_p(x_in), base=_p(base), vec=_p(vec), y1=_p(y1), y2=_p(y2), x_out=_p(x_out), split=_p(s), w=_p(norm), b=_p(bias), h=_p(h),
                       eps=eps, norm_kind=NORM_KINDS[kind], T=T, D=D, act_dtype=ctx.act)
    S.check(S.lib().b2l_seq_residual_step(C.byref(a), ctx.stream), "b2l_seq_residual_step")
    return s if split else h


class LoopInjection:
    """What stands before every pass of a looped stretch of layers:  x <- W_in [x; x0] + step[t],  x0 the embedding output and t
    the number of the pass.

    The half of the product on x0 is the same for every pass, so a portion computes it once (`start`).  The other half reads
    the f32 stream: as it is (few tokens, float32 mode), or, where the library takes bf16 operands, as the pair hi + lo of
    bf16 numbers in one product of twice the length, so that passing through W_in does not round the stream to 8 digits."""

    def __init__(self, w_in: torch.Tensor, step: torch.Tensor) -> None:
        D = w_in.shape[0]
        if w_in.shape[1] != 2 * D or step.dim() != 2 or step.shape[1] != D:
            raise ValueError(f"loop injection: {tuple(w_in.shape)} and {tuple(step.shape)} do not fit")
        self.width, self.times = D, step.shape[0]
        self.w_x, self.w_0 = w_in[:, :D].contiguous(), w_in[:, D:].contiguous()
        self.w_xx = torch.cat([self.w_x, self.w_x], dim=1).contiguous() if w_in.dtype != torch.float32 else self.w_x
        self.step = step.contiguous()

    def wants_split(self, ctx: StepContext) -> bool:
        """Whether `forward` takes the stream as the pair of act numbers that residual_step(split=True) returns."""
        return ctx.T > FEW_TOKENS and ctx.dtype != torch.float32

    def start(self, x0: torch.Tensor, h0: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        """W_in's half on the embedding output: x0 in f32, h0 the same in the activation type.  f32 [T, width]."""
        if ctx.T > FEW_TOKENS:
            return linear_f32(h0, self.w_0)
        return self._few(self.w_0, x0, None, None, ctx)

    def _few(self, w, x, base, vec, ctx: StepContext) -> torch.Tensor:
        out = torch.empty((ctx.T, self.width), dtype=torch.float32, device=x.device)
        S.check(S.lib().b2l_seq_linear_few(_p(w), _p(x), _p(base), _p(vec), _p(out), ctx.T, self.width, self.width, ctx.act, ctx.stream),
                "b2l_seq_linear_few")
        return out

    def forward(self, x: torch.Tensor, split: Optional[torch.Tensor], base: torch.Tensor, t: int, ctx: StepContext, *, norm: torch.Tensor,
                bias: Optional[torch.Tensor], kind: str, eps: float) -> Tuple[torch.Tensor, torch.Tensor]:
        """The stream x (f32; `split` as residual_step returns it when `wants_split`) before pass t -> (new stream, its norm)."""
        if ctx.T <= FEW_TOKENS:
            new = self._few(self.w_x, x, base, self.step[t], ctx)
            return new, norm_rows(new, norm, bias, kind, eps, ctx)
        new = linear_f32(split, self.w_xx) if split is not None else F.linear(x, self.w_x)
        return new, residual_step(new, new, ctx, base=base, vec=self.step[t], norm=norm, bias=bias, kind=kind, eps=eps)


class DepthAverage:
    """The residual stream of layers that read a learned average over everything before them.  With X_0 the embedding
    output and X_(i+1) = x_i + (what layer i's sublayers add to their input x_i), the next layer's input is
    x_(i+1) = sum_(j <= i+1) avg_i[j] X_j (avg_i None: X_(i+1) itself, the ordinary residual stream).  `history` holds the
    X_j of one portion ([layers + 1, T, width] f32); `step` writes X_(i+1), forms x_(i+1) and the next norm in one launch."""

    def __init__(self, weights: List[Optional[torch.Tensor]]) -> None:
        self.avg = []
        for i, w in enumerate(weights):
            if w is not None and w.numel() != i + 2:
                raise ValueError(f"layer {i}: {w.numel()} depth weights, {i + 2} earlier results")
            self.avg.append(w.to(torch.float32).contiguous() if w is not None else None)

    def history(self, ctx: StepContext, width: int, device) -> torch.Tensor:
        return torch.empty((len(self.avg) + 1, ctx.T, width), dtype=torch.float32, device=device)

    def step(self, i: int, hist: torch.Tensor, x_in: torch.Tensor, x_out: torch.Tensor, y1: torch.Tensor, y2: Optional[torch.Tensor], ctx: StepContext, *,
             norm: Optional[torch.Tensor] = None, bias: Optional[torch.Tensor] = None, kind: str = "layer", eps: float = 0.0) -> Optional[torch.Tensor]:
        """Layer i's results y1 (+ y2) on its input x_in -> the next input in x_out (may be x_in), and its norm (act) when `norm` is given."""
        T, D = x_in.shape
        h = torch.empty((T, D), dtype=ctx.dtype, device=x_in.device) if norm is not None else None
        S.check(S.lib().b2l_seq_depth_step(_p(y1), _p(y2), _p(x_in), _p(hist), i + 2, _p(self.avg[i]), _p(x_out), _p(norm), _p(bias), NORM_KINDS[kind],
                                           eps, _p(h), T, D, ctx.act, ctx.stream), "b2l_seq_depth_step")
        return h


class PairHashEmbedding:
    """x = embed[token] * scale + pair[(previous token * mul_prev + token * mul_cur) mod buckets], the first token of a
    sequence reading the pair table's last row (number `buckets`); written into `streams` equal residual streams
    [T, streams, width] (f32).  `pair` None: the token embedding alone.  State per sequence: its last token."""

    def __init__(self, name: str, embed: torch.Tensor, pair: Optional[torch.Tensor], *, buckets: int = 0, mul_prev: int = 0, mul_cur: int = 0,
                 scale: float = 1.0, streams: int = 1) -> None:
        self.name, self.embed, self.pair = name, embed.contiguous(), pair.contiguous() if pair is not None else None
        self.vocab, self.width = self.embed.shape
        self.buckets, self.mul_prev, self.mul_cur, self.scale, self.streams = int(buckets), int(mul_prev), int(mul_cur), float(scale), int(streams)
        if self.pair is not None and tuple(self.pair.shape) != (self.buckets + 1, self.width):
            raise ValueError(f"pair embedding is {tuple(self.pair.shape)}, {self.buckets} buckets and a first-token row need {(self.buckets + 1, self.width)}")

    def state_specs(self) -> Dict[str, StateSpec]:
        return {self.name + ".prev": StateSpec((1,), torch.int32)} if self.pair is not None else {}

    def forward(self, tokens: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        x = torch.empty((ctx.T, self.streams, self.width), dtype=torch.float32, device=self.embed.device)
        prev = ctx.state[self.name + ".prev"] if self.pair is not None else None
        S.check(S.lib().b2l_seq_embed_pair(_p(tokens), int(tokens.dtype == torch.int64), _p(self.embed), _p(self.pair), self.scale, _p(prev),
                                           _p(ctx.meta), self.mul_prev, self.mul_cur, self.buckets, _p(x), ctx.T, self.width, self.vocab,
                                           self.streams, ctx.act, ctx.stream), "b2l_seq_embed_pair")
        return x


class HyperConnection:
    """One sublayer over `streams` residual streams: it reads u = sum_s read[s] x_s, and its result y is written as
    x_t <- sum_s mix[s, t] x_s + write[t] y for all streams at once (mix indexed [from, to]).  The weights are f32 on
    the device; `plain(streams)` is the ordinary residual step (one stream, all weights 1).  `step()` fuses the write
    of one sublayer with the read and the RMS norm of the next."""

    def __init__(self, read: torch.Tensor, mix: torch.Tensor, write: torch.Tensor) -> None:
        self.streams = int(read.numel())
        if tuple(mix.shape) != (self.streams, self.streams) or write.numel() != self.streams:
            raise ValueError(f"hyper-connection: read {tuple(read.shape)}, mix {tuple(mix.shape)}, write {tuple(write.shape)} do not fit")
        self.read, self.mix, self.write = (t.to(torch.float32).contiguous() for t in (read, mix, write))

    @classmethod
    def plain(cls, device, streams: int = 1) -> "HyperConnection":
        if streams != 1:
            raise ValueError("a plain residual step has one stream")
        one = torch.ones(1, dtype=torch.float32, device=device)
        return cls(one, one.reshape(1, 1), one)

    @staticmethod
    def step(x: torch.Tensor, ctx: StepContext, *, y: Optional[torch.Tensor] = None, wrote: Optional["HyperConnection"] = None,
             reads: Optional["HyperConnection"] = None, read_weights: Optional[torch.Tensor] = None, norm: Optional[torch.Tensor] = None,
             eps: float = 0.0, rows: Optional[torch.Tensor] = None, n_rows: Optional[int] = None) -> Optional[torch.Tensor]:
        """x [T, streams, width] f32, updated in place with sublayer `wrote`'s result y; then, with `norm`, the input of
        the next sublayer `reads` (or any read weights, e.g. ones for the sum of the streams): act [n_rows, width]."""
        T, n_s, D = x.shape
        n = T if n_rows is None else n_rows
        rw = reads.read if reads is not None else read_weights
        h = torch.empty((n, D), dtype=ctx.dtype, device=x.device) if norm is not None else None
        S.check(S.lib().b2l_seq_hc_step(_p(y), _p(x), _p(wrote.mix) if y is not None else None, _p(wrote.write) if y is not None else None,
                                        _p(rw) if norm is not None else None, _p(norm), _p(h), eps, _p(rows), n, D, n_s, ctx.act, ctx.stream),
                "b2l_seq_hc_step")
        return h


# ------------------------------------------------------------------------------------------------ latent attention
class LatentAttention:
    """Causal softmax attention over a cached latent.

        c_q = rmsnorm(W_dq h) w_q;  q = W_uq c_q, or (q_rank None) q = W_q h;  per head [dim unrotated | rot_dim rotated]
        [c' | k_r] = W_dkv h;  c = rmsnorm(c') w_kv (kv_rank);  k_r rotated by position, shared by all heads
        key_h = [W_uk,h c | k_r],  value_h = W_uv,h c,  score = q . key * scale
        weights exp(s_j) / (exp(sink_h) + sum_j exp(s_j)),  y = W_o concat_h(sum_j weight_j value_j), with `gate` times
        sigmoid(W_g h) per channel before W_o

    over every earlier position, or with `window` over the query's own position and the window - 1 before it; without a
    `sink` tensor the softmax is the ordinary one.  A YaRN `scaling` of the rotation stretches the slow frequencies and
    multiplies cos and sin of q_r and k_r; `scale` is taken as given.

    Only [c | k_r] is cached per position.  Single tokens and short portions attend in the latent space: the query is
    multiplied by W_uk once (q' = W_uk,h^T q_h), scores are q' . c + q_r . k_r, the weighted sum of latents is mapped
    through W_uv afterwards (up to FEW_TOKENS tokens in the launch that merges the key splits and gates, and with direct
    queries W_uk is applied in the launch that turns the rotated parts); every head reads the same cached row, once.  Portions of `expand_from` tokens or more
    expand [value_h | key_h] of every cached position with one product and attend per head, which costs several times
    fewer operations per (query, key) pair.  Both forms run the same kernel.  `rot`: {"base", "dims"} on the first
    `dims` entries of the rotated part, pairs (2i, 2i+1) when `interleaved`."""

    expand_from: int = 64                 # portions at least this long take the expanded form
    expand_limit: int = 1 << 31           # ... unless the expansion would have more elements than this

    def __init__(self, name: str, W: Dict[str, torch.Tensor], p: str, *, heads: int, dim: int, rot_dim: int, vdim: int, q_rank: Optional[int],
                 kv_rank: int, scale: float, eps: float, rot: Optional[dict], max_positions: int, interleaved: bool = True,
                 window: Optional[int] = None, gate: bool = False) -> None:
        if max_positions <= 0:
            raise ValueError("latent attention caches every position: it needs max_positions")
        self.window = int(window) if window else 0
        if self.window < 0:
            raise ValueError("latent attention: negative window")
        self.name, self.H, self.dn, self.dr, self.dv, self.rq, self.rk = name, heads, dim, rot_dim, vdim, q_rank, kv_rank
        self.scale, self.eps, self.max_positions, self.interleaved = float(scale), eps, int(max_positions), bool(interleaved)
        w_q = W[p + "q"] if q_rank is None else W[p + "dq"]
        assert w_q.shape[0] == (heads * (dim + rot_dim) if q_rank is None else q_rank) and W[p + "dkv"].shape[0] == kv_rank + rot_dim, \
            "latent attention: the input projections do not fit"
        self.w_in, offs = stack_rows([w_q, W[p + "dkv"]] + ([W[p + "g"]] if gate else []))
        self.o_q, self.o_kv, self.o_g = offs[0], offs[1], (offs[2] if gate else None)
        assert not gate or W[p + "g"].shape[0] == heads * vdim, "latent attention: the gate does not fit"
        self.kv_norm = W[p + "dkv.norm"].contiguous()
        self.q_norm = self.w_uq = None
        if q_rank is not None:
            self.q_norm, self.w_uq = W[p + "dq.norm"].contiguous(), W[p + "uq"].contiguous()
            assert self.w_uq.shape == (heads * (dim + rot_dim), q_rank), "latent attention: query up-projection does not fit"
        uk, uv = W[p + "uk"].reshape(heads, dim, kv_rank), W[p + "uv"].reshape(heads, vdim, kv_rank)
        self.w_uk = uk.contiguous()                                                            # q' = q_h W_uk,h
        self.w_uv = uv.contiguous()                                                            # value = W_uv,h o'
        self.w_expand = torch.cat([uv, uk], dim=1).reshape(heads * (vdim + dim), kv_rank).contiguous()   # per head [value | key] rows
        self.sink = W[p + "sink"].to(torch.float32).contiguous() if (p + "sink") in W else None
        self.w_o = W[p + "o"].contiguous()
        self.rot_dims, self.rot_mult, self.freq = 0, 1.0, None
        if rot and rot_dim:
            self.rot_dims = int(rot["dims"])
            if self.rot_dims > rot_dim:
                raise ValueError(f"latent attention: {self.rot_dims} rotated entries in a part of {rot_dim}")
            f, self.rot_mult = rope_frequencies(self.rot_dims, float(rot["base"]), rot.get("scaling"))
            self.freq = f.to(self.w_o.device)

    def state_specs(self) -> Dict[str, StateSpec]:
        return {self.name + ".kv": StateSpec((self.max_positions, self.rk + self.dr), self.w_o.dtype, zero_on_acquire=False)}

    def _splits(self, ctx: StepContext, hpg: int) -> int:
        """Key splits: fill the machine when there are few rows; never a function of the position inside a captured step."""
        T = ctx.T
        n_keys = self.max_positions if ctx.pos_hint is None else min(self.max_positions, ctx.pos_hint + T)
        if self.window:
            n_keys = min(n_keys, self.window + 4 * S.lib().b2l_seq_latent_attention_warps(T, hpg) // hpg)     # what one CTA's rows see
        warps = S.lib().b2l_seq_latent_attention_warps(T, hpg)
        ctas = -(-T * hpg // (4 * warps)) * (self.H // hpg)
        if ctas >= 444:                       # a full wave of three CTAs per SM
            return 1
        return max(1, min(-(-444 // ctas), -(-n_keys // 32)))

    def _attend(self, ctx: StepContext, out: Optional[torch.Tensor], vdim: int, splits: int, **kw) -> Optional[torch.Tensor]:
        """The attention kernel into `out`, or (out None) its partial results: f32 [splits, T * heads, vdim + 2]."""
        dev = ctx.meta.device
        work = torch.empty((splits, ctx.T * self.H, vdim + 2), dtype=torch.float32, device=dev) if splits > 1 or out is None else None
        a = S.LatentAttnArgs(sink=_p(self.sink), meta=_p(ctx.meta), out=_p(out), ldo=self.H * vdim, work=_p(work), scale=self.scale, T=ctx.T,
                             heads=self.H, vdim=vdim, splits=splits, act_dtype=ctx.act, window=self.window, partial=int(out is None), **kw)
        S.check(S.lib().b2l_seq_latent_attention(C.byref(a), ctx.stream), "b2l_seq_latent_attention")
        return work

    def _rope(self, x: torch.Tensor, off: int, rot_off: int, size: int, out: torch.Tensor, ctx: StepContext) -> None:
        """Entries [off, off + size) of every head of x -> out (f32), the rotated entries from rot_off on turned by position."""
        H, dq = self.H, self.dn + self.dr
        S.check(S.lib().b2l_seq_rope(_p(x, off), H * dq, int(x.dtype == torch.float32), _p(self.freq), self.rot_dims, int(self.interleaved), rot_off, 1.0,
                                     self.rot_mult, _p(ctx.meta), _p(out), H * size, 1, ctx.T, H, size, dq, size, ctx.act, ctx.stream), "b2l_seq_rope")

    def _queries(self, h: torch.Tensor, cache: torch.Tensor, ctx: StepContext, expanded: bool):
        """Projections of the portion: appends its latents to the cache and returns (gate, q32, q_lat, q_rot): q32 f32
        [T, H * (dim + rot_dim)] for the expanded form, or q_lat f32 [H, T, rank] and q_rot f32 [T, H, rot_dim]."""
        lib, T, dev, H, dn, dr = S.lib(), ctx.T, h.device, self.H, self.dn, self.dr
        dq, f32 = dn + dr, h.dtype == torch.float32
        proj = linear_f32(h, self.w_in)
        gate = (proj, self.o_g) if self.o_g is not None else None
        q32 = torch.empty((T, H * dq), dtype=torch.float32, device=dev) if expanded else None
        q_rot = torch.empty((T, H, max(dr, 1)), dtype=torch.float32, device=dev) if not expanded else None
        qn = q_lat = None
        if self.rq is None:
            if not expanded:
                if T <= FEW_TOKENS:
                    q_lat = torch.empty((H, T, self.rk), dtype=torch.float32, device=dev)
                else:
                    qn = torch.empty((H, T, dn), dtype=h.dtype, device=dev)
            a = S.LatentOperandsArgs(proj=_p(proj), ld=proj.shape[1], q_off=self.o_q, kv_off=self.o_kv, heads=H, dn=dn, dr=dr, rank=self.rk, w_kv=_p(self.kv_norm),
                                     freq=_p(self.freq), rot_dims=self.rot_dims, interleaved=int(self.interleaved), rot_mult=self.rot_mult, eps=self.eps,
                                     meta=_p(ctx.meta), cache=_p(cache), max_pos=self.max_positions, q_full=_p(q32), q_nope=_p(qn), q_rot=_p(q_rot),
                                     w_uk=_p(self.w_uk) if q_lat is not None else None, q_lat=_p(q_lat), T=T, act_dtype=ctx.act)
            S.check(lib.b2l_seq_latent_operands(C.byref(a), ctx.stream), "b2l_seq_latent_operands")
        else:
            cq = torch.empty((T, self.rq), dtype=h.dtype, device=dev)
            S.check(lib.b2l_seq_latent_prep(_p(proj), proj.shape[1], self.o_q, self.rq, _p(self.q_norm), _p(cq), self.o_kv, self.rk, _p(self.kv_norm),
                                            dr, _p(self.freq), self.rot_dims, int(self.interleaved), self.rot_mult, self.eps, _p(ctx.meta), _p(cache),
                                            self.max_positions, T, ctx.act, ctx.stream), "b2l_seq_latent_prep")
            q = linear(cq, self.w_uq)                                               # [T, H * (dim + rot_dim)]
            if expanded:
                self._rope(q, 0, dn, dq, q32, ctx)
            else:
                qn = q.view(T, H, dq)[:, :, :dn].transpose(0, 1)                     # [H, T, dim]
                if dr:
                    self._rope(q, dn, 0, dr, q_rot, ctx)
        if not expanded and q_lat is None:
            q_lat = torch.bmm(qn, self.w_uk) if f32 else torch.bmm(qn, self.w_uk, out_dtype=torch.float32)
        return gate, q32, q_lat, q_rot

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        lib, T, dev, H, dn, dv, dr = S.lib(), ctx.T, h.device, self.H, self.dn, self.dv, self.dr
        cache, Kd, dq = ctx.state[self.name + ".kv"], self.rk + self.dr, self.dn + self.dr
        n_pos = None if ctx.pos_hint is None or ctx.slot_hint is None else ctx.pos_hint + T
        expanded = n_pos is not None and T >= self.expand_from and n_pos * H * (dv + dn) <= self.expand_limit
        gate, q32, q_lat, q_rot = self._queries(h, cache, ctx, expanded)
        gp, ldg = (_p(*gate), gate[0].shape[1]) if gate is not None else (None, 0)
        shared_b = dict(key_b=_p(cache, self.rk), ldkb=Kd, slot_stride_b=self.max_positions * Kd, n_b=dr)
        att = torch.empty((T, H * dv), dtype=h.dtype, device=dev)
        if expanded:                            # [value_h | key_h] of positions 0 .. n_pos-1 from the cached latents, one product
            lo = max(0, ctx.pos_hint - self.window + 1) if self.window else 0       # the first position any query of the portion sees
            kv = linear(cache[ctx.slot_hint, lo:n_pos, :self.rk], self.w_expand)     # [n_pos - lo, H * (vdim + dim)]: row j - lo is position j
            self._attend(ctx, att, dv, self._splits(ctx, 1), q_a=_p(q32), ldqa_t=H * dq, ldqa_h=dq, q_b=_p(q32, dn), ldqb_t=H * dq, ldqb_h=dq,
                         key_a=_p(kv, -lo * H * (dv + dn)), ldka=H * (dv + dn), hska=dv + dn, slot_stride_a=0, n_a=dv + dn, score_off=dv, heads_per_group=1,
                         gate=gp, ldg=ldg, **shared_b)
            return linear(att, self.w_o)
        latent = dict(q_a=_p(q_lat), ldqa_t=self.rk, ldqa_h=T * self.rk, q_b=_p(q_rot), ldqb_t=H * max(dr, 1), ldqb_h=max(dr, 1), key_a=_p(cache), ldka=Kd, hska=0,
                      slot_stride_a=self.max_positions * Kd, n_a=self.rk, score_off=0, heads_per_group=H, **shared_b)
        splits = self._splits(ctx, H)
        if T <= FEW_TOKENS:                     # merge of the splits, W_uv and gate in one launch
            work = self._attend(ctx, None, self.rk, splits, **latent)
            S.check(lib.b2l_seq_latent_up(_p(work), _p(self.sink), _p(self.w_uv), gp, ldg, _p(att), H * dv, T, H, self.rk, dv, splits, ctx.act, ctx.stream),
                    "b2l_seq_latent_up")
            return linear(att, self.w_o)
        o_lat = torch.empty((T, H * self.rk), dtype=h.dtype, device=dev)
        self._attend(ctx, o_lat, self.rk, splits, **latent)
        v = torch.bmm(o_lat.view(T, H, self.rk).transpose(0, 1), self.w_uv.transpose(1, 2))      # [H, T, vdim]
        S.check(lib.b2l_seq_head_gate(_p(v), dv, T * dv, gp, ldg, _p(att), H * dv, T, H, dv, ctx.act, ctx.stream), "b2l_seq_head_gate")
        return linear(att, self.w_o)


# ------------------------------------------------------------------------------------------------ retention
class RetentionMixer:
    """Linear attention with one fixed decay per head, no softmax and no denominator:

        q, k rotated by position (first rot.dims entries of each head; entry i with entry i + dims/2), k times dim^-1/2
        S_t = decay_h S_(t-1) + k_t v_t^T;  o_t = S_t^T q_t
        y = W_o (concat_h(o_t,h / rms(o_t,h)) * silu(W_g h))

    State per sequence: S (f32, heads x vdim x dim), zero at the start."""

    def __init__(self, name: str, W: Dict[str, torch.Tensor], p: str, *, heads: int, dim: int, vdim: int, decay: List[float], eps: float,
                 rot: Optional[dict], interleaved: bool = False) -> None:
        self.name, self.H, self.K, self.V, self.eps, self.interleaved = name, heads, dim, vdim, eps, bool(interleaved)
        if len(decay) != heads:
            raise ValueError(f"retention: {len(decay)} decays for {heads} heads")
        self.w_in, (self.o_q, self.o_k, self.o_v, self.o_g) = stack_rows([W[p + "q"], W[p + "k"], W[p + "v"], W[p + "g"]])
        assert W[p + "q"].shape[0] == heads * dim and W[p + "v"].shape[0] == heads * vdim and W[p + "g"].shape[0] == heads * vdim
        self.w_o = W[p + "o"].contiguous()
        dev = self.w_o.device
        self.decay = torch.tensor([float(d) for d in decay], dtype=torch.float32, device=dev)
        self.ones = torch.ones(vdim, dtype=self.w_o.dtype, device=dev)
        self.rot_dims, self.freq = 0, None
        if rot:
            self.rot_dims = int(rot["dims"])
            f, _ = rope_frequencies(self.rot_dims, float(rot["base"]), rot.get("scaling"))
            self.freq = f.to(dev)

    def state_specs(self) -> Dict[str, StateSpec]:
        return {self.name + ".S": StateSpec((self.H, self.V, self.K), torch.float32)}

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        lib, T, dev, H, K, V = S.lib(), ctx.T, h.device, self.H, self.K, self.V
        proj = linear(h, self.w_in)
        ld, f32in = proj.shape[1], int(proj.dtype == torch.float32)
        qkv = torch.empty((T, 2 * H * K + H * V), dtype=torch.float32, device=dev)
        n = qkv.shape[1]
        for off_in, off_out, mult in ((self.o_q, 0, 1.0), (self.o_k, H * K, K ** -0.5)):
            S.check(lib.b2l_seq_rope(_p(proj, off_in), ld, f32in, _p(self.freq), self.rot_dims, int(self.interleaved), 0, mult, 1.0, _p(ctx.meta),
                                     _p(qkv, off_out), n, 1, T, H, K, K, K, ctx.act, ctx.stream), "b2l_seq_rope")
        S.check(lib.b2l_seq_cast_f32(_p(proj, self.o_v), ld, _p(qkv, 2 * H * K), n, T, H * V, ctx.act, ctx.stream), "b2l_seq_cast_f32")
        o = torch.empty((T, H * V), dtype=torch.float32, device=dev)
        _scan(ctx, q=_p(qkv), ldq=n, k=_p(qkv, H * K), ldk=n, v=_p(qkv, 2 * H * K), ldv=n, q_mult=1.0, decay=_p(self.decay), ldd=0,
              per_channel=False, state=ctx.state[self.name + ".S"], out=_p(o), ldo=H * V, heads=H, qk_heads=H, K=K, V=V)
        y = torch.empty((T, H * V), dtype=h.dtype, device=dev)
        S.check(lib.b2l_seq_group_norm_gate(_p(o), H * V, _p(self.ones), 1, _p(proj, self.o_g), ld, S.ACT_SILU, 0, self.eps, 1.0, _p(y), H * V, T,
                                            H * V, V, ctx.act, ctx.stream), "b2l_seq_group_norm_gate")
        return linear(y, self.w_o)


# ------------------------------------------------------------------------------------------------ routed experts
class MoEFeedForward:
    """y = sum over the chosen experts of weight_e * expert_e(h).

        s = softmax(W_router h) over all experts, or sigmoid of each logit (`score`), f32;  choice = s + correction
        (steers the choice only); experts form `groups` equal groups of neighbours; a group is worth the sum of its
        `group_top` largest choice scores (1: its best); only experts of the `keep` best groups can be chosen; the `top`
        largest choice scores win;  weight = s / (sum of the chosen s + 1e-20) when `renormalize`, else s itself, times
        `weight_scale`;  or (`score` = "chosen_softmax") the choice is made on the logits z = W_router h + bias and the weights
        are the softmax of z over the chosen experts
        expert e < experts: W_down unit(W_gate x, W_up x) with unit(a, b) = act(a) * b, or the clamped unit
        min(a, limit) * sigmoid(1.702 min(a, limit)) * (clamp(b, -limit, limit) + 1) (`act` = "clamped_swish");
        x = h and the weight scales the expert's output, or (`weight_on` = "input") x = weight * h and the outputs are
        summed unweighted;  the last `identity` outputs of the router: h itself
        with `shared_ff` one more expert of that size runs on every token's h and is added unweighted

    A few tokens (also the captured single-token step) run with the expert index read on the device; longer portions
    sort the assignments by expert and run one pair of products per expert that received tokens."""

    SMALL = FEW_TOKENS
    grouped = True        # bf16, 16-byte rows: the library's grouped product instead of one product per expert

    SCORES = {"softmax": S.SCORE_SOFTMAX, "sigmoid": S.SCORE_SIGMOID, "chosen_softmax": S.SCORE_CHOSEN_SOFTMAX}

    def __init__(self, W: Dict[str, torch.Tensor], p: str, *, experts: int, identity: int, top: int, groups: int, keep: int, ff: int,
                 act: str = "silu", limit: float = 0.0, score: str = "softmax", renormalize: bool = True, weight_on: str = "output",
                 group_top: int = 1, weight_scale: float = 1.0, shared_ff: int = 0) -> None:
        self.group_top, self.weight_scale = int(group_top), float(weight_scale)
        if self.group_top < 1:
            raise ValueError("routed experts: a group's score needs at least its best member")
        self.E, self.I, self.top, self.groups, self.keep, self.ff = int(experts), int(identity), int(top), int(groups), int(keep), int(ff)
        self.n = self.E + self.I
        if self.n % self.groups or not (1 <= self.keep <= self.groups) or self.keep * (self.n // self.groups) < self.top:
            raise ValueError("routed experts: groups / keep / top do not fit the expert count")
        self.act, self.limit = GatedMLP.ACTS[act], float(limit)
        if self.act == S.ACT_CLAMPED_SWISH and not self.limit > 0.0:
            raise ValueError("routed experts: the clamped unit needs a positive limit")
        if score not in self.SCORES or weight_on not in ("output", "input"):
            raise ValueError(f"routed experts: unknown score function {score!r} or weight placement {weight_on!r}")
        self.score, self.renorm, self.weight_input = self.SCORES[score], int(bool(renormalize)), int(weight_on == "input")
        if score == "chosen_softmax" and not renormalize:
            raise ValueError("routed experts: a softmax over the chosen logits sums to one")
        if self.weight_input and self.I:
            raise ValueError("routed experts: identity experts with weights on the input are not built")
        self.w_router = W[p + "router"].contiguous()
        assert self.w_router.shape[0] == self.n, "routed experts: the router does not have experts + identity outputs"
        bias = p + ("router.b" if score == "chosen_softmax" else "correction")      # the kernels' `correction`: of the choice, or of the logits
        self.correction = W[bias].to(torch.float32).contiguous() if bias in W else None
        dev, dt = self.w_router.device, W[p + "router"].dtype
        if self.E:
            self.w_gu = torch.stack([torch.cat([W[f"{p}e{e}.gate"], W[f"{p}e{e}.up"]], dim=0) for e in range(self.E)]).contiguous()
            self.w_down = torch.stack([W[f"{p}e{e}.down"] for e in range(self.E)]).contiguous()
            assert self.w_gu.shape[1] == 2 * self.ff, "routed experts: expert size does not fit"
        else:
            self.w_gu = self.w_down = torch.zeros(0, dtype=dt, device=dev)
        self.shared: Optional[GatedMLP] = None
        if shared_ff:
            self.shared = GatedMLP(W[p + "shared.gate"], W[p + "shared.up"], W[p + "shared.down"], act=act, limit=limit)
            assert self.shared.ff == int(shared_ff), "routed experts: the shared expert does not have its size"
        self.last_idx: Optional[torch.Tensor] = None       # the routing of the last call (tests, diagnostics)

    def state_specs(self) -> Dict[str, StateSpec]:
        return {}

    def route(self, h: torch.Tensor, ctx: StepContext) -> Tuple[torch.Tensor, torch.Tensor]:
        lib, T, dev, D = S.lib(), ctx.T, h.device, h.shape[1]
        if torch.backends.cuda.matmul.allow_tf32:
            raise RuntimeError("router logits need true 32-bit products: torch.backends.cuda.matmul.allow_tf32 is on")
        idx = torch.empty((T, self.top), dtype=torch.int32, device=dev)
        wgt = torch.empty((T, self.top), dtype=torch.float32, device=dev)
        if T <= self.SMALL:        # a few tokens: the logits and the routing in one launch
            S.check(lib.b2l_seq_moe_route_fused(_p(h), D, _p(self.w_router), _p(self.correction), D, self.n, self.groups, self.keep, self.top,
                                                self.score, self.renorm, self.group_top, self.weight_scale, _p(idx), _p(wgt), T, ctx.act,
                                                ctx.stream), "b2l_seq_moe_route_fused")
            self.last_idx = idx
            return idx, wgt
        # f32 logits: bf16 activations and router weights are exact in f32, the product keeps its f32 accumulator
        z = linear_f32(h, self.w_router)
        S.check(lib.b2l_seq_moe_route(_p(z), self.n, _p(self.correction), self.n, self.groups, self.keep, self.top, self.score, self.renorm,
                                      self.group_top, self.weight_scale, _p(idx), _p(wgt), T, ctx.stream), "b2l_seq_moe_route")
        self.last_idx = idx
        return idx, wgt

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        lib, T, dev, D, E, top, ff = S.lib(), ctx.T, h.device, h.shape[1], self.E, self.top, self.ff
        idx, wgt = self.route(h, ctx)
        y = torch.empty((T, D), dtype=h.dtype, device=dev)
        N = T * top
        if T <= self.SMALL or E == 0:
            sh = self.shared
            mid = torch.empty((N * ff + (T * sh.ff if sh is not None else 0),), dtype=h.dtype, device=dev)
            S.check(lib.b2l_seq_moe_experts_small(_p(h), D, _p(self.w_gu) if E else None, _p(self.w_down) if E else None, _p(idx), _p(wgt), _p(mid),
                                                  _p(y), D, T, D, ff, E, top, self.act, self.limit, self.weight_input, _p(sh.w_in) if sh is not None else None,
                                                  _p(sh.w_down) if sh is not None else None, sh.ff if sh is not None else 0, ctx.act, ctx.stream),
                    "b2l_seq_moe_experts_small")
            return y
        y_shared = self.shared.forward(h, ctx) if self.shared is not None else None
        meta = torch.empty((2 * (E + 1) + 2 * N,), dtype=torch.int32, device=dev)
        offsets, cursor, perm, inv = meta[:E + 1], meta[E + 1:2 * E + 2], meta[2 * E + 2:2 * E + 2 + N], meta[2 * E + 2 + N:]
        S.check(lib.b2l_seq_moe_sort(_p(idx), N, E, _p(offsets), _p(cursor), _p(perm), _p(inv), ctx.stream), "b2l_seq_moe_sort")
        xg = torch.empty((N + 8, D), dtype=h.dtype, device=dev)       # rows past the last group's end are never read
        S.check(lib.b2l_seq_moe_gather(_p(h), D, _p(perm), _p(offsets, E), _p(wgt) if self.weight_input else None, top, _p(xg), N, D, ctx.act,
                                       ctx.stream), "b2l_seq_moe_gather")
        gu = torch.empty((N, 2 * ff), dtype=h.dtype, device=dev)
        mid = torch.empty((N + 8, ff), dtype=h.dtype, device=dev)
        if self.grouped and h.dtype == torch.bfloat16 and D % 8 == 0 and ff % 8 == 0:
            # the library's grouped product: every expert's rows in one launch, group ends read on the device
            ends = offsets[1:]
            gu = F.grouped_mm(xg, self.w_gu.transpose(1, 2), offs=ends)
            S.check(lib.b2l_seq_gated_act(_p(gu), 2 * ff, _p(mid), N, ff, self.act, self.limit, ctx.act, ctx.stream), "b2l_seq_gated_act")
            yg = F.grouped_mm(mid, self.w_down.transpose(1, 2), offs=ends)
        else:
            off = offsets.cpu().tolist()                               # the one host read of a long portion
            for e in range(E):
                if off[e + 1] > off[e]:
                    torch.mm(xg[off[e]:off[e + 1]], self.w_gu[e].t(), out=gu[off[e]:off[e + 1]])
            S.check(lib.b2l_seq_gated_act(_p(gu), 2 * ff, _p(mid), off[E], ff, self.act, self.limit, ctx.act, ctx.stream), "b2l_seq_gated_act")
            yg = torch.empty((N, D), dtype=h.dtype, device=dev)
            for e in range(E):
                if off[e + 1] > off[e]:
                    torch.mm(mid[off[e]:off[e + 1]], self.w_down[e].t(), out=yg[off[e]:off[e + 1]])
        S.check(lib.b2l_seq_moe_combine(_p(yg), _p(inv), None if self.weight_input else _p(wgt), _p(h), D, _p(y_shared), D, _p(y), D, T, D, top,
                                        ctx.act, ctx.stream), "b2l_seq_moe_combine")
        return y
