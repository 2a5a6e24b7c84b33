"""The gated delta rule: a state per head that decays and is corrected, token by token, towards v along k.

    q, k, v <- silu(causal convolution over the last ``conv_taps`` tokens of W. h, per channel)
    q <- q / |q| * head_dim^(-1/2),  k <- k / |k|      per key head, |x| = sqrt(sum x^2 + UNIT_EPS); head n uses n // (heads / kv_heads)
    beta = sigmoid(Wb h)                               one a head
    g = exp(-exp(A_log) softplus(z + dt_bias))         z = Wa h, one a head (``decay`` "per_head"), or
                                                       z = Wa2 (Wa1 h), one a head and key channel ("per_channel")
    S <- g S;  w = beta (v - S^T k);  S <- S + k w^T;  o = S^T q         S [head_dim, v_head_dim] per head, 32-bit
    out = Wo (o / rms(o) * norm * gate)                rms per head; gate = silu(Wg h) ("silu") or sigmoid(Wg2 (Wg1 h)) ("sigmoid_low_rank")

What a sequence keeps, whatever its length: the state (stored [heads, v_head_dim, head_dim]: a column of S is one run of
memory) and the convolution's last conv_taps - 1 inputs, both 32-bit.  One stacked product makes every column block from the
layer's input (of a narrow product W2 (W1 h) the inner values are among them; the outer product is a tensor-core product for
prompts and a small kernel for few tokens); one kernel prepares the recurrence's inputs in 32-bit; one kernel carries the
step's tokens through the recurrence with the state in registers (token after token for single tokens and short pieces; four at
a time for prompts, from vectors that one more kernel prepares); one kernel normalises and gates.  The inner ranks of narrow products are sizes of the tensors, given as ``decay_rank`` and
``gate_rank``.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import kernels
from ..cache.requirements import BundleRequirement, StateRequirement
from ..config.specs import MixerSpec, tensor_names
from ..errors import ConfigError
from ..profile import scope
from ..weights.decl import TensorDecl
from .base import BuildEnv, DeferredNorm, Mixer, register_mixer
from .linear import Linear

UNIT_EPS = 1e-6                # under the root of a unit vector's length

CHUNKS_MIN_TOKENS = 16         # a step whose longest sequence brings more tokens runs the recurrence four tokens at a time

LOW_RANK_MAX_TOKENS = 64       # up to it the outer half of a narrow product is the small kernel for few tokens

TENSOR_NAMES = {"q": "q_proj", "k": "k_proj", "v": "v_proj", "o": "o_proj", "q_conv": "q_conv", "k_conv": "k_conv", "v_conv": "v_conv",
                "beta": "b_proj", "decay": "a_proj", "decay_in": "a_in", "decay_out": "a_out", "a_log": "A_log", "dt_bias": "dt_bias",
                "gate": "g_proj", "gate_in": "g_in", "gate_out": "g_out", "norm": "o_norm"}

DECAYS = ("per_head", "per_channel")
GATES = ("silu", "sigmoid_low_rank")


@register_mixer("gated_delta")
class GatedDelta(Mixer):
    graph_safe = True

    def __init__(self, spec: MixerSpec, hidden: int, env: BuildEnv):
        p = spec.params
        self.env = env
        self.hidden = hidden
        self.heads = int(p["n_heads"])
        self.kv = int(p.get("n_kv_heads") or self.heads)
        self.hd = int(p["head_dim"])
        self.vd = int(p.get("v_head_dim") or self.hd)
        self.taps = int(p.get("conv_taps", 1))
        self.decay = p.get("decay", "per_head")
        self.gate = p.get("gate", "silu")
        self.norm_eps = float(p.get("out_norm_eps", 1e-6))
        self.unit_eps = float(p.get("unit_eps", UNIT_EPS))
        if min(self.heads, self.kv, self.hd, self.vd) <= 0 or self.heads % self.kv:
            raise ConfigError(f"gated_delta: {self.heads} heads cannot share {self.kv} query/key heads of {self.hd} (values of {self.vd})")
        if self.hd > kernels.DELTA_MAX_DIM:
            raise ConfigError(f"gated_delta: heads of {self.hd} are not built (at most {kernels.DELTA_MAX_DIM})")
        if not 1 <= self.taps <= kernels.DELTA_MAX_TAPS:
            raise ConfigError(f"gated_delta: a convolution of {self.taps} taps is not built (1 to {kernels.DELTA_MAX_TAPS})")
        if self.decay not in DECAYS or self.gate not in GATES:
            raise ConfigError(f"gated_delta: decay is one of {DECAYS} and gate one of {GATES}, found {self.decay!r} and {self.gate!r}")
        if spec.position.kind != "none":
            raise ConfigError("gated_delta: a position encoding inside the mixer is not part of it")
        self.per_channel = self.decay == "per_channel"
        self.narrow_gate = self.gate == "sigmoid_low_rank"
        self.decay_rank = int(p.get("decay_rank") or 0) if self.per_channel else 0
        self.gate_rank = int(p.get("gate_rank") or 0) if self.narrow_gate else 0
        for need, rank, what in ((self.per_channel, self.decay_rank, "decay_rank"), (self.narrow_gate, self.gate_rank, "gate_rank")):
            if need and rank <= 0:
                raise ConfigError(f"gated_delta: {what} (the inner size of a narrow product) is not known")
        try:
            self.names = n = tensor_names(p, TENSOR_NAMES)
        except ValueError as e:
            raise ConfigError(f"gated_delta: {e}") from None
        self.kd, self.inner = self.kv * self.hd, self.heads * self.vd
        self.channels = 2 * self.kd + self.inner                      # what the convolution sees: q | k | v
        # column blocks of the projection: q | k | v | gate (whole, or its inner values) | decay's inner values | decay | beta
        blocks = [("q", self.kd), ("k", self.kd), ("v", self.inner),
                  ("gate_in", self.gate_rank) if self.narrow_gate else ("gate", self.inner),
                  ("decay_in", self.decay_rank) if self.per_channel else ("decay", self.heads), ("beta", self.heads)]
        self.off, at = {}, 0
        for role, width in blocks:
            self.off[role] = at
            at += width
        self.in_stems, self.in_outs = [n[r] for r, _ in blocks], [w for _, w in blocks]
        self.out_width = self.inner                                   # what the output product reads
        self.rows = kernels.DeltaRows(self.heads, self.kv, self.hd, self.vd, self.per_channel)
        self.proj = Linear(self.in_stems, self.in_outs, hidden, False, env)
        self.o = Linear([n["o"]], [hidden], self.inner, False, env)
        self.decay_out = Linear([n["decay_out"]], [self.heads * self.hd], self.decay_rank, False, env) if self.per_channel else None
        self.gate_out = Linear([n["gate_out"]], [self.inner], self.gate_rank, False, env) if self.narrow_gate else None
        self.conv_w: Optional[torch.Tensor] = None        # float32 [taps, channels]
        self.dt_bias = self.a_log = self.norm_w = None
        self.result_factor = 1.0                          # a constant on the result, folded into the norm's weight at load time

    def cache_requirement(self):
        main = StateRequirement((self.heads, self.vd, self.hd), torch.float32)
        if self.taps == 1:
            return main
        return BundleRequirement.of(main, conv=StateRequirement((self.taps - 1, self.channels), torch.float32))

    # ---- tensors ----------------------------------------------------------------------------------
    def _small(self, prefix: str):
        n = self.names
        return [(f"{prefix}{n['q_conv']}.weight", (self.kd, self.taps), "matrix"), (f"{prefix}{n['k_conv']}.weight", (self.kd, self.taps), "matrix"),
                (f"{prefix}{n['v_conv']}.weight", (self.inner, self.taps), "matrix"), (f"{prefix}{n['a_log']}.weight", (self.heads,), "norm"),
                (f"{prefix}{n['dt_bias']}.weight", (self.heads * self.hd if self.per_channel else self.heads,), "norm"),
                (f"{prefix}{n['norm']}.weight", (self.vd,), "norm")]

    def declare_inner(self, prefix: str) -> List[TensorDecl]:
        """The tensors beside the input and the output product."""
        out = [TensorDecl(name, shape, role) for name, shape, role in self._small(prefix)]
        for lin in (self.decay_out, self.gate_out):
            if lin is not None:
                out += lin.declare(prefix)
        return out

    def declare(self, prefix: str) -> List[TensorDecl]:
        return self.proj.declare(prefix) + self.o.declare(prefix) + self.declare_inner(prefix)

    def load_inner(self, tensors: Dict[str, torch.Tensor], prefix: str) -> None:
        names = [name for name, _, _ in self._small(prefix)]
        q, k, v, a_log, dt_bias, norm = (tensors[x].float() for x in names)      # 32-bit: they enter the recurrence
        self.conv_w = torch.cat([q, k, v], dim=0).t().contiguous()
        self.a_log, self.dt_bias = a_log.contiguous(), dt_bias.contiguous()
        self.norm_w = (norm * self.result_factor).repeat(self.heads).contiguous()
        for lin in (self.decay_out, self.gate_out):
            if lin is not None:
                lin.load(tensors, prefix)

    def load(self, tensors: Dict[str, torch.Tensor], prefix: str) -> None:
        self.proj.load(tensors, prefix)
        self.proj.pad_rows(8)
        self.o.load(tensors, prefix)
        self.load_inner(tensors, prefix)

    # ---- accounts -----------------------------------------------------------------------------------
    def inner_bytes(self) -> int:
        n = sum(lin.weight_bytes() for lin in (self.decay_out, self.gate_out) if lin is not None)
        return n + 4 * (self.channels * self.taps + 2 * self.heads + self.inner)

    def weight_bytes(self) -> int:
        return self.proj.weight_bytes() + self.o.weight_bytes() + self.inner_bytes()

    def inner_workspace(self, n_tokens: int) -> int:
        esz = 4 if self.env.mode == "float32" else 2
        narrow = (self.heads * self.hd if self.per_channel else 0) + (self.inner if self.narrow_gate else 0)
        work = self.heads * (4 * (kernels.delta_padded_dim(self.hd) or 0) + kernels.DELTA_CHUNK_NUMBERS) if n_tokens > CHUNKS_MIN_TOKENS else 0
        return n_tokens * (4 * (self.rows.width + self.inner + narrow + work) + self.inner * esz)

    def workspace_bytes(self, n_tokens: int) -> int:
        esz = 4 if self.env.mode == "float32" else 2
        parts = 8 if n_tokens <= 128 else 1
        return n_tokens * (self.proj.n * max(esz, 4 * parts if parts > 1 else esz) + self.hidden * 4 * parts) + self.inner_workspace(n_tokens)

    def inner_cost(self, q_lens, kv_lens):
        from ..profile import cost as C
        T = sum(q_lens)
        live = sum(1 for n in q_lens if n > 0)
        parts = [C.delta_scan(T, live, self.heads, self.kv, self.hd, self.vd, self.per_channel)]
        parts += [lin.cost(T) for lin in (self.decay_out, self.gate_out) if lin is not None]
        return sum(p[0] for p in parts), sum(p[1] for p in parts)

    def cost(self, q_lens, kv_lens):
        T = sum(q_lens)
        parts = [self.proj.cost(T), self.o.cost(T), self.inner_cost(q_lens, kv_lens)]
        return sum(p[0] for p in parts), sum(p[1] for p in parts)

    # ---- the pass -----------------------------------------------------------------------------------
    def mix_rows(self, proj, batch, view, out=None):
        """The rows that the output product reads, from the layer's projection rows ([T, >= sum(in_outs)], or float32 partial sums
        [S, T, ..]).  ``out`` [T, out_width] (any row stride) receives them if given."""
        T = batch.n_tokens
        dev, act = self.env.device, self.env.act_dtype
        off = self.off
        # the outer halves of the narrow products
        z, gate, gate_off, gate_inner = proj[..., off.get("decay", 0):], proj, off.get("gate", 0), None
        if self.per_channel or self.narrow_gate:
            a, b = self.decay_out, self.gate_out
            if T <= LOW_RANK_MAX_TOKENS and max(self.decay_rank, self.gate_rank) <= kernels.LOW_RANK_MAX:
                both = [(off["decay_in"], a.weight) if a is not None else None, (off["gate_in"], b.weight) if b is not None else None]
                both = [x for x in both if x is not None]
                narrow = torch.empty((T, sum(w.shape[0] for _, w in both)), dtype=torch.float32, device=dev)
                with scope(op="narrow_products"):
                    kernels.low_rank(proj, T, both[0][0], both[0][1], *(both[1] if len(both) > 1 else (0, None)), narrow)
                if a is not None:
                    z = narrow[:, :a.n]
                if b is not None:
                    gate, gate_off = narrow, a.n if a is not None else 0
            else:
                inner = proj if proj.dim() == 2 else self._summed(proj, act)
                if a is not None:
                    z = torch.empty((T, a.n), dtype=torch.float32, device=dev)
                    a.forward(inner[:, off["decay_in"]:off["decay_in"] + self.decay_rank], z, T)
                gate_inner = inner
        u = torch.empty((T, self.rows.width), dtype=torch.float32, device=dev)
        kept = view.extras["conv"].state if self.taps > 1 else None
        with scope(op="delta_prep"):
            kernels.delta_prep(proj, T, off["q"], off["k"], off["v"], off["beta"], self.heads, self.kv, self.hd, self.vd, self.taps,
                               self.conv_w, kept, z, self.dt_bias, self.a_log, self.per_channel, self.unit_eps, self.hd ** -0.5,
                               batch.seq_slot, batch.cu_q, batch.n_seqs, batch.max_q_len, u, self.rows)
        o = torch.empty((T, self.inner), dtype=torch.float32, device=dev)
        with scope(op="delta_scan"):
            sizes = (self.rows, self.heads, self.kv, self.hd, self.vd, self.per_channel, view.state, batch.seq_slot, batch.cu_q, batch.n_seqs)
            dimp = kernels.delta_padded_dim(self.hd)
            if batch.max_q_len > CHUNKS_MIN_TOKENS and dimp is not None:
                vecs = torch.empty((self.heads, T, 3, dimp), dtype=torch.float32, device=dev)
                firsts = torch.empty((self.heads, T // 4 + batch.n_seqs, dimp + kernels.DELTA_CHUNK_NUMBERS), dtype=torch.float32, device=dev)
                kernels.delta_scan_chunks(u, T, *sizes, batch.max_q_len, o, vecs, firsts)
            else:
                kernels.delta_scan(u, T, *sizes, o)
        if gate_inner is not None and self.narrow_gate:
            gate, gate_off = torch.empty((T, self.inner), dtype=act, device=dev), 0
            self.gate_out.forward(gate_inner[:, off["gate_in"]:off["gate_in"] + self.gate_rank], gate, T)
        if out is None:
            out = torch.empty((T, self.inner), dtype=act, device=dev)
        with scope(op="norm_gate"):
            kernels.group_norm_gate(o, gate, gate_off, self.norm_w, self.norm_eps, self.heads, "sigmoid" if self.narrow_gate else "silu",
                                    out, batch.slot_of_token, T)
        return out

    @staticmethod
    def _summed(proj, act):
        """Partial sums as one result in the activations' type (a step whose product was split, with too many tokens for the
        small kernel)."""
        total = torch.zeros(proj.shape[1:], dtype=torch.float32, device=proj.device)
        kernels.residual_inject(total, proj)
        if act == torch.float32:
            return total
        out = torch.empty(total.shape, dtype=act, device=proj.device)
        kernels.cast(total, out)
        return out

    def forward(self, xn, batch, view):
        T = batch.n_tokens
        if isinstance(xn, DeferredNorm):
            xn = xn.materialize()
        return self.o.forward_delta(self.mix_rows(self.proj.forward_auto(xn, T), batch, view), T)
