"""A matrix memory with exponential gates and a running maximum (the mLSTM of xLSTM).

    q = Wq h / sqrt(head_dim),  k = Wk h          [heads, head_dim]
    v = Wv h                                      [heads, v_head_dim]
    i = cap tanh((Wi h + bi) / cap),  f = log sigmoid(cap tanh((Wf h + bf) / cap))        log gates, one a head
    m_t = max(f + m_(t-1), i)                     starts at 0
    S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k v^T;  n_t the same with k alone
    o = S_t^T q / (max(|n_t . q|, e^(-m_t)) + MEMORY_EPS)
    out = Wo (rms_head(o) * norm * sigmoid(Wg h))

What a sequence keeps, whatever its length: S, n and m (32-bit).  One stacked product makes q | k | v | gate | i | f from the layer's
input; the gates' columns leave it in 32-bit (for prompts, whose rows are otherwise bfloat16, by a small product of their own over the
same stacked weight).  Single tokens: one kernel (gates, update, result, divisor).  Anything longer: the gates' running maximum along
each sequence, then the recurrence by blocks of 64 tokens side by side.  One kernel divides, normalises and gates; the output product is
the one every mixer uses.  From the projections on everything is 32-bit."""
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

MEMORY_EPS = 1e-6              # beside the divisor

TENSOR_NAMES = {"q": "q_proj", "k": "k_proj", "v": "v_proj", "gate": "g_proj", "i": "i_gate", "f": "f_gate", "o": "o_proj",
                "out_norm": "out_norm"}


@register_mixer("mlstm")
class MatrixLSTM(Mixer):
    graph_safe = True

    def __init__(self, spec: MixerSpec, hidden: int, env: BuildEnv):
        p = spec.params
        self.env = env
        self.hidden = hidden
        self.heads = int(p["n_heads"])
        self.hd = int(p["head_dim"])
        self.vd = int(p.get("v_head_dim") or self.hd)
        self.cap = float(p["gate_cap"])
        self.norm_eps = float(p.get("out_norm_eps", 1e-6))
        self.mem_eps = float(p.get("memory_eps", MEMORY_EPS))
        if min(self.heads, self.hd, self.vd) <= 0 or self.hd > 4096:
            raise ConfigError("mlstm: heads and head sizes must be positive (queries and keys of at most 4096)")
        if not self.cap > 0:
            raise ConfigError(f"mlstm: gate_cap must be positive, found {self.cap}")
        if spec.position.kind != "none":
            raise ConfigError("mlstm: a position encoding inside the mixer is not part of it")
        try:
            self.names = n = tensor_names(p, TENSOR_NAMES)
        except ValueError as e:
            raise ConfigError(f"mlstm: {e}") from None
        qk, vw = self.heads * self.hd, self.heads * self.vd
        self.inner = vw
        self.q_off, self.k_off, self.v_off, self.g_off, self.i_off, self.f_off = 0, qk, 2 * qk, 2 * qk + vw, 2 * qk + 2 * vw, 2 * qk + 2 * vw + self.heads
        self.proj = Linear([n[r] for r in ("q", "k", "v", "gate", "i", "f")], [qk, qk, vw, vw, self.heads, self.heads], hidden,
                           [n["i"], n["f"]], env)
        self.o = Linear([n["o"]], [hidden], vw, False, env)
        self.norm_w: Optional[torch.Tensor] = None
        self.main = self.gates = None           # the stack's rows as two products (see ``_project``)

    def cache_requirement(self):
        return BundleRequirement.of(StateRequirement((self.heads, self.hd, self.vd), torch.float32),
                                    norm=StateRequirement((self.heads, self.hd), torch.float32),
                                    peak=StateRequirement((self.heads, 2), torch.float32))

    def declare(self, prefix: str) -> List[TensorDecl]:
        return self.proj.declare(prefix) + self.o.declare(prefix) + \
            [TensorDecl(f"{prefix}{self.names['out_norm']}.weight", (self.inner,), "norm")]

    def load(self, tensors: Dict[str, torch.Tensor], prefix: str) -> None:
        self.proj.load(tensors, prefix)
        self.proj.pad_rows(8)
        self.o.load(tensors, prefix)
        self.norm_w = tensors[f"{prefix}{self.names['out_norm']}.weight"].float().contiguous()
        # the same rows once more, without a copy: what may be rounded, and the gates
        self.main, self.gates = self.proj.rows(0, self.i_off, "q+k+v+g"), self.proj.rows(self.i_off, self.proj.n, "i+f")

    def weight_bytes(self) -> int:
        return self.proj.weight_bytes() + self.o.weight_bytes()

    def workspace_bytes(self, n_tokens: int) -> int:
        esz = 4 if self.env.mode == "float32" else 2
        parts = 8 if n_tokens <= 128 else 1
        blocks = (n_tokens // kernels.MLSTM_BLOCK + 8) * self.heads * (self.hd * (self.vd + 1) + kernels.MLSTM_BLOCK ** 2) * 4 if n_tokens > 1 else 0
        return n_tokens * (self.proj.n * max(esz, 4 * parts if parts > 1 else esz) + self.inner * (4 + esz) + self.hidden * 4 * parts
                           + 16 * self.heads) + blocks

    def cost(self, q_lens, kv_lens):
        from ..profile import cost as C
        T = sum(q_lens)
        esz = 4 if self.env.mode == "float32" else 2
        live = sum(1 for n in q_lens if n > 0)
        parts = [self.proj.cost(T), self.o.cost(T), C.mlstm(T, live, self.heads, self.hd, self.vd, esz)]
        return sum(p[0] for p in parts), sum(p[1] for p in parts)

    def _project(self, xn, T):
        """(projection rows, the rows that hold the gates, the gates' columns there); the gates' are 32-bit."""
        if self.env.mode == "float32" or not self.proj.one_piece(xn, T):
            proj = self.proj.forward_auto(xn, T)
            if proj.dtype == torch.float32:
                return proj, proj, self.i_off, self.f_off
        gates = self.gates.forward_delta(xn, T)
        proj = torch.empty((T, self.main.n), dtype=xn.dtype, device=xn.device)
        return self.main.forward(xn, proj, T), gates, 0, self.heads

    def forward(self, xn, batch, view):
        T = batch.n_tokens
        dev, act = self.env.device, self.env.act_dtype
        if isinstance(xn, DeferredNorm):
            xn = xn.materialize()
        proj, gates, i_off, f_off = self._project(xn, T)
        o = torch.empty((T, self.inner), dtype=torch.float32, device=dev)
        den = torch.empty((T, self.heads), dtype=torch.float32, device=dev)
        n, m = view.extras["norm"].state, view.extras["peak"].state
        if batch.is_decode:
            with scope(op="mlstm_step"):
                kernels.mlstm_step(proj, self.q_off, self.k_off, self.v_off, gates, i_off, f_off, self.cap, self.hd ** -0.5, self.mem_eps,
                                   self.heads, self.hd, self.vd, view.state, n, m, batch.seq_slot, batch.cu_q, batch.positions,
                                   batch.n_seqs, o, den)
        else:
            keep, add, em = (torch.empty((self.heads, T), dtype=torch.float32, device=dev) for _ in range(3))
            with scope(op="mlstm_gates"):
                kernels.mlstm_gates(gates, T, i_off, f_off, self.cap, self.heads, m, batch.seq_slot, batch.cu_q, batch.positions,
                                    batch.n_seqs, batch.max_q_len, keep, add, em)
            with scope(op="mlstm_blocks"):
                kernels.mlstm_blocks(proj, T, self.q_off, self.k_off, self.v_off, self.hd ** -0.5, self.mem_eps, self.heads, self.hd,
                                     self.vd, keep, add, em, view.state, n, batch.seq_slot, batch.cu_q, batch.n_seqs, o, den)
        y = torch.empty((T, self.inner), dtype=act, device=dev)
        with scope(op="norm_gate"):
            kernels.group_norm_gate(o, proj, self.g_off, self.norm_w, self.norm_eps, self.heads, "sigmoid", y, batch.slot_of_token, T,
                                    divisor=den)
        return self.o.forward_delta(y, T)
