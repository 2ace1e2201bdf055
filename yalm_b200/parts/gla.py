"""Gated linear attention (Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient
Training"), H heads of key size dk and value size dv:

    q, k = Wq h, Wk h  [H, dk];   v = Wv h  [H, dv];   q times dk^-1/2
    alpha = sigmoid(Wa2 (Wa1 h) + b)^(1/tau)              a decay per head and key channel
    S <- diag(alpha) S + k v^T;   o = S^T q               the read-out sees the current token
    out = Wo (n(o) w silu(Wg h))                          n: each head over its own root mean square

The state is a fixed-size cache need per sequence (float32 [H, dv, dk], a column's rows neighbours).  The five
projections that read h are one product; the decay's second half, a few multiply-adds per channel, is formed in
32 bits where the decay is.  Decays, state, output norm and gate are 32-bit.
"""
from __future__ import annotations

import torch

from ..cache import CacheNeed
from ..csrc import ops
from ..weights import TensorNeed
from .base import register_mixer
from .linear import matmul_partials, stacked_rows


@register_mixer("gated_linear_attention")
class GatedLinearAttention:
    def __init__(self, params: dict, rt):
        self.rt = rt
        self.D = int(params["hidden_size"])
        self.H = int(params["num_heads"])
        self.dk = int(params["key_dim"])
        self.dv = int(params["value_dim"])
        self.rank = int(params["decay_rank"])
        self.tau = float(params["tau"])
        self.eps = float(params["eps"])
        if min(self.H, self.dk, self.dv, self.rank) <= 0 or self.dk > 256 or self.rank > 1024 or self.dv > 1024 \
                or not self.tau > 0:
            raise ValueError(f"gated_linear_attention: {self.H} heads of {self.dk} (up to 256) and {self.dv} (up to "
                             f"1,024), decay rank {self.rank} (up to 1,024), tau {self.tau}")
        self.w_in = self.w_o = self.w_a2 = self.bias = self.norm = None

    def tensor_needs(self):
        H, dk, dv, D = self.H, self.dk, self.dv, self.D
        return {"q": TensorNeed((H * dk, D)), "k": TensorNeed((H * dk, D)), "v": TensorNeed((H * dv, D)),
                "g": TensorNeed((H * dv, D)), "a1": TensorNeed((self.rank, D)), "a2": TensorNeed((H * dk, self.rank)),
                "a2.b": TensorNeed((H * dk,), init="around_zero"), "norm": TensorNeed((dv,), init="ones"),
                "o": TensorNeed((D, H * dv))}

    def bind(self, tensors) -> None:
        rt = self.rt
        w, self.cols = stacked_rows([tensors[k] for k in ("q", "k", "v", "g", "a1")])
        self.w_in, self.w_o = rt.matrix(w), rt.matrix(tensors["o"])
        self.w_a2 = rt.vector(tensors["a2"].t())
        self.bias = rt.vector(tensors["a2.b"])
        self.norm = rt.vector(tensors["norm"]).repeat(self.H).contiguous()

    def cache_need(self) -> CacheNeed:
        return CacheNeed("state", state_shape=(self.H, self.dv, self.dk), state_dtype=torch.float32)

    def cache_read_bytes(self, contexts, element_size: int) -> int:
        return 2 * len(contexts) * self.H * self.dk * self.dv * 4        # the state, read and written

    def flops(self, q_lens, past) -> float:
        n = sum(q_lens)
        H, dk, dv, D = self.H, self.dk, self.dv, self.D
        return 2.0 * n * ((2 * H * dk + 2 * H * dv + self.rank) * D + H * dk * self.rank + D * H * dv) + 4.0 * n * H * dk * dv

    def forward(self, h, batch, stream, view, shared: bool = False):
        if shared:
            raise RuntimeError("a recurrent state cannot be read by another run entry")
        rt, H, dk, dv = self.rt, self.H, self.dk, self.dv
        n = batch.n_tokens
        z, S = matmul_partials(rt, h, self.w_in, "gla_in")
        cq, ck, cv, cg, ca = self.cols
        act = rt.buffer("gla_act", (n, 3 * H * dk + H * dv), torch.float32)
        marks = rt.buffer("gla_marks", (n, H), torch.int32)
        o = rt.buffer("gla_o", (n, H * dv), torch.float32)
        ops.gla(z, S, (cq, ck, cv, ca), self.rank, self.w_a2, self.bias, self.tau, act, marks, batch, view.state, o,
                H, dk, dv)
        out = rt.buffer("gla_normed", (n, H * dv), rt.dtype)
        ops.gated_heads(o, self.norm, z, S, cg, out, H, dv, self.eps, silu=True)
        stream.add_linear(out, self.w_o)
        return None
