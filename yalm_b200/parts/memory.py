"""The matrix memory of xLSTM ("mLSTM"; Beck et al., "xLSTM: Extended Long Short-Term Memory"), H heads of key
size dk and value size dv:

    q, k = Wq h, Wk h  [H, dk];   v = Wv h  [H, dv];   q times dk^-1/2
    i = cap tanh((Wi h + b_i) / cap),   f = logsigmoid(cap tanh((Wf h + b_f) / cap))      one each per head
    m' = max(f + m, i),  m from 0;   S <- e^(f + m - m') S + e^(i - m') k v^T,   n likewise with k alone
    o = S^T q / (max(|n.q|, e^-m') + 1e-6)
    out = Wo (n(o) w sigmoid(Wg h))                       n: each head over its own root mean square

S is the state of a state-space scan (``ops.ssd_scan``) whose decays and inputs are given, n one more column of
it.  Two fixed-size cache needs per sequence: S with n (float32 [H, columns, dk], columns = dv + 1 rounded up to
a multiple of four) and m (float32 [H]).  The six projections that read h are one product.  Gates, maxima,
decays, state, output norm and gate are 32-bit.
"""
from __future__ import annotations

import torch

from ..cache import CacheNeed
from ..csrc import ops
from ..weights import TensorNeed
from .base import register_mixer
from .linear import matmul_partials, stacked_rows


@register_mixer("matrix_memory")
class MatrixMemory:
    def __init__(self, params: dict, rt):
        self.rt = rt
        self.D = int(params["hidden_size"])
        self.H = int(params["num_heads"])
        self.dk = int(params["key_dim"])
        self.dv = int(params["value_dim"])
        self.cap = float(params["gate_cap"])
        self.eps = float(params["eps"])
        if min(self.H, self.dk, self.dv) <= 0 or self.dk > 256 or self.dv > 1024 or not self.cap > 0:
            raise ValueError(f"matrix_memory: {self.H} heads of {self.dk} (up to 256) and {self.dv} (up to 1,024), "
                             f"gates within {self.cap}")
        self.P = -(-(self.dv + 1) // 4) * 4            # the state's columns: the values', n's, and padding
        self.w_in = self.w_o = self.i_bias = self.f_bias = self.norm = None

    def tensor_needs(self):
        H, dk, dv, D = self.H, self.dk, self.dv, self.D
        return {"q": TensorNeed((H * dk, D)), "k": TensorNeed((H * dk, D)), "v": TensorNeed((H * dv, D)),
                "g": TensorNeed((H * dv, D)), "i": TensorNeed((H, D)), "i.b": TensorNeed((H,), init="around_zero"),
                "f": TensorNeed((H, D)), "f.b": TensorNeed((H,), init="around_zero"),
                "norm": TensorNeed((H * dv,), init="ones"), "o": TensorNeed((D, H * dv))}

    def bind(self, tensors) -> None:
        rt = self.rt
        w, self.cols = stacked_rows([tensors[k] for k in ("q", "k", "v", "g", "i", "f")])
        self.w_in, self.w_o = rt.matrix(w), rt.matrix(tensors["o"])
        self.i_bias, self.f_bias = rt.vector(tensors["i.b"]), rt.vector(tensors["f.b"])
        self.norm = rt.vector(tensors["norm"])

    def cache_need(self):
        return {"state": CacheNeed("state", state_shape=(self.H, self.P, self.dk), state_dtype=torch.float32),
                "maximum": CacheNeed("state", state_shape=(self.H,), state_dtype=torch.float32)}

    def cache_read_bytes(self, contexts, element_size: int) -> int:
        return 2 * len(contexts) * self.H * (self.dk * (self.dv + 1) + 1) * 4      # read and written

    def flops(self, q_lens, past) -> float:
        n = sum(q_lens)
        H, dk, dv, D = self.H, self.dk, self.dv, self.D
        return 2.0 * n * ((2 * H * dk + 2 * H * dv + 2 * H) * D + D * H * dv) + 4.0 * n * H * dk * (dv + 1)

    def forward(self, h, batch, stream, view, shared: bool = False):
        if shared:
            raise RuntimeError("a recurrent state cannot be read by another run entry")
        rt, H, dk, dv, P = self.rt, self.H, self.dk, self.dv, self.P
        n = batch.n_tokens
        z, S = matmul_partials(rt, h, self.w_in, "memory_in")
        cq, ck, cv, cg, ci, cf = self.cols
        act = rt.buffer("memory_act", (n, H * P + 2 * H * dk), torch.float32)
        la, put, floor = (rt.buffer(f"memory_{k}", (n, H), torch.float32) for k in ("decay", "put", "floor"))
        ops.mlstm_prep(z, S, (cq, ck, cv, ci, cf), self.i_bias, self.f_bias, self.cap, act, la, put, floor,
                       view["maximum"].state, batch, H, dk, dv, P)
        y = rt.buffer("memory_y", (n, H * P), torch.float32)
        ops.ssd_scan(act, None, 0, 0, None, None, None, batch, view["state"].state, y, H, H, P, dk, steps=(la, put))
        out = rt.buffer("memory_normed", (n, H * dv), rt.dtype)
        ops.gated_heads(y, self.norm, z, S, cg, out, H, dv, self.eps, silu=False, floor=floor)
        stream.add_linear(out, self.w_o)
        return None
