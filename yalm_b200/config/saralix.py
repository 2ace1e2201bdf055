"""Typed configuration of the Saralix decoder, read from its ``config.json``.

The design: a token embedding; layers whose sublayers are normed before AND after
(x <- x + n1b(mixer(n1(x))), x <- x + n2b(ff(n2(x)))) by layer norms with a weight and no bias; three
kinds of mixer in any order -- "latent_attention" (causal attention over one cached latent row per
token, a rotated key part shared by the heads, an output gate per head), "latent_attention_2" (the same
over a sliding window, with a learned sink per head in the softmax's denominator and no gate) and
"mamba2" (a state-space recurrence with one decay per head, a short convolution in front and a gated
norm in groups behind) --; a gated feed-forward with clamps, a mixture of experts or none.  The head is
the embedding table.  Every size and constant is read from config.json:

    architecture          "Saralix"
    vocab, width          vocabulary and residual width
    norm.eps              epsilon of every norm
    layers[i]             {type, mixer: {...}, mlp: null | {...}}
      latent_attention    {heads, dim, rot_dim, vdim, kv_rank, scale, rot: {base, dims, scaling:
                           {factor, original, fast, slow}}}
      latent_attention_2  the same and mask: {size}
      mamba2              {heads, vdim, state, groups, conv, norm_groups}
      mlp                 {kind: "dense", ff, limit} | {kind: "moe", expert: {ff}, router: {experts, top}}

Checkpoint tensors: ``embed``, ``final.norm``; per layer ``l<i>.norm{1,1b,2,2b}``; latent attention:
``l<i>.mix.{q,dkv,dkv.norm,uk,uv,o}`` and ``.g`` (per-head gate) or ``.sink``; mamba2:
``l<i>.mix.{in,conv,conv.b,dt_bias,A_log,D,norm,o}``; feed-forward: ``l<i>.mlp.{gate,up,down}`` or
``l<i>.mlp.router`` and ``l<i>.mlp.e<j>.{gate,up,down}``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .llama import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry

NO_POSITION_LIMIT = 1 << 30
DEFAULT_CONTEXT = 1 << 16
# the design's own: the dense feed-forward is down(g sigmoid(SLOPE g) (u + SHIFT))
GLU_SLOPE, GLU_SHIFT = 1.702, 1.0


def _need(d: Dict[str, Any], key: str, where: str):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"config.json lacks {where}{key}")
    return d[key]


@dataclass(frozen=True)
class SaralixLayer:
    kind: str                        # "latent_attention", "latent_attention_2" or "mamba2"
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]


@dataclass(frozen=True)
class SaralixConfig:
    vocab: int
    width: int
    eps: float
    layers: List[SaralixLayer]
    raw: Dict[str, Any] = field(default_factory=dict, compare=False)

    architecture = "Saralix"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    # ---- reading -------------------------------------------------------------------------
    @staticmethod
    def _check_latent(kind: str, m: Dict[str, Any], where: str) -> None:
        heads, dim, rd, vdim, rank = (int(_need(m, k, where)) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        if min(heads, dim, vdim, rank) <= 0 or rd < 0 or rd % 2:
            raise ConfigError(f"{where}: heads, dim, vdim, kv_rank must be positive, rot_dim even")
        if not float(_need(m, "scale", where)) > 0:
            raise ConfigError(f"{where}scale must be positive")
        if rd:
            rot = _need(m, "rot", where)
            base, dims = float(_need(rot, "base", where + "rot.")), int(_need(rot, "dims", where + "rot."))
            if dims != rd or not base > 1:
                raise ConfigError(f"{where}rot: dims={dims} must equal rot_dim={rd}; base > 1")
            sc = rot.get("scaling")
            if sc:
                for k in ("factor", "original", "fast", "slow"):
                    if not float(_need(sc, k, where + "rot.scaling.")) > 0:
                        raise ConfigError(f"{where}rot.scaling.{k} must be positive")
        if kind == "latent_attention_2":
            if int(_need(_need(m, "mask", where), "size", where + "mask.")) <= 0:
                raise ConfigError(f"{where}mask.size must be positive")
        elif m.get("mask"):
            raise ConfigError(f"{where}mask: a latent_attention layer sees every earlier position")

    @staticmethod
    def _check_mamba2(m: Dict[str, Any], where: str) -> None:
        heads, vdim, state, groups, conv, ng = (int(_need(m, k, where)) for k in
                                                ("heads", "vdim", "state", "groups", "conv", "norm_groups"))
        if min(heads, vdim, state, groups, ng) <= 0 or heads % groups or (heads * vdim) % ng:
            raise ConfigError(f"{where}: heads={heads} must be a multiple of groups={groups}, heads * vdim of "
                              f"norm_groups={ng}")
        if state > 256 or not 2 <= conv <= 8:
            raise ConfigError(f"{where}: state={state} up to 256 and convolutions of 2 to 8 taps ({conv}) are supported")

    @staticmethod
    def _check_mlp(mlp, where: str) -> None:
        kind = mlp.get("kind")
        if kind == "dense":
            if int(_need(mlp, "ff", where)) <= 0 or not float(_need(mlp, "limit", where)) > 0:
                raise ConfigError(f"{where}: ff and limit must be positive")
        elif kind == "moe":
            r = _need(mlp, "router", where)
            experts, top = int(_need(r, "experts", where + "router.")), int(_need(r, "top", where + "router."))
            if not 0 < top <= experts:
                raise ConfigError(f"{where}router: top={top} of {experts} experts")
            if int(_need(_need(mlp, "expert", where), "ff", where + "expert.")) <= 0:
                raise ConfigError(f"{where}expert.ff must be positive")
        else:
            raise ConfigError(f"{where}kind={kind!r} is not supported ('dense', 'moe')")

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "SaralixConfig":
        layers: List[SaralixLayer] = []
        for i, ld in enumerate(_need(d, "layers", "")):
            where = f"layers[{i}]."
            kind = _need(ld, "type", where)
            mixer = copy.deepcopy(_need(ld, "mixer", where))
            mlp = copy.deepcopy(ld.get("mlp")) or None
            if kind in ("latent_attention", "latent_attention_2"):
                cls._check_latent(kind, mixer, where + "mixer.")
            elif kind == "mamba2":
                cls._check_mamba2(mixer, where + "mixer.")
            else:
                raise ConfigError(f"{where}type={kind!r} is not supported ('latent_attention', 'latent_attention_2', "
                                  f"'mamba2')")
            if mlp:
                cls._check_mlp(mlp, where + "mlp.")
            layers.append(SaralixLayer(kind, mixer, mlp))
        if not layers:
            raise ConfigError("config.json lists no layers")
        cfg = cls(vocab=int(_need(d, "vocab", "")), width=int(_need(d, "width", "")),
                  eps=float(_need(_need(d, "norm", ""), "eps", "norm.")), layers=layers, raw=copy.deepcopy(d))
        if cfg.vocab <= 0 or cfg.width <= 0 or not cfg.eps > 0:
            raise ConfigError("vocab, width and norm.eps must be positive")
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        return copy.deepcopy(self.raw)

    def ignorable_tensor(self, name: str) -> bool:
        """The norms of a layer's absent feed-forward may be in a checkpoint; they are not read."""
        return any(layer.mlp is None and name in (f"l{i}.norm2", f"l{i}.norm2b") for i, layer in enumerate(self.layers))

    # ---- the architecture as a list of parts ---------------------------------------------------
    def _norm(self, name: str) -> PartSpec:
        return PartSpec("layernorm", {"size": self.width, "eps": self.eps}, {"weight": name})

    def _mixer(self, i: int, layer: SaralixLayer) -> PartSpec:
        D, m, p = self.width, layer.mixer, f"l{i}.mix"
        names = lambda *keys: {k: f"{p}.{k}" for k in keys}
        if layer.kind == "mamba2":
            return PartSpec("mamba2", {"hidden_size": D, "num_heads": int(m["heads"]), "head_dim": int(m["vdim"]),
                                       "state": int(m["state"]), "groups": int(m["groups"]), "conv": int(m["conv"]),
                                       "norm_groups": int(m["norm_groups"]), "eps": self.eps},
                            names("in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o"))
        windowed = layer.kind == "latent_attention_2"
        rot = m.get("rot") or {}
        return PartSpec("latent_attention",
                        {"hidden_size": D, "num_heads": int(m["heads"]), "head_dim": int(m["dim"]),
                         "rot_dim": int(m["rot_dim"]), "value_dim": int(m["vdim"]), "kv_rank": int(m["kv_rank"]),
                         "scale": float(m["scale"]), "rot_base": float(rot.get("base", 2.0)), "rot_layout": "halves",
                         "rot_scaling": rot.get("scaling") or None, "eps": self.eps,
                         "gate": None if windowed else "head", "sink": windowed,
                         "window": int(m["mask"]["size"]) if windowed else None},
                        names("q", "dkv", "dkv.norm", "uk", "uv", "o", "sink" if windowed else "g"))

    def _feed_forward(self, i: int, mlp: Dict[str, Any]) -> PartSpec:
        D, p = self.width, f"l{i}.mlp"
        if mlp["kind"] == "dense":
            return PartSpec("clamped_glu", {"hidden_size": D, "intermediate_size": int(mlp["ff"]),
                                            "limit": float(mlp["limit"]), "slope": GLU_SLOPE, "shift": GLU_SHIFT},
                            {"gate": f"{p}.gate", "up": f"{p}.up", "down": f"{p}.down"})
        r = mlp["router"]
        tensors = {"router": f"{p}.router"}
        for j in range(int(r["experts"])):
            tensors.update({f"gate.{j}": f"{p}.e{j}.gate", f"up.{j}": f"{p}.e{j}.up", f"down.{j}": f"{p}.e{j}.down"})
        # the softmax over the chosen logits is the softmax over all of them divided by the chosen ones' sum
        return PartSpec("routed_experts",
                        {"hidden_size": D, "intermediate_size": int(mlp["expert"]["ff"]), "experts": int(r["experts"]),
                         "top": int(r["top"]), "renormalise": True}, tensors)

    def to_spec(self) -> ModelSpec:
        D = self.width
        layers = []
        for i, layer in enumerate(self.layers):
            p = f"l{i}"
            parts = {"mixer_norm": self._norm(f"{p}.norm1"), "mixer": self._mixer(i, layer),
                     "mixer_post_norm": self._norm(f"{p}.norm1b")}
            if layer.mlp:
                parts["feed_forward_norm"] = self._norm(f"{p}.norm2")
                parts["feed_forward"] = self._feed_forward(i, layer.mlp)
                parts["feed_forward_post_norm"] = self._norm(f"{p}.norm2b")
            layers.append(LayerSpec("prepost_norm", parts))
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=D,
            max_positions=NO_POSITION_LIMIT, default_context=DEFAULT_CONTEXT,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "size": D}, {"weight": "embed"}),
            layers=layers, run_order=[RunEntry(i) for i in range(len(layers))],
            final_norm=self._norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "size": D, "tied": True}, {"weight": "embed"}),
            overlapped_launches=False,
        )
        spec.validate()
        return spec
