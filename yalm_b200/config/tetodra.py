"""Typed configuration of the Tetodra decoder, read from its ``config.json``.

The design: a scaled token embedding; layers whose two sublayers read the SAME layer-normed input and
join the residual stream in one sum, x <- x + r (mixer(h) ls1 + ff(h) ls2) with a stored factor per
feature on either and a constant r; three kinds of mixer in any order -- "parallel" (attention whose
keys are its values, with norms per head, a temperature that grows with the position, a learned bias
per distance and a sink, beside the matrix memory of xLSTM), "parallel_2" (rotary grouped-query
attention with a value size of its own beside gated linear attention with a decay per key channel)
and "delta" (the gated delta rule with one decay per head and short convolutions) --; a SwiGLU
feed-forward or none.  The head is the embedding table.  Every size and constant is read from
config.json:

    architecture          "Tetodra"
    vocab, width          vocabulary and residual width
    embedding.scale       factor on the looked-up row
    norm.eps              epsilon of every norm
    residual_mult         r
    layers[i]             {type, mixer: {...}, mlp: null | {kind: "dense", ff}}
      parallel            {left: {heads, kv_heads, dim, vdim, scale, bias_max, q_temp: {coef, every}},
                           right: {heads, dim, vdim, gate_cap}, left_scale, right_scale}
      parallel_2          {left: {heads, kv_heads, dim, vdim, scale, rot: {base, dims}},
                           right: {heads, dim, vdim, tau}, left_scale, right_scale}
      delta               {heads, kv_heads, dim, vdim, conv}

Checkpoint tensors: ``embed``, ``final.norm``; per layer ``l<i>.norm1``, ``l<i>.ls1``, ``l<i>.ls2``;
parallel: ``l<i>.mix.left.{q,k,q.norm,k.norm,rel,sink,o}`` (``rel`` [rows of the bias table, heads]),
``l<i>.mix.right.{q,k,v,g,o,norm,i,i.b,f,f.b}``; parallel_2: ``l<i>.mix.left.{q,k,v,o}``,
``l<i>.mix.right.{q,k,v,g,o,norm,a1,a2,a2.b}`` (the inner size of the decay's projection is the first
dimension of ``a1``); delta: ``l<i>.mix.{q,k,v}`` and their ``.conv``, ``l<i>.mix.{b,A_log,a,dt_bias,g,norm,o}``;
feed-forward: ``l<i>.mlp.{gate,up,down}``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field, replace
from typing import Any, Dict, List, Optional, Tuple

from .llama import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, RunEntry

NO_POSITION_LIMIT = 1 << 30
DEFAULT_CONTEXT = 1 << 16
# random-weights mode, when neither the configuration nor a tensor names them
DEFAULT_RANK = 16
DEFAULT_BIAS_ROWS = 32
KINDS = ("parallel", "parallel_2", "delta")


def _need(d: Dict[str, Any], key: str, where: str):
    if not isinstance(d, dict) or key not in d or d[key] is None:
        raise ConfigError(f"config.json lacks {where}{key}")
    return d[key]


def _positive(d: Dict[str, Any], where: str, *keys: str) -> List[int]:
    out = [int(_need(d, k, where)) for k in keys]
    if min(out) <= 0:
        raise ConfigError(f"{where}: {', '.join(keys)} must be positive")
    return out


@dataclass(frozen=True)
class TetodraLayer:
    kind: str                        # "parallel", "parallel_2" or "delta"
    mixer: Dict[str, Any]
    mlp: Optional[Dict[str, Any]]
    bias_rows: int = DEFAULT_BIAS_ROWS       # parallel: rows of the distance table
    decay_rank: int = DEFAULT_RANK           # parallel_2: inner size of the decay's projection


@dataclass(frozen=True)
class TetodraConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    residual_mult: float
    layers: List[TetodraLayer]
    raw: Dict[str, Any] = field(default_factory=dict, compare=False)

    architecture = "Tetodra"

    @property
    def vocab_size(self) -> int:
        return self.vocab

    # ---- reading -------------------------------------------------------------------------
    @staticmethod
    def _check_attention(m: Dict[str, Any], where: str) -> None:
        heads, kv, dim, vdim = _positive(m, where, "heads", "kv_heads", "dim", "vdim")
        if heads % kv:
            raise ConfigError(f"{where}: heads={heads} must be a multiple of kv_heads={kv}")
        if dim > 256 or vdim > 256:
            raise ConfigError(f"{where}: dim={dim} and vdim={vdim} up to 256 are supported")
        if not float(_need(m, "scale", where)) > 0:
            raise ConfigError(f"{where}scale must be positive")

    @classmethod
    def _check_mixer(cls, kind: str, m: Dict[str, Any], where: str) -> None:
        if kind == "delta":
            heads, kv, dim, _, conv = _positive(m, where, "heads", "kv_heads", "dim", "vdim", "conv")
            if heads % kv or dim > 256 or not 2 <= conv <= 8:
                raise ConfigError(f"{where}: heads={heads} must be a multiple of kv_heads={kv}; key sizes up to 256 "
                                  f"({dim}) and convolutions of 2 to 8 taps ({conv}) are supported")
            return
        left, right = _need(m, "left", where), _need(m, "right", where)
        cls._check_attention(left, where + "left.")
        _, dim, _ = _positive(right, where + "right.", "heads", "dim", "vdim")
        if dim > 256:
            raise ConfigError(f"{where}right.dim={dim}: key sizes up to 256 are supported")
        for k in ("left_scale", "right_scale"):
            float(_need(m, k, where))
        if kind == "parallel":
            if int(left["vdim"]) != int(left["dim"]):
                raise ConfigError(f"{where}left: the values are the keys, vdim={left['vdim']} must be dim={left['dim']}")
            if not float(_need(left, "bias_max", where + "left.")) > 1:
                raise ConfigError(f"{where}left.bias_max must be larger than 1")
            qt = _need(left, "q_temp", where + "left.")
            float(_need(qt, "coef", where + "left.q_temp."))
            if not float(_need(qt, "every", where + "left.q_temp.")) > 0:
                raise ConfigError(f"{where}left.q_temp.every must be positive")
            if not float(_need(right, "gate_cap", where + "right.")) > 0:
                raise ConfigError(f"{where}right.gate_cap must be positive")
        else:
            rot = left.get("rot")
            if rot:
                dims, base = int(_need(rot, "dims", where + "left.rot.")), float(_need(rot, "base", where + "left.rot."))
                if dims % 2 or not 0 <= dims <= int(left["dim"]) or not base > 0:
                    raise ConfigError(f"{where}left.rot: dims={dims} must be even and at most {left['dim']}; base > 0")
            if not float(_need(right, "tau", where + "right.")) > 0:
                raise ConfigError(f"{where}right.tau must be positive")

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "TetodraConfig":
        layers: List[TetodraLayer] = []
        for i, ld in enumerate(_need(d, "layers", "")):
            where = f"layers[{i}]."
            kind = _need(ld, "type", where)
            if kind not in KINDS:
                raise ConfigError(f"{where}type={kind!r} is not supported {KINDS}")
            mixer = copy.deepcopy(_need(ld, "mixer", where))
            mlp = copy.deepcopy(ld.get("mlp")) or None
            cls._check_mixer(kind, mixer, where + "mixer.")
            if mlp:
                if mlp.get("kind", "dense") != "dense":
                    raise ConfigError(f"{where}mlp.kind={mlp['kind']!r} is not supported ('dense')")
                _positive(mlp, where + "mlp.", "ff")
            side = lambda s, k, default: int((mixer.get(s) or {}).get(k) or default)
            layers.append(TetodraLayer(kind, mixer, mlp, side("left", "bias_rows", DEFAULT_BIAS_ROWS),
                                       side("right", "decay_rank", DEFAULT_RANK)))
        if not layers:
            raise ConfigError("config.json lists no layers")
        cfg = cls(vocab=int(_need(d, "vocab", "")), width=int(_need(d, "width", "")),
                  eps=float(_need(_need(d, "norm", ""), "eps", "norm.")),
                  embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                  residual_mult=float(d.get("residual_mult", 1.0)), layers=layers, raw=copy.deepcopy(d))
        if cfg.vocab <= 0 or cfg.width <= 0 or not cfg.eps > 0:
            raise ConfigError("vocab, width and norm.eps must be positive")
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        d = copy.deepcopy(self.raw)
        for ld, layer in zip(d.get("layers", []), self.layers):
            if layer.kind == "parallel":
                ld["mixer"]["left"]["bias_rows"] = layer.bias_rows
            elif layer.kind == "parallel_2":
                ld["mixer"]["right"]["decay_rank"] = layer.decay_rank
        return d

    def with_tensor_shapes(self, shapes: Dict[str, Tuple[int, ...]]) -> "TetodraConfig":
        """Sizes that only the checkpoint's tensors give: the rows of a distance table and the inner size
        of a decay's low-rank projection."""
        layers = []
        for i, layer in enumerate(self.layers):
            for kind, name, attr in (("parallel", f"l{i}.mix.left.rel", "bias_rows"),
                                     ("parallel_2", f"l{i}.mix.right.a1", "decay_rank")):
                if layer.kind == kind and len(shapes.get(name, ())) == 2:
                    layer = replace(layer, **{attr: int(shapes[name][0])})
            layers.append(layer)
        return replace(self, layers=layers)

    def ignorable_tensor(self, name: str) -> bool:
        """The factors of a layer's absent feed-forward may be in a checkpoint; they are not read."""
        return any(layer.mlp is None and name == f"l{i}.ls2" for i, layer in enumerate(self.layers))

    # ---- the architecture as a list of parts ---------------------------------------------------
    def _attention(self, layer: TetodraLayer) -> PartSpec:
        m = layer.mixer["left"]
        params = {"hidden_size": self.width, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]),
                  "head_dim": int(m["dim"]), "value_dim": int(m["vdim"]), "scale": float(m["scale"])}
        if layer.kind == "parallel":
            qt = m["q_temp"]
            params.update(values_from_keys=True, qk_head_norm={"eps": self.eps}, sink=True,
                          q_temperature={"coef": float(qt["coef"]), "every": float(qt["every"])},
                          distance_bias={"rows": layer.bias_rows, "largest": float(m["bias_max"])})
        elif m.get("rot"):
            params["rotation"] = {"dims": int(m["rot"]["dims"]), "base": float(m["rot"]["base"])}
        return PartSpec("exact_attention", params)

    def _mixer(self, i: int, layer: TetodraLayer) -> PartSpec:
        D, m, p = self.width, layer.mixer, f"l{i}.mix"
        names = lambda side, *keys: {f"{side}{k}": f"{p}.{side}{k}" for k in keys}
        if layer.kind == "delta":
            return PartSpec("gated_delta_rule",
                            {"hidden_size": D, "num_heads": int(m["heads"]), "num_kv_heads": int(m["kv_heads"]),
                             "key_dim": int(m["dim"]), "value_dim": int(m["vdim"]), "conv": int(m["conv"]),
                             "decay": "head", "gate": "silu", "eps": self.eps},
                            names("", "q", "k", "v", "q.conv", "k.conv", "v.conv", "b", "A_log", "a", "dt_bias", "g",
                                  "norm", "o"))
        r = m["right"]
        sizes = {"hidden_size": D, "num_heads": int(r["heads"]), "key_dim": int(r["dim"]), "value_dim": int(r["vdim"]),
                 "eps": self.eps}
        if layer.kind == "parallel":
            right = PartSpec("matrix_memory", {**sizes, "gate_cap": float(r["gate_cap"])})
            tensors = {**names("left.", "q", "k", "q.norm", "k.norm", "rel", "sink", "o"),
                       **names("right.", "q", "k", "v", "g", "o", "norm", "i", "i.b", "f", "f.b")}
        else:
            right = PartSpec("gated_linear_attention", {**sizes, "tau": float(r["tau"]), "decay_rank": layer.decay_rank})
            tensors = {**names("left.", "q", "k", "v", "o"),
                       **names("right.", "q", "k", "v", "g", "o", "norm", "a1", "a2", "a2.b")}
        return PartSpec("parallel_branches",
                        {"hidden_size": D, "eps": self.eps, "branch_norm": False,
                         "scales": [float(m["left_scale"]), float(m["right_scale"])],
                         "branches": [("left", self._attention(layer)), ("right", right)]}, tensors)

    def to_spec(self) -> ModelSpec:
        D = self.width
        norm = lambda name: PartSpec("layernorm", {"size": D, "eps": self.eps}, {"weight": name})
        scale = lambda name: PartSpec("layer_scale", {"size": D, "factor": self.residual_mult}, {"weight": name})
        layers = []
        for i, layer in enumerate(self.layers):
            p = f"l{i}"
            parts = {"norm": norm(f"{p}.norm1"), "mixer": self._mixer(i, layer), "mixer_scale": scale(f"{p}.ls1")}
            if layer.mlp:
                parts["feed_forward"] = PartSpec("swiglu", {"hidden_size": D, "intermediate_size": int(layer.mlp["ff"])},
                                                 {k: f"{p}.mlp.{k}" for k in ("gate", "up", "down")})
                parts["feed_forward_scale"] = scale(f"{p}.ls2")
            layers.append(LayerSpec("parallel_prenorm", parts))
        spec = ModelSpec(
            architecture=self.architecture, vocab_size=self.vocab, hidden_size=D,
            max_positions=NO_POSITION_LIMIT, default_context=DEFAULT_CONTEXT,
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "size": D, "scale": self.embedding_scale},
                               {"weight": "embed"}),
            layers=layers, run_order=[RunEntry(i) for i in range(len(layers))],
            final_norm=norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": self.vocab, "size": D, "tied": True}, {"weight": "embed"}),
            overlapped_launches=False,
        )
        spec.validate()
        return spec
