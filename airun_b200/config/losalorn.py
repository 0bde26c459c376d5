"""Configuration of the Losalorn decoder, read from its config.json keys.

A Losalorn layer norms the input and the output of each sub-layer (parts/block.py: ``sandwich``).  Its mixer is a gated
delta rule with one decay per head and a silu gate ("delta"), or a windowed softmax attention whose values are its keys
ahead of the rotation and whose softmax has a one added to its denominator ("attention").  A run of layers may be gone
through several times with the same weights and a cache or state per pass; ahead of every pass the residual stream is
mixed with the embedding (parts/residual_input.py).  The head is the embedding table, its logits are capped by a tanh.

``architecture``        "Losalorn"
``vocab``, ``width``    vocabulary and residual width
``embedding.scale``     every embedded row is multiplied by it (absent: 1)
``norm.eps``            eps of every root mean square
``logit_softcap``       c in logits <- c tanh(logits / c) (absent or null: none)
``layers``              one entry per layer: ``type`` ("delta" | "attention"), ``mixer`` (its sizes and constants) and
                        ``mlp`` ({"kind": "dense", "ff", "limit"}, or null for none)
``loop``                {"start", "stop", "times"}: layers start .. stop-1 run ``times`` times in a row (absent: once, and
                        nothing is mixed)

Mixer keys.  "delta": ``heads``, ``kv_heads``, ``dim`` (key channels a head), ``vdim`` (value channels a head), ``conv`` (taps).
"attention": ``heads``, ``kv_heads``, ``dim``, ``vdim`` (equal to ``dim``), ``scale``, ``mask.size`` (sliding window; absent:
none) and ``rot`` {``dims``, ``base``, ``scaling`` {factor, low, high, original}} (absent: no rotation).

Tensor names: ``embed``, ``loop.in``, ``final.norm`` and per layer ``l<i>.norm1|norm1b|norm2|norm2b``,
``l<i>.mix.{q,k,v,q.conv,k.conv,v.conv,b,a,A_log,dt_bias,g,norm,o}`` or ``l<i>.mix.{q,k,o}``, ``l<i>.mlp.{gate,up,down}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .base import ConfigError, LayerCall, LayerSpec, ModelConfig

MIXERS = ("delta", "attention")


@dataclass(frozen=True)
class LosalornConfig(ModelConfig):
    vocab_size: int
    hidden_size: int
    embedding_scale: float
    norm_eps: float
    logit_softcap: Optional[float]
    layers: Tuple[Dict[str, Any], ...]
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    architecture: str = "Losalorn"
    tie_word_embeddings: bool = True
    max_position_embeddings: int = 1 << 20       # the cache alone bounds a request

    # ---- reading ----
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "LosalornConfig":
        problems: List[str] = []

        def integer(where, key: str, what: str, default=None, least: int = 1) -> int:
            v = where.get(key, default) if isinstance(where, dict) else default
            if isinstance(v, bool) or not isinstance(v, int):
                problems.append(f"{what} must be an integer, found {v!r}")
                return least
            if v < least:
                problems.append(f"{what} must be at least {least}, found {v}")
                return least
            return v

        def number(where, key: str, what: str, default=None, positive: bool = False) -> float:
            v = where.get(key, default) if isinstance(where, dict) else default
            if isinstance(v, bool) or not isinstance(v, (int, float)):
                problems.append(f"{what} must be a number, found {v!r}")
                return 1.0
            if positive and not v > 0:
                problems.append(f"{what} must be positive, found {v}")
                return 1.0
            return float(v)

        def heads(m, w: str) -> Dict[str, Any]:
            a: Dict[str, Any] = dict(heads=integer(m, "heads", f"{w}.heads"), dim=integer(m, "dim", f"{w}.dim"))
            a["kv_heads"] = integer(m, "kv_heads", f"{w}.kv_heads", a["heads"])
            if a["heads"] % a["kv_heads"]:
                problems.append(f"{w}.heads ({a['heads']}) must be a multiple of kv_heads ({a['kv_heads']})")
            a["vdim"] = integer(m, "vdim", f"{w}.vdim", a["dim"])
            return a

        V = integer(d, "vocab", "vocab")
        H = integer(d, "width", "width")
        scale = number(d.get("embedding") or {}, "scale", "embedding.scale", 1.0)
        eps = number(d.get("norm") or {}, "eps", "norm.eps", positive=True)
        cap = None if d.get("logit_softcap") is None else number(d, "logit_softcap", "logit_softcap", positive=True)
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json cannot be used: 'layers' must be a non-empty list")
        layers: List[Dict[str, Any]] = []
        for i, l in enumerate(raw):
            w = f"layers[{i}]"
            if not isinstance(l, dict) or l.get("type") not in MIXERS or not isinstance(l.get("mixer"), dict):
                problems.append(f"{w} needs a 'type' out of {list(MIXERS)} and a 'mixer' object")
                layers.append(dict(type=None, mixer={}, mlp=None))
                continue
            m, w = l["mixer"], f"layers[{i}].mixer"
            mixer = heads(m, w)
            if l["type"] == "delta":
                mixer["conv"] = integer(m, "conv", f"{w}.conv")
            else:
                if mixer["vdim"] != mixer["dim"]:
                    problems.append(f"{w}.vdim ({mixer['vdim']}) must equal dim ({mixer['dim']}): the values are the keys")
                mixer["scale"] = number(m, "scale", f"{w}.scale", mixer["dim"] ** -0.5)
                if m.get("mask") is not None:
                    mixer["mask"] = dict(size=integer(m["mask"], "size", f"{w}.mask.size"))
                rot = m.get("rot")
                if rot is not None:
                    r: Dict[str, Any] = dict(dims=integer(rot, "dims", f"{w}.rot.dims", mixer["dim"], least=0),
                                             base=number(rot, "base", f"{w}.rot.base", 10000.0, positive=True))
                    if r["dims"] % 2 or r["dims"] > mixer["dim"]:
                        problems.append(f"{w}.rot.dims must be even and at most dim ({mixer['dim']}), found {r['dims']}")
                    sc = rot.get("scaling") if isinstance(rot, dict) else None
                    if sc is not None:
                        r["scaling"] = {k: number(sc, k, f"{w}.rot.scaling.{k}", positive=True) for k in ("factor", "low", "high", "original")}
                        if r["scaling"]["high"] < r["scaling"]["low"]:
                            problems.append(f"{w}.rot.scaling.high must be at least low")
                    mixer["rot"] = r
            mlp = l.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind", "dense") != "dense":
                    problems.append(f"layers[{i}].mlp must be null or an object of kind 'dense'")
                    mlp = None
                else:
                    mlp = dict(kind="dense", ff=integer(mlp, "ff", f"layers[{i}].mlp.ff"),
                               limit=number(mlp, "limit", f"layers[{i}].mlp.limit", positive=True))
            layers.append(dict(type=l["type"], mixer=mixer, mlp=mlp))
        L = len(raw)
        loop = d.get("loop") or {}
        start = integer(loop, "start", "loop.start", 0, least=0)
        stop = integer(loop, "stop", "loop.stop", start, least=0)
        times = integer(loop, "times", "loop.times", 1, least=0)
        if not (0 <= start <= stop <= L):
            problems.append(f"loop must satisfy 0 <= start <= stop <= {L}, found start {start}, stop {stop}")
        if problems:
            raise ConfigError("config.json cannot be used: " + "; ".join(problems))
        return cls(vocab_size=V, hidden_size=H, embedding_scale=scale, norm_eps=eps, logit_softcap=cap, layers=tuple(layers),
                   loop_start=start, loop_stop=stop, loop_times=times, architecture=str(d.get("architecture", "Losalorn")))

    def to_dict(self) -> Dict[str, Any]:
        def copy(v):
            return {k: copy(x) for k, x in v.items()} if isinstance(v, dict) else v
        return {"architecture": self.architecture, "embedding": {"scale": self.embedding_scale},
                "layers": [copy(dict(l)) for l in self.layers], "logit_softcap": self.logit_softcap,
                "loop": {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times},
                "norm": {"eps": self.norm_eps}, "vocab": self.vocab_size, "width": self.hidden_size}

    # ---- what the model is made of ----
    def tensor_names(self) -> Dict[str, str]:
        return dict(embed="embed", layer="l{i}", mixer="mix", ffn="mlp", norm1="norm1", norm1_post="norm1b", norm2="norm2",
                    norm2_post="norm2b", final_norm="final.norm", head="head")

    def embedding(self) -> Tuple[str, dict]:
        return "token_embedding", {"scale": self.embedding_scale}

    def head(self) -> Tuple[str, dict]:
        return "lm_head", {"soft_cap": self.logit_softcap}

    def final_norm(self) -> Tuple[str, dict]:
        return "rmsnorm", dict(size=self.hidden_size, eps=self.norm_eps, weight_name="")

    def loops(self) -> bool:
        return self.loop_times > 0 and self.loop_stop > self.loop_start

    def residual_input(self) -> Optional[Tuple[str, str, dict]]:
        return ("mix_with_embedding", "loop.in", dict(hidden_size=self.hidden_size)) if self.loops() else None

    def layer_specs(self) -> List[LayerSpec]:
        H, specs = self.hidden_size, []
        for l in self.layers:
            m = l["mixer"]
            if l["type"] == "delta":
                mixer, args = "gated_delta_rule", dict(
                    hidden_size=H, num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["vdim"],
                    conv_taps=m["conv"], norm_eps=self.norm_eps, decay="head", gate="silu")
            else:
                rot = m.get("rot") or {}
                turns = rot.get("dims", 0) > 0
                mixer, args = "softmax_attention", dict(
                    hidden_size=H, num_heads=m["heads"], num_kv_heads=m["kv_heads"], key_dim=m["dim"], value_dim=m["dim"],
                    scale=m["scale"], norm_eps=self.norm_eps, values="keys", sink="one", window=(m.get("mask") or {}).get("size", 0),
                    position="rotary_neox_by_wavelength" if turns else "none",
                    position_args=dict(rotary_dim=rot["dims"], theta=rot["base"], scaling=rot.get("scaling")) if turns else {})
            mlp = l["mlp"]
            specs.append(LayerSpec(
                mixer=mixer, mixer_args=args, feed_forward="clamped_glu" if mlp else "",
                ffn_args=dict(hidden_size=H, intermediate_size=mlp["ff"], limit=mlp["limit"]) if mlp else {},
                norm="rmsnorm", norm_args=dict(size=H, eps=self.norm_eps, weight_name=""), arrangement="sandwich"))
        return specs

    def execution_order(self) -> List[LayerCall]:
        """Layers before the loop once, the looped layers ``times`` times (each pass with caches of its own, the stream
        mixed with the embedding before its first layer), then the rest."""
        order = [LayerCall(i) for i in range(self.loop_start)]
        for _ in range(self.loop_times):
            order += [LayerCall(i, reinject=i == self.loop_start) for i in range(self.loop_start, self.loop_stop)]
        return order + [LayerCall(i) for i in range(self.loop_stop, len(self.layers))]

    def ignorable_tensors(self) -> List[str]:
        """Tensors a model file may hold although nothing reads them: the second norms of a layer without feed-forward and
        the matrix of a loop that runs no layer."""
        return [f"l{i}.{n}" for i, l in enumerate(self.layers) if not l["mlp"] for n in ("norm2", "norm2b")] + \
            ([] if self.loops() else ["loop.in"])

    def summary(self) -> str:
        kinds = "".join("d" if l["type"] == "delta" else "a" for l in self.layers)
        loop = f", layers {self.loop_start}..{self.loop_stop - 1} x {self.loop_times}" if self.loops() else ""
        return (f"{self.architecture}: {len(self.layers)} layers with norms on both sides ({kinds}: d gated delta rule, a windowed "
                f"attention over its own keys), width {self.hidden_size}, vocab {self.vocab_size}{loop}, "
                f"{len(self.execution_order())} layer runs a token")
