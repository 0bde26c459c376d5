"""Configuration of the Pirerax decoder, read from its config.json keys.

A pre-norm decoder whose layers pick one of three mixers: attention over a cached latent with a rotated key part shared
by all heads, a sink and a sigmoid gate per head ("latent_attention"); grouped attention with one norm over the whole q
and k projections, a query temperature instead of a rotation, a sink and a sigmoid gate per element ("attention"); or
two mixers side by side whose results are normed and averaged ("parallel"): a rotated attention of that kind, without
temperature and sink, beside a gated delta rule with one decay per head.  The feed-forward is a mixture of clamped gated
units, routed by sigmoid scores in groups, or absent.

``architecture``        "Pirerax"
``vocab``, ``width``    vocabulary and residual width
``norm.eps``            eps of every root mean square
``layers``              one entry per layer: ``type`` ("latent_attention" | "attention" | "parallel"), ``mixer`` and ``mlp``
                        (null for none)

"latent_attention" mixer keys: ``heads``, ``dim`` (unrotated) and ``rot_dim`` (rotated query/key dimensions a head),
``vdim``, ``kv_rank``, ``scale``, ``rot`` {``dims``, ``base``}.
"attention" mixer keys: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``q_temp`` {``coef``, ``every``} (absent: none).
"parallel" mixer keys: ``left`` {``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``rot`` {``dims``, ``base``}}, ``right``
{``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` (taps)}.
``mlp``: {``kind``: "moe", ``expert``: {``ff``, ``limit``}, ``router``: {``experts``, ``top``, ``groups``: {``count``, ``keep``}}}.

Tensor names: ``embed``, ``head``, ``final.norm`` and per layer ``l<i>.norm1|norm2``, ``l<i>.mix.{q,dkv,dkv.norm,uk,uv,sink,g,o}``,
``l<i>.mix.{q,k,v,q.norm,k.norm,sink,g,o}``, or ``l<i>.mix.left.{q,k,v,q.norm,k.norm,g,o,out}`` with
``l<i>.mix.right.{q,k,v,q.conv,k.conv,v.conv,b,a,A_log,dt_bias,norm,g,o,out}``; ``l<i>.mlp.router`` and
``l<i>.mlp.e<j>.{gate,up,down}``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Tuple

from .base import ConfigError, LayerSpec, ModelConfig

MIXERS = ("latent_attention", "attention", "parallel")


@dataclass(frozen=True)
class PireraxConfig(ModelConfig):
    vocab_size: int
    hidden_size: int
    norm_eps: float
    layers: Tuple[Dict[str, Any], ...]
    architecture: str = "Pirerax"
    tie_word_embeddings: bool = False
    max_position_embeddings: int = 1 << 20       # the cache alone bounds a request

    # ---- reading ----
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "PireraxConfig":
        problems: List[str] = []

        def integer(where, key: str, what: str, default=None, least: int = 1) -> int:
            v = where.get(key, default) if isinstance(where, dict) else default
            if isinstance(v, float) and v.is_integer():
                v = int(v)
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

        def rotation(m, w: str, most: int, default: int) -> Dict[str, Any]:
            r = dict(dims=integer(m["rot"], "dims", f"{w}.rot.dims", default, least=0),
                     base=number(m["rot"], "base", f"{w}.rot.base", 10000.0, positive=True))
            if r["dims"] % 2 or r["dims"] > most:
                problems.append(f"{w}.rot.dims must be even and at most {most}, found {r['dims']}")
            return r

        def latent(m, w: str) -> Dict[str, Any]:
            a: Dict[str, Any] = {k: integer(m, k, f"{w}.{k}") for k in ("heads", "dim", "kv_rank")}
            a["rot_dim"] = integer(m, "rot_dim", f"{w}.rot_dim", 0, least=0)
            a["vdim"] = integer(m, "vdim", f"{w}.vdim", a["dim"])
            a["scale"] = number(m, "scale", f"{w}.scale", (a["dim"] + a["rot_dim"]) ** -0.5)
            if m.get("rot") is not None:
                a["rot"] = rotation(m, w, a["rot_dim"], a["rot_dim"])
            return a

        def attention(m, w: str, rotated: bool) -> Dict[str, Any]:
            a = heads(m, w)
            a["scale"] = number(m, "scale", f"{w}.scale", a["dim"] ** -0.5)
            if rotated and m.get("rot") is not None:
                a["rot"] = rotation(m, w, a["dim"], a["dim"])
            if not rotated and m.get("q_temp") is not None:
                a["q_temp"] = dict(coef=number(m["q_temp"], "coef", f"{w}.q_temp.coef"), every=integer(m["q_temp"], "every", f"{w}.q_temp.every"))
            return a

        def moe(mlp, w: str) -> Dict[str, Any]:
            r, ex = mlp.get("router") or {}, mlp.get("expert") or {}
            g = r.get("groups") or {}
            router = dict(experts=integer(r, "experts", f"{w}.router.experts"), top=integer(r, "top", f"{w}.router.top"),
                          groups=dict(count=integer(g, "count", f"{w}.router.groups.count", 1),
                                      keep=integer(g, "keep", f"{w}.router.groups.keep", 1)))
            E, gc, gk = router["experts"], router["groups"]["count"], router["groups"]["keep"]
            if E % gc or gk > gc:
                problems.append(f"{w}.router: {gc} groups must divide the {E} experts, and keep ({gk}) cannot exceed them")
            elif router["top"] > E // gc * gk:
                problems.append(f"{w}.router.top exceeds the experts of the kept groups")
            return dict(kind="moe", expert=dict(ff=integer(ex, "ff", f"{w}.expert.ff"),
                                                limit=number(ex, "limit", f"{w}.expert.limit", positive=True)), router=router)

        V = integer(d, "vocab", "vocab")
        H = integer(d, "width", "width")
        eps = number(d.get("norm") or {}, "eps", "norm.eps", positive=True)
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json cannot be used: 'layers' must be a non-empty list")
        layers: List[Dict[str, Any]] = []
        for i, l in enumerate(raw):
            w = f"layers[{i}]"
            if not isinstance(l, dict) or l.get("type") not in MIXERS or not isinstance(l.get("mixer"), dict):
                problems.append(f"{w} needs a 'type' out of {list(MIXERS)} and a 'mixer' object")
                continue
            m = l["mixer"]
            if l["type"] == "latent_attention":
                mixer = latent(m, f"{w}.mixer")
            elif l["type"] == "attention":
                mixer = attention(m, f"{w}.mixer", False)
            elif not isinstance(m.get("left"), dict) or not isinstance(m.get("right"), dict):
                problems.append(f"{w}.mixer needs 'left' and 'right' objects")
                continue
            else:
                right = heads(m["right"], f"{w}.mixer.right")
                right["conv"] = integer(m["right"], "conv", f"{w}.mixer.right.conv")
                mixer = dict(left=attention(m["left"], f"{w}.mixer.left", True), right=right)
            mlp = l.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
                    problems.append(f"{w}.mlp must be null or an object of kind 'moe'")
                    continue
                mlp = moe(mlp, f"{w}.mlp")
            layers.append(dict(type=l["type"], mixer=mixer, mlp=mlp))
        if problems:
            raise ConfigError("config.json cannot be used: " + "; ".join(problems))
        return cls(vocab_size=V, hidden_size=H, norm_eps=eps, layers=tuple(layers), architecture=str(d.get("architecture", "Pirerax")))

    def to_dict(self) -> Dict[str, Any]:
        def copy(v):
            return {k: copy(x) for k, x in v.items()} if isinstance(v, dict) else v
        return {"architecture": self.architecture, "layers": [copy(dict(l)) for l in self.layers], "norm": {"eps": self.norm_eps},
                "vocab": self.vocab_size, "width": self.hidden_size}

    # ---- what the model is made of ----
    def tensor_names(self) -> Dict[str, str]:
        return dict(embed="embed", layer="l{i}", mixer="mix", ffn="mlp", norm1="norm1", norm2="norm2", final_norm="final.norm", head="head")

    def final_norm(self) -> Tuple[str, dict]:
        return "rmsnorm", dict(size=self.hidden_size, eps=self.norm_eps, weight_name="")

    def _attention_args(self, a: Dict[str, Any]) -> dict:
        rot, temp = a.get("rot") or {}, a.get("q_temp") or {}
        turns = rot.get("dims", 0) > 0
        return dict(num_heads=a["heads"], num_kv_heads=a["kv_heads"], key_dim=a["dim"], value_dim=a["vdim"], scale=a["scale"],
                    norm_eps=self.norm_eps, qk_norm="projection", gate="element", temp_coef=temp.get("coef", 0.0),
                    temp_every=temp.get("every", 0), position="rotary_neox" if turns else "none",
                    position_args=dict(rotary_dim=rot["dims"], theta=rot["base"]) if turns else {})

    def layer_specs(self) -> List[LayerSpec]:
        H, eps, specs = self.hidden_size, self.norm_eps, []
        for l in self.layers:
            m = l["mixer"]
            if l["type"] == "latent_attention":
                rot = m.get("rot") or {}
                turns = rot.get("dims", 0) > 0
                mixer, args = "latent_attention", dict(
                    hidden_size=H, num_heads=m["heads"], head_dim=m["dim"], rot_dim=m["rot_dim"], value_dim=m["vdim"], q_rank=0,
                    kv_rank=m["kv_rank"], scale=m["scale"], norm_eps=eps, sink=True, gate="head",
                    position="rotary_neox" if turns else "none",
                    position_args=dict(rotary_dim=rot["dims"], theta=rot["base"]) if turns else {})
            elif l["type"] == "attention":
                mixer, args = "softmax_attention", dict(hidden_size=H, sink=True, **self._attention_args(m))
            else:
                r = m["right"]
                mixer, args = "side_by_side", dict(
                    hidden_size=H, combine="norms", norm_eps=eps, left="softmax_attention", left_args=self._attention_args(m["left"]),
                    right="gated_delta_rule",
                    right_args=dict(num_heads=r["heads"], num_kv_heads=r["kv_heads"], key_dim=r["dim"], value_dim=r["vdim"],
                                    conv_taps=r["conv"], norm_eps=eps, decay="head", gate="silu"))
            mlp = l["mlp"]
            fargs: Dict[str, Any] = {}
            if mlp:
                r = mlp["router"]
                fargs = dict(hidden_size=H, intermediate_size=mlp["expert"]["ff"], num_experts=r["experts"], top=r["top"],
                             scores="sigmoid", weight_on="output", expert="clamped_glu", limit=mlp["expert"]["limit"],
                             routing="grouped", groups=r["groups"]["count"], keep_groups=r["groups"]["keep"], group_best=2)
            specs.append(LayerSpec(mixer=mixer, mixer_args=args, feed_forward="routed_experts" if mlp else "", ffn_args=fargs,
                                   norm="rmsnorm", norm_args=dict(size=H, eps=eps, weight_name="")))
        return specs

    def ignorable_tensors(self) -> List[str]:
        """Tensors a model file may hold although nothing reads them: the second norm of a layer without feed-forward."""
        return [f"l{i}.norm2" for i, l in enumerate(self.layers) if not l["mlp"]]

    def summary(self) -> str:
        kinds = "".join({"latent_attention": "l", "attention": "a", "parallel": "p"}[l["type"]] for l in self.layers)
        return (f"{self.architecture}: {len(self.layers)} pre-norm layers ({kinds}: l attention over a latent, a attention with a query "
                f"temperature, p rotated attention beside a gated delta rule), width {self.hidden_size}, vocab {self.vocab_size}")
