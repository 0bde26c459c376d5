"""A plain, slow implementation of the Pirerax decoder for the tests: whole sequences, no cache, torch on the CPU in
float64 unless told otherwise, one function per mechanism.  It shares no code with the package.

Notation: T tokens, width W; a linear weight is [out, in] and applied as x @ w.T.  ``rnd`` (optional) rounds a tensor
where the bfloat16 engine stores one in bfloat16; it is the identity for the exact result.

A pre-norm decoder whose layers pick one of three mixers: attention over a cached latent with a rotated key part shared
by all heads, a sink and one sigmoid gate per head (``latent_attention``); grouped attention with a norm over the whole
q and k projections, a query temperature, a sink and a sigmoid gate per element (``attention``); or two mixers side by
side (``parallel``), a rotated attention of that kind beside a gated delta rule with one decay per head, whose outputs
are normed over the width and averaged.  The feed-forward routes every token to clamped gated units in groups.
"""
from __future__ import annotations

import json
import math
import os
from typing import Callable, Dict, List, Optional, Tuple

import torch

Rounding = Optional[Callable[[torch.Tensor], torch.Tensor]]


def _r(rnd: Rounding, t: torch.Tensor) -> torch.Tensor:
    return t if rnd is None else rnd(t)


def to_bf16_and_back(t: torch.Tensor) -> torch.Tensor:
    return t.to(torch.bfloat16).to(t.dtype)


# ----------------------------------------------------------------------------- small pieces
def plain_rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def plain_rmsnorm(x, w, eps: float):
    return plain_rms_unit(x, eps) * w


def plain_silu(z):
    return z * torch.sigmoid(z)


def plain_rotate_half(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, n]: dimensions i and i + dims/2 turn by positions * base^(-2i/dims); the rest pass."""
    out = x.clone()
    half = dims // 2
    for i in range(half):
        a = positions.to(torch.float64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype).unsqueeze(-1), torch.sin(a).to(x.dtype).unsqueeze(-1)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def plain_query_temperature(positions: torch.Tensor, coef: float, every: int) -> torch.Tensor:
    return 1.0 + coef * torch.log(torch.div(positions + 1, every, rounding_mode="floor").to(torch.float64) + 1.0)


def plain_softmax_with_sink(s: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """exp(s) / (exp(sink) + sum exp(s)) along the last axis (-inf entries weigh nothing); without a sink the plain softmax."""
    if sink is None:
        return torch.softmax(s, dim=-1)
    m = torch.clamp(s.max(dim=-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - m)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink - m))


def plain_causal(T: int) -> torch.Tensor:
    pos = torch.arange(T)
    return pos[:, None] >= pos[None, :]


# ----------------------------------------------------------------------------- attention over a latent
def plain_latent_core(h, W, p: str, m: dict, eps: float, rnd: Rounding = None):
    """The heads' results ahead of the gate, [T, heads, vdim]: keys and values are built per head from the latent."""
    T = h.shape[0]
    H, D, rd, Dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ W[p + ".q"].T).view(T, H, D + rd)
    down = h @ W[p + ".dkv"].T
    c = _r(rnd, plain_rmsnorm(down[:, :R], W[p + ".dkv.norm"], eps))
    kr, qr = down[:, None, R:], q[..., D:]
    rot = m.get("rot")
    if rot and rd:
        kr, qr = plain_rotate_half(kr, pos, rot["dims"], rot["base"]), plain_rotate_half(qr, pos, rot["dims"], rot["base"])
    kr, qr, qn = _r(rnd, kr), _r(rnd, qr), _r(rnd, q[..., :D])
    uk, uv = W[p + ".uk"].view(H, D, R), W[p + ".uv"].view(H, Dv, R)
    vis = plain_causal(T)
    out = torch.zeros(T, H, Dv, dtype=h.dtype)
    for hd in range(H):
        if rnd is None:
            s = qn[:, hd] @ (c @ uk[hd].T).T
        else:                                  # the engine carries the query into the latent space and rounds it there
            s = _r(rnd, qn[:, hd] @ uk[hd]) @ c.T
        s = ((s + qr[:, hd] @ kr[:, 0].T) * m["scale"]).masked_fill(~vis, -math.inf)
        pr = plain_softmax_with_sink(s, W[p + ".sink"][hd])
        out[:, hd] = (pr @ (c @ uv[hd].T)) if rnd is None else _r(rnd, pr @ c) @ uv[hd].T
    return out


def plain_latent_attention(h, W, p: str, m: dict, eps: float, rnd: Rounding = None):
    T = h.shape[0]
    o = plain_latent_core(h, W, p, m, eps, rnd) * torch.sigmoid(h @ W[p + ".g"].T)[:, :, None]
    return _r(rnd, o.reshape(T, -1)) @ W[p + ".o"].T


# ----------------------------------------------------------------------------- grouped attention
def plain_grouped_attention(h, W, p: str, m: dict, eps: float, sink: bool, rnd: Rounding = None):
    """One norm over all rows of q (and of k), the rotation and the temperature when the entry has them, a gate per element."""
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = plain_rmsnorm(h @ W[p + ".q"].T, W[p + ".q.norm"], eps).view(T, H, D)
    k = plain_rmsnorm(h @ W[p + ".k"].T, W[p + ".k.norm"], eps).view(T, G, D)
    v = _r(rnd, h @ W[p + ".v"].T).view(T, G, Dv)
    rot, temp = m.get("rot"), m.get("q_temp")
    if rot and rot["dims"]:
        q, k = plain_rotate_half(q, pos, rot["dims"], rot["base"]), plain_rotate_half(k, pos, rot["dims"], rot["base"])
    if temp:
        q = q * plain_query_temperature(pos, temp["coef"], temp["every"]).to(q.dtype)[:, None, None]
    q, k = _r(rnd, q), _r(rnd, k)
    vis = plain_causal(T)
    out = torch.zeros(T, H, Dv, dtype=h.dtype)
    for hd in range(H):
        kv = hd // (H // G)
        s = (q[:, hd] @ k[:, kv].T * m["scale"]).masked_fill(~vis, -math.inf)
        out[:, hd] = plain_softmax_with_sink(s, W[p + ".sink"][hd] if sink else None) @ v[:, kv]
    o = out.reshape(T, H * Dv) * torch.sigmoid(h @ W[p + ".g"].T)
    return _r(rnd, o) @ W[p + ".o"].T


# ----------------------------------------------------------------------------- gated delta rule
def plain_short_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x [T, C], w [C, taps]: y[t, c] = sum_j w[c, j] * x[t - (taps - 1) + j, c], zeros ahead of the first row."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * x[:T - back]
    return y


def plain_unit(x: torch.Tensor, eps: float = 1e-6) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + eps)


def plain_head_decay(a, dt_bias, a_log):
    """[T, heads] in (0, 1): exp(-exp(A_log) * softplus(a + dt_bias))."""
    return torch.exp(-torch.exp(a_log) * torch.nn.functional.softplus(a + dt_bias))


def plain_delta_recurrence(q, k, v, g, beta, state=None):
    """q, k: [T, heads, D]; v: [T, heads, Dv]; g, beta [T, heads].  Token by token: the state shrinks by g; what it then
    predicts for k is taken off v, the rest times beta is written along k; q reads after the write."""
    T, Hh, D = q.shape
    S = torch.zeros(Hh, D, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    o = torch.zeros(T, Hh, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o, S


def plain_delta(h, W, p: str, m: dict, eps: float, rnd: Rounding = None):
    T = h.shape[0]
    heads, kvh, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (plain_silu(plain_short_conv(h @ W[f"{p}.{n}"].T, W[f"{p}.{n}.conv"])) for n in ("q", "k", "v"))
    q = (plain_unit(q.view(T, kvh, D)) * D ** -0.5).repeat_interleave(heads // kvh, dim=1)
    k = plain_unit(k.view(T, kvh, D)).repeat_interleave(heads // kvh, dim=1)
    beta = torch.sigmoid(h @ W[p + ".b"].T)
    g = plain_head_decay(h @ W[p + ".a"].T, W[p + ".dt_bias"], W[p + ".A_log"])
    o, _ = plain_delta_recurrence(q, k, v.view(T, heads, Dv), g, beta)
    y = plain_rms_unit(o, eps) * W[p + ".norm"] * plain_silu(h @ W[p + ".g"].T).view(T, heads, Dv)
    return _r(rnd, y.reshape(T, heads * Dv)) @ W[p + ".o"].T


def plain_parallel(h, W, p: str, m: dict, eps: float, rnd: Rounding = None):
    left = plain_grouped_attention(h, W, p + ".left", m["left"], eps, False, rnd)
    right = plain_delta(h, W, p + ".right", m["right"], eps, rnd)
    return 0.5 * (plain_rmsnorm(left, W[p + ".left.out"], eps) + plain_rmsnorm(right, W[p + ".right.out"], eps))


# ----------------------------------------------------------------------------- routed experts
def plain_route(z: torch.Tensor, top: int, groups: int, keep: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """z [T, E] -> (ids, weights [T, top]), token by token: a group of neighbours scores the sum of its two largest
    sigmoids, experts of the ``keep`` best groups are ranked by theirs, the weights are those scores as they are."""
    T, E = z.shape
    per = E // groups
    s = torch.sigmoid(z)
    ids = torch.zeros(T, top, dtype=torch.long)
    for t in range(T):
        row = s[t].tolist()
        strength = [sum(sorted(row[g * per:(g + 1) * per], reverse=True)[:2]) for g in range(groups)]
        kept = sorted(range(groups), key=lambda g: (-strength[g], g))[:keep]
        able = [e for e in range(E) if e // per in kept]
        ids[t] = torch.tensor(sorted(able, key=lambda e: (-float(z[t, e]), e))[:top])
    return ids, s.gather(1, ids)


def plain_clamped_unit(g, u, limit: float):
    g = torch.clamp(g, max=limit)
    u = torch.clamp(u, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def plain_moe(h, W, p: str, mlp: dict, rnd: Rounding = None, chosen: Optional[list] = None):
    """``chosen`` collects the ids."""
    r = mlp["router"]
    g = r.get("groups") or dict(count=1, keep=1)
    z = h @ W[p + ".router"].T
    ids, wts = plain_route(z, r["top"], g["count"], g["keep"])
    if chosen is not None:
        chosen.append(ids)
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        at = (ids == e).nonzero()
        if len(at):
            rows = at[:, 0]
            a = plain_clamped_unit(h[rows] @ W[f"{p}.e{e}.gate"].T, h[rows] @ W[f"{p}.e{e}.up"].T, mlp["expert"]["limit"])
            out[rows] += wts[rows, at[:, 1]][:, None] * (_r(rnd, a) @ W[f"{p}.e{e}.down"].T)
    return out


def plain_router_margin(z: torch.Tensor, top: int, groups: int, keep: int) -> torch.Tensor:
    """[T]: how far the choice is from another one, the smaller of the gap between the last kept and the first dropped
    group and that between the last chosen and the first passed-over expert of the kept groups (in scores)."""
    T, E = z.shape
    per = E // groups
    s = torch.sigmoid(z)
    out = torch.full((T,), math.inf, dtype=z.dtype)
    for t in range(T):
        row = s[t].tolist()
        strength = [sum(sorted(row[g * per:(g + 1) * per], reverse=True)[:2]) for g in range(groups)]
        order = sorted(range(groups), key=lambda g: (-strength[g], g))
        if keep < groups:
            out[t] = strength[order[keep - 1]] - strength[order[keep]]
        able = sorted((row[e] for e in range(E) if e // per in order[:keep]), reverse=True)
        if top < len(able):
            out[t] = min(float(out[t]), able[top - 1] - able[top])
    return out


# ----------------------------------------------------------------------------- the model
def plain_mixer(h, W, p: str, layer: dict, eps: float, rnd: Rounding = None):
    if layer["type"] == "latent_attention":
        return plain_latent_attention(h, W, p, layer["mixer"], eps, rnd)
    if layer["type"] == "attention":
        return plain_grouped_attention(h, W, p, layer["mixer"], eps, True, rnd)
    return plain_parallel(h, W, p, layer["mixer"], eps, rnd)


def plain_forward(cfg: dict, W: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64, rnd: Rounding = None,
                  residuals: Optional[list] = None, margins: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of the whole sequence.  ``residuals`` collects the stream after every layer, ``margins`` how
    clear every routing decision was ([T] per routed layer)."""
    W = {n: t.to(dtype) for n, t in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}"
        x = x + plain_mixer(_r(rnd, plain_rmsnorm(x, W[p + ".norm1"], eps)), W, p + ".mix", layer, eps, rnd)
        if layer.get("mlp"):
            h = _r(rnd, plain_rmsnorm(x, W[p + ".norm2"], eps))
            if margins is not None:
                r = layer["mlp"]["router"]
                g = r.get("groups") or dict(count=1, keep=1)
                margins.append(plain_router_margin(h @ W[p + ".mlp.router"].T, r["top"], g["count"], g["keep"]))
            x = x + plain_moe(h, W, p + ".mlp", layer["mlp"], rnd)
        if residuals is not None:
            residuals.append(x.clone())
    return _r(rnd, plain_rmsnorm(x, W["final.norm"], eps)) @ W["head"].T


def plain_greedy(cfg, W, prompt: List[int], n_new: int) -> List[int]:
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(plain_forward(cfg, W, toks)[-1])))
    return toks[len(prompt):]


# ----------------------------------------------------------------------------- configurations and weights
def moe(ff: int, limit: float, experts: int, top: int, groups: Optional[Tuple[int, int]] = None) -> dict:
    """``groups``: (count, keep)."""
    router = dict(experts=experts, top=top)
    if groups is not None:
        router["groups"] = dict(count=groups[0], keep=groups[1])
    return dict(kind="moe", expert=dict(ff=ff, limit=limit), router=router)


def latent_layer(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0, mlp=None) -> dict:
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale,
                                                    rot=dict(dims=rot_dim, base=base)), mlp=mlp)


def attention_layer(heads, kv_heads, dim, vdim, scale, temp=None, mlp=None) -> dict:
    """``temp``: (coef, every)."""
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if temp is not None:
        m["q_temp"] = dict(coef=temp[0], every=temp[1])
    return dict(type="attention", mixer=m, mlp=mlp)


def parallel_layer(left, right, mlp=None) -> dict:
    """``left``: (heads, kv_heads, dim, vdim, scale, rotated dims, base); ``right``: (heads, kv_heads, dim, vdim, taps)."""
    return dict(type="parallel", mixer=dict(
        left=dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), left[:5]), rot=dict(dims=left[5], base=left[6])),
        right=dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right))), mlp=mlp)


def make_config(vocab: int, width: int, layers: List[dict], eps: float = 1e-5) -> dict:
    return dict(architecture="Pirerax", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)


def all_experts(cfg: dict) -> dict:
    """The same model with routers that choose every expert."""
    cfg = json.loads(json.dumps(cfg))
    for l in cfg["layers"]:
        if l.get("mlp"):
            r = l["mlp"]["router"]
            r["top"] = r["experts"]
            if "groups" in r:
                r["groups"]["keep"] = r["groups"]["count"]
    return cfg


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    Wd = cfg["width"]
    shapes = {"embed": (cfg["vocab"], Wd), "head": (cfg["vocab"], Wd), "final.norm": (Wd,)}

    def grouped(x: str, m: dict) -> None:
        H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        shapes.update({x + "q": (H * D, Wd), x + "k": (G * D, Wd), x + "v": (G * Dv, Wd), x + "q.norm": (H * D,), x + "k.norm": (G * D,),
                       x + "g": (H * Dv, Wd), x + "o": (Wd, H * Dv)})

    for i, l in enumerate(cfg["layers"]):
        m, x = l["mixer"], f"l{i}.mix."
        shapes[f"l{i}.norm1"] = (Wd,)
        if l["type"] == "latent_attention":
            H, D, rd, Dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            shapes.update({x + "q": (H * (D + rd), Wd), x + "dkv": (R + rd, Wd), x + "dkv.norm": (R,), x + "uk": (H * D, R),
                           x + "uv": (H * Dv, R), x + "sink": (H,), x + "g": (H, Wd), x + "o": (Wd, H * Dv)})
        elif l["type"] == "attention":
            grouped(x, m)
            shapes[x + "sink"] = (m["heads"],)
        else:
            grouped(x + "left.", m["left"])
            r, y = m["right"], x + "right."
            kd, vd = r["kv_heads"] * r["dim"], r["heads"] * r["vdim"]
            shapes.update({y + "q": (kd, Wd), y + "k": (kd, Wd), y + "v": (vd, Wd), y + "q.conv": (kd, r["conv"]), y + "k.conv": (kd, r["conv"]),
                           y + "v.conv": (vd, r["conv"]), y + "b": (r["heads"], Wd), y + "a": (r["heads"], Wd), y + "A_log": (r["heads"],),
                           y + "dt_bias": (r["heads"],), y + "norm": (r["vdim"],), y + "g": (vd, Wd), y + "o": (Wd, vd),
                           x + "left.out": (Wd,), x + "right.out": (Wd,)})
        if l.get("mlp"):
            ff = l["mlp"]["expert"]["ff"]
            shapes.update({f"l{i}.norm2": (Wd,), f"l{i}.mlp.router": (l["mlp"]["router"]["experts"], Wd)})
            for e in range(l["mlp"]["router"]["experts"]):
                shapes.update({f"l{i}.mlp.e{e}.gate": (ff, Wd), f"l{i}.mlp.e{e}.up": (ff, Wd), f"l{i}.mlp.e{e}.down": (Wd, ff)})
    return shapes


def random_weights(cfg: dict, seed: int, gain: float = 1.0) -> Dict[str, torch.Tensor]:
    """Weights large enough that every mechanism moves the logits: matrices N(0, gain^2 / fan_in), gates, routers and the
    experts' gates twice that, norm weights near 1, sinks near 1, decays spread between slow and fast; all rounded to
    bfloat16, the file's type."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "conv":
            t = 0.6 * torch.randn(shape, generator=g)
        elif len(shape) == 2:
            std = 1.0 if name == "embed" else gain / math.sqrt(shape[1])
            if leaf in ("gate", "g", "router"):
                std *= 2.0
            t = torch.randn(shape, generator=g) * std
        elif leaf.startswith("norm") or leaf == "out":
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif leaf == "A_log":
            t = torch.randn(shape, generator=g) - 1.0
        elif leaf == "sink":
            t = 1.0 + torch.randn(shape, generator=g)
        else:                                               # dt_bias
            t = 0.5 * torch.randn(shape, generator=g)
        W[name] = t.to(torch.bfloat16)
    return W


def write_folder(folder: str, cfg: dict, W: Dict[str, torch.Tensor]) -> str:
    from safetensors.torch import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in W.items()}, os.path.join(folder, "model.safetensors"))
    return folder
