"""A plain, slow implementation of the Losalorn decoder for the tests: whole sequences, no cache, torch on the CPU in
float64 unless told otherwise, one function per mechanism.  It shares no code with the package.

Notation: T tokens, width W; a linear weight is [out, in] and applied as x @ w.T.  ``rnd`` (optional) rounds a tensor
where the bfloat16 engine stores one in bfloat16; it is the identity for the exact result.

A layer norms the input AND the output of each sub-layer, x += n_post(sub(n_pre(x))).  Mixers: a gated delta rule with
one decay per head and a silu gate (``delta``), and a windowed attention whose values are its own unrotated keys and
whose softmax has a one added to its denominator (``attention``).  A run of layers may be gone through several times;
ahead of every pass the stream is mixed with the embedding by one matrix, x <- M [x; x0].
"""
from __future__ import annotations

import json
import math
import os
from typing import Callable, Dict, List, Optional

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


def plain_clamped_unit(g, u, limit: float):
    g = torch.clamp(g, max=limit)
    u = torch.clamp(u, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def plain_feed_forward(h, w_gate, w_up, w_down, limit: float, rnd: Rounding = None):
    return _r(rnd, plain_clamped_unit(h @ w_gate.T, h @ w_up.T, limit)) @ w_down.T


def plain_pass_input(x, x0, w_in):
    """x <- M [x; x0], the stream first."""
    return torch.cat([x, x0], dim=-1) @ w_in.T


def plain_soft_cap(z, cap: Optional[float]):
    return z if cap is None else cap * torch.tanh(z / cap)


# ----------------------------------------------------------------------------- gated delta rule
def plain_short_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x [T, C], w [C, taps]: y[t, c] = sum_j w[c, j] * x[t - (taps - 1) + j, c], zeros ahead of the first row."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            src = t - (taps - 1) + j
            if src >= 0:
                y[t] = y[t] + w[:, j] * x[src]
    return y


def plain_unit(x: torch.Tensor, eps: float = 1e-6) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + eps)


def plain_head_decay(a, dt_bias, a_log):
    """[T, heads] in (0, 1): exp(-exp(A_log) * softplus(a + dt_bias))."""
    return torch.exp(-torch.exp(a_log) * torch.nn.functional.softplus(a + dt_bias))


def plain_delta_recurrence(q, k, v, g, beta, state=None):
    """q, k: [T, heads, D]; v: [T, heads, Dv]; g, beta [T, heads].  Token by token and head by head: the state shrinks
    by g; what it then predicts for k is taken off v, the rest times beta is written along k; q reads after the write."""
    T, Hh, D = q.shape
    Dv = v.shape[-1]
    S = torch.zeros(Hh, D, Dv, dtype=q.dtype) if state is None else state.clone()
    o = torch.zeros(T, Hh, Dv, dtype=q.dtype)
    for t in range(T):
        for h in range(Hh):
            Sh = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - Sh.T @ k[t, h])
            Sh = Sh + torch.outer(k[t, h], u)
            o[t, h] = Sh.T @ q[t, h]
            S[h] = Sh
    return o, S


def plain_delta(h, W, p: str, m: dict, eps: float, rnd: Rounding = None):
    T = h.shape[0]
    heads, kvh, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rep = heads // kvh
    q = plain_silu(plain_short_conv(h @ W[p + ".q"].T, W[p + ".q.conv"])).view(T, kvh, D)
    k = plain_silu(plain_short_conv(h @ W[p + ".k"].T, W[p + ".k.conv"])).view(T, kvh, D)
    v = plain_silu(plain_short_conv(h @ W[p + ".v"].T, W[p + ".v.conv"])).view(T, heads, Dv)
    q = (plain_unit(q) * D ** -0.5).repeat_interleave(rep, dim=1)
    k = plain_unit(k).repeat_interleave(rep, dim=1)
    beta = torch.sigmoid(h @ W[p + ".b"].T)
    g = plain_head_decay(h @ W[p + ".a"].T, W[p + ".dt_bias"], W[p + ".A_log"])
    o, _ = plain_delta_recurrence(q, k, v, g, beta)
    y = plain_rms_unit(o, eps) * W[p + ".norm"] * plain_silu(h @ W[p + ".g"].T).view(T, heads, Dv)
    return _r(rnd, y.reshape(T, heads * Dv)) @ W[p + ".o"].T


# ----------------------------------------------------------------------------- attention
def plain_frequencies(dims: int, base: float, scaling: Optional[dict]) -> List[float]:
    """One frequency per rotated pair.  With ``scaling``: pairs whose wavelength is short against the original context
    keep it, long ones are slowed by ``factor``, a linear blend in between."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            wave = 2.0 * math.pi / f
            if wave > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif not wave < scaling["original"] / scaling["high"]:
                s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def plain_rotate_half(x: torch.Tensor, positions, dims: int, freqs: List[float]) -> torch.Tensor:
    """x [T, heads, n]: dimensions i and i + dims/2 turn by positions * freqs[i]."""
    out = x.clone()
    half = dims // 2
    for i in range(half):
        a = positions.to(torch.float64) * freqs[i]
        c, s = torch.cos(a).to(x.dtype).unsqueeze(-1), torch.sin(a).to(x.dtype).unsqueeze(-1)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def plain_window(T: int, size: int) -> torch.Tensor:
    """[T, T] mask: query i sees key j iff 0 <= i - j < size (size 0: every earlier key)."""
    pos = torch.arange(T)
    d = pos[:, None] - pos[None, :]
    return (d >= 0) & ((d < size) if size > 0 else torch.ones_like(d, dtype=torch.bool))


def plain_softmax_plus_one(s: torch.Tensor) -> torch.Tensor:
    """exp(s) / (1 + sum exp(s)) along the last axis (-inf entries weigh nothing)."""
    m = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - m)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(-m))


def plain_attention(h, W, p: str, m: dict, rnd: Rounding = None):
    T = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W[p + ".q"].T).view(T, H, D)
    k = (h @ W[p + ".k"].T).view(T, G, D)
    v = _r(rnd, k)
    rot = m.get("rot")
    if rot and rot["dims"] > 0:
        pos = torch.arange(T)
        freqs = plain_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
        q, k = plain_rotate_half(q, pos, rot["dims"], freqs), plain_rotate_half(k, pos, rot["dims"], freqs)
    q, k = _r(rnd, q), _r(rnd, k)
    vis = plain_window(T, (m.get("mask") or {}).get("size", 0))
    out = torch.zeros(T, H, D, dtype=h.dtype)
    for hd in range(H):
        kv = hd // (H // G)
        s = (q[:, hd] @ k[:, kv].T * m["scale"]).masked_fill(~vis, -math.inf)
        out[:, hd] = plain_softmax_plus_one(s) @ v[:, kv]
    return _r(rnd, out.reshape(T, H * D)) @ W[p + ".o"].T


# ----------------------------------------------------------------------------- the model
def run_order(cfg: dict) -> List[tuple]:
    """(layer, whether a pass begins with it) in the order of execution."""
    L = len(cfg["layers"])
    loop = cfg.get("loop") or dict(start=0, stop=0, times=0)
    order = [(i, False) for i in range(loop["start"])]
    for _ in range(loop["times"]):
        order += [(i, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, False) for i in range(loop["stop"], L)]


def plain_forward(cfg: dict, W: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64, rnd: Rounding = None,
                  residuals: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of the whole sequence.  ``residuals`` collects the stream after every layer run."""
    W = {n: t.to(dtype) for n, t in W.items()}
    eps = cfg["norm"]["eps"]
    x0 = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    x = x0
    for i, begins in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}"
        if begins:
            x = plain_pass_input(x, x0, W["loop.in"])
        h = _r(rnd, plain_rmsnorm(x, W[p + ".norm1"], eps))
        if layer["type"] == "delta":
            y = plain_delta(h, W, p + ".mix", layer["mixer"], eps, rnd)
        else:
            y = plain_attention(h, W, p + ".mix", layer["mixer"], rnd)
        x = x + plain_rmsnorm(y, W[p + ".norm1b"], eps)
        if layer.get("mlp"):
            h = _r(rnd, plain_rmsnorm(x, W[p + ".norm2"], eps))
            y = plain_feed_forward(h, W[p + ".mlp.gate"], W[p + ".mlp.up"], W[p + ".mlp.down"], layer["mlp"]["limit"], rnd)
            x = x + plain_rmsnorm(y, W[p + ".norm2b"], eps)
        if residuals is not None:
            residuals.append(x.clone())
    z = _r(rnd, plain_rmsnorm(x, W["final.norm"], eps)) @ W["embed"].T
    return plain_soft_cap(z, cfg.get("logit_softcap"))


def plain_greedy(cfg, W, prompt: List[int], n_new: int) -> List[int]:
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(torch.argmax(plain_forward(cfg, W, toks)[-1])))
    return toks[len(prompt):]


# ----------------------------------------------------------------------------- configurations and weights
def dense(ff: int, limit: float) -> dict:
    return dict(kind="dense", ff=ff, limit=limit)


def delta_layer(heads, kv_heads, dim, vdim, conv, mlp=None) -> dict:
    return dict(type="delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), mlp=mlp)


def attention_layer(heads, kv_heads, dim, window=None, rot=None, base=10000.0, scaling=None, scale=None, mlp=None) -> dict:
    """``rot``: rotated dimensions; ``scaling``: (factor, low, high, original)."""
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale if scale is not None else dim ** -0.5)
    if rot:
        m["rot"] = dict(dims=rot, base=base)
        if scaling is not None:
            m["rot"]["scaling"] = dict(factor=scaling[0], low=scaling[1], high=scaling[2], original=scaling[3])
    if window is not None:
        m["mask"] = dict(size=window)
    return dict(type="attention", mixer=m, mlp=mlp)


def make_config(vocab, width, layers, loop=None, eps=1e-5, emb_scale=3.0, cap=12.0) -> dict:
    """``loop``: (start, stop, times)."""
    cfg = dict(architecture="Losalorn", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=emb_scale),
               logit_softcap=cap, layers=layers)
    if loop is not None:
        cfg["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return cfg


def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    Wd = cfg["width"]
    shapes = {"embed": (cfg["vocab"], Wd), "final.norm": (Wd,)}
    if any(b for _, b in run_order(cfg)):
        shapes["loop.in"] = (Wd, 2 * Wd)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}", l["mixer"]
        x = p + ".mix."
        shapes.update({p + ".norm1": (Wd,), p + ".norm1b": (Wd,)})
        if l["type"] == "delta":
            kd, vd = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
            shapes.update({x + "q": (kd, Wd), x + "k": (kd, Wd), x + "v": (vd, Wd), x + "q.conv": (kd, m["conv"]),
                           x + "k.conv": (kd, m["conv"]), x + "v.conv": (vd, m["conv"]), x + "b": (m["heads"], Wd),
                           x + "A_log": (m["heads"],), x + "norm": (m["vdim"],), x + "a": (m["heads"], Wd),
                           x + "dt_bias": (m["heads"],), x + "g": (vd, Wd), x + "o": (Wd, vd)})
        else:
            H, G, D = m["heads"], m["kv_heads"], m["dim"]
            shapes.update({x + "q": (H * D, Wd), x + "k": (G * D, Wd), x + "o": (Wd, H * D)})
        if l.get("mlp"):
            ff = l["mlp"]["ff"]
            shapes.update({p + ".norm2": (Wd,), p + ".norm2b": (Wd,), p + ".mlp.gate": (ff, Wd), p + ".mlp.up": (ff, Wd),
                           p + ".mlp.down": (Wd, ff)})
    return shapes


def random_weights(cfg: dict, seed: int, gain: float = 1.0) -> Dict[str, torch.Tensor]:
    """Weights large enough that every mechanism moves the logits: matrices N(0, gain^2 / fan_in), norm weights near 1,
    decays spread between slow and fast; all rounded to bfloat16, the file's type."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "conv":
            t = 0.6 * torch.randn(shape, generator=g)
        elif len(shape) == 2:
            std = 0.5 if name == "embed" else gain / math.sqrt(shape[1])
            if leaf == "gate":
                std *= 2.0
            t = torch.randn(shape, generator=g) * std
        elif leaf.startswith("norm"):
            t = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif leaf == "A_log":
            t = torch.randn(shape, generator=g) - 1.0
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
