"""Plain, slow restatement of the Bovitar decoder -- TEST INFRASTRUCTURE, NOT PRODUCT CODE.

One function per mechanism, written from the design's equations in torch on the CPU, in one
floating-point type (float64 by default).  It shares nothing with gpustack_b200/: no kernels, no
cache, no scheduler; a sequence is processed whole, token by token where the design is a recurrence.

The design: pre-norm layers, x <- x + mixer(norm(x)), x <- x + ff(norm(x)), with RMS norms.  A layer may
use another layer's tensors (its state is its own).  Mixers:
  delta     a gated delta rule on convolved, silu-activated, unit-length queries and keys;
  parallel  causal softmax attention (convolved q / k / v, q and k normed over the whole projection, scaled
            half-split rotation, capped scores) beside a state-space recurrence with scalar decays (convolved
            inputs, gate before a grouped norm); half the sum of the two RMS-normed outputs.
Feed-forward: softmax-scored experts chosen by corrected scores inside the best groups of neighbours, weights not
renormalized, plus a shared expert.  Logits: head of the normed stream times a constant.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


# ------------------------------------------------------------------------------ norms
def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over its root mean square along the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit(x: torch.Tensor, eps: float = 1e-6) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + eps)


def grouped_rms(x: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """x [T, C]: `parts` equal neighbours, each over its own root mean square."""
    T, C = x.shape
    return rms(x.view(T, parts, C // parts), eps).view(T, C)


# ------------------------------------------------------------------------------ short causal convolution
def causal_conv(u: torch.Tensor, w: torch.Tensor, b: Optional[torch.Tensor] = None) -> torch.Tensor:
    """u [T, C] from a sequence's first token, w [C, taps] whose LAST column multiplies the current token; zeros
    before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u) if b is None else b.expand_as(u).clone()
    for back in range(taps):
        if back < T:
            y[back:] += w[:, taps - 1 - back] * u[:T - back]
    return y


# ------------------------------------------------------------------------------ rotation
def scaled_frequencies(rot: dict) -> List[float]:
    """dims / 2 angular frequencies; long wavelengths slowed by `factor`, short ones kept, a linear blend between."""
    out = []
    sc = rot.get("scaling")
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        if sc:
            wave = 2.0 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_half(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, dim]: entries i and i + dims/2 are turned by the angle position * f_i."""
    n = rot["dims"] // 2
    f = torch.tensor(scaled_frequencies(rot), dtype=torch.float64)
    a = (positions.to(torch.float64)[:, None] * f).to(x.dtype)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), x[..., 2 * n:]], dim=-1)


# ------------------------------------------------------------------------------ attention side
def capped_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, cap: float) -> torch.Tensor:
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]; head h reads key head h // (H / G), causal."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    later = torch.ones(T, T, dtype=torch.bool).triu(1)
    for h in range(H):
        g = h // (H // G)
        s = cap * torch.tanh((q[:, h] @ k[:, g].T) * scale / cap)
        out[:, h] = torch.softmax(s.masked_fill(later, -float("inf")), dim=-1) @ v[:, g]
    return out


def attention_inputs(h: torch.Tensor, w: Dict[str, torch.Tensor], mx: dict, eps: float) -> tuple:
    """Convolved projections; q and k normed over the whole projection, then rotated."""
    T = h.shape[0]
    H, G, dk, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    pos = torch.arange(T)
    q = rms(causal_conv(h @ w["q"].T, w["q.conv"]), eps) * w["q.norm"]
    k = rms(causal_conv(h @ w["k"].T, w["k.conv"]), eps) * w["k.norm"]
    v = causal_conv(h @ w["v"].T, w["v.conv"])
    return (rotate_half(q.view(T, H, dk), pos, mx["rot"]), rotate_half(k.view(T, G, dk), pos, mx["rot"]), v.view(T, G, dv))


def attention_side(h: torch.Tensor, w: Dict[str, torch.Tensor], mx: dict, eps: float) -> torch.Tensor:
    q, k, v = attention_inputs(h, w, mx, eps)
    return capped_attention(q, k, v, mx["scale"], mx["softcap"]).reshape(h.shape[0], -1) @ w["o"].T


# ------------------------------------------------------------------------------ state-space side
def ssd_scan(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, A_log: torch.Tensor,
             D: torch.Tensor) -> torch.Tensor:
    """x [T, H, P], B / C [T, G, N], dt [T, H] (positive) -> y [T, H, P]; state N x P per head, zero at the start."""
    T, H, P = x.shape
    G, N = B.shape[1], B.shape[2]
    y = torch.zeros_like(x)
    S = torch.zeros(H, N, P, dtype=x.dtype)
    of = torch.arange(H) // (H // G)                     # the group a head reads
    for t in range(T):
        S = torch.exp(-torch.exp(A_log) * dt[t])[:, None, None] * S + dt[t][:, None, None] * (B[t, of][:, :, None] * x[t][:, None, :])
        y[t] = torch.einsum("hnp,hn->hp", S, C[t, of]) + D[:, None] * x[t]
    return y


def state_space_side(h: torch.Tensor, w: Dict[str, torch.Tensor], mx: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, P, N, G = mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    x, B, C = torch.split(silu(causal_conv(xbc, w["conv"], w["conv.b"])), [inner, G * N, G * N], dim=-1)
    y = ssd_scan(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w["dt_bias"]), w["A_log"], w["D"])
    return (grouped_rms(y.reshape(T, inner) * silu(z), mx["norm_groups"], eps) * w["norm"]) @ w["o"].T


def parallel_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], mx: dict, eps: float) -> torch.Tensor:
    left = attention_side(h, _part(w, "left."), mx["left"], eps)
    right = state_space_side(h, _part(w, "right."), mx["right"], eps)
    return 0.5 * (rms(left, eps) * w["left.out"] + rms(right, eps) * w["right.out"])


# ------------------------------------------------------------------------------ gated delta rule
def delta_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor) -> torch.Tensor:
    """q, k [T, G, dk] as they enter the rule, v [T, H, dv], g / beta [T, H] -> o [T, H, dv]."""
    T, H, dv = v.shape
    G, dk = k.shape[1], k.shape[2]
    o = torch.zeros_like(v)
    S = torch.zeros(H, dk, dv, dtype=v.dtype)
    of = torch.arange(H) // (H // G)                     # the query / key head a value head reads
    for t in range(T):
        kt, qt = k[t, of], q[t, of]
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, kt))
        S = S + kt[:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, qt)
    return o


def delta_inputs(h: torch.Tensor, w: Dict[str, torch.Tensor], mx: dict) -> tuple:
    T = h.shape[0]
    H, G, dk, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in "qkv")
    g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    return (unit(q.view(T, G, dk)) * dk ** -0.5, unit(k.view(T, G, dk)), v.view(T, H, dv), g, torch.sigmoid(h @ w["b"].T))


def delta_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], mx: dict, eps: float) -> torch.Tensor:
    o = rms(delta_scan(*delta_inputs(h, w, mx)), eps) * w["norm"]
    return (o.reshape(h.shape[0], -1) * silu(h @ w["g"].T)) @ w["o"].T


# ------------------------------------------------------------------------------ routed feed-forward
def expert(x: torch.Tensor, w: Dict[str, torch.Tensor], name: str) -> torch.Tensor:
    return (silu(x @ w[name + ".gate"].T) * (x @ w[name + ".up"].T)) @ w[name + ".down"].T


def route(z: torch.Tensor, correction: torch.Tensor, router: dict) -> tuple:
    """z [T, E] logits -> chosen experts [T, top] and their weights."""
    s = torch.softmax(z, dim=-1)
    c = s + correction
    gr = router.get("groups")
    if gr:
        T, E = c.shape
        best = c.view(T, gr["count"], E // gr["count"]).max(dim=-1).values
        kept = torch.zeros_like(best, dtype=torch.bool).scatter(1, torch.topk(best, gr["keep"], dim=-1).indices, True)
        c = c.masked_fill(~kept.repeat_interleave(E // gr["count"], dim=1), -float("inf"))
    idx = torch.topk(c, router["top"], dim=-1).indices
    return idx, torch.gather(s, 1, idx) * router.get("scale", 1.0)


def moe_ff(x: torch.Tensor, w: Dict[str, torch.Tensor], mlp: dict) -> torch.Tensor:
    idx, wt = route(x @ w["router"].T, w["correction"], mlp["router"])
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for e, p in zip(idx[t].tolist(), wt[t]):
            out[t] += p * expert(x[t], w, f"e{e}")
    return out + expert(x, w, "shared") if mlp.get("shared") else out


# ------------------------------------------------------------------------------ the model
def _part(w: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


MIXERS = {"delta": delta_mixer, "parallel": parallel_mixer}


def owner(cfg: dict, l: int) -> int:
    """The layer whose tensors layer l uses."""
    while cfg["layers"][l].get("weights_of") is not None:
        l = cfg["layers"][l]["weights_of"]
    return l


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], trace: Optional[list] = None,
            dtype=torch.float64) -> torch.Tensor:
    """Logits [T, vocab] of one sequence from its first token.  trace: receives the residual after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)]
    for l, layer in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, l)}."
        x = x + MIXERS[layer["type"]](rms(x, eps) * w[p + "norm1"], _part(w, p + "mix."), layer["mixer"], eps)
        if layer.get("mlp"):
            x = x + moe_ff(rms(x, eps) * w[p + "norm2"], _part(w, p + "mlp."), layer["mlp"])
        if trace is not None:
            trace.append(x.clone())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T * cfg["logit_scale"]


# ------------------------------------------------------------------------------ random checkpoints
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    W, V = cfg["width"], cfg["vocab"]
    out: Dict[str, tuple] = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}

    def convolved(p, n, rows, taps):
        out[p + n], out[p + n + ".conv"] = (rows, W), (rows, taps)

    for l, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, mx, mlp = f"l{l}.mix.", layer["mixer"], layer.get("mlp")
        out[f"l{l}.norm1"] = (W,)
        if layer["type"] == "delta":
            H, G, dk, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
            for n, rows in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                convolved(p, n, rows, mx["conv"])
            out[p + "a"] = out[p + "b"] = (H, W)
            out[p + "A_log"] = out[p + "dt_bias"] = (H,)
            out[p + "g"], out[p + "norm"], out[p + "o"] = (H * dv, W), (dv,), (W, H * dv)
        else:
            a, r = mx["left"], mx["right"]
            for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                convolved(p + "left.", n, rows, a["conv"])
                if n != "v":
                    out[p + f"left.{n}.norm"] = (rows,)
            out[p + "left.o"] = (W, a["heads"] * a["vdim"])
            inner, bc = r["heads"] * r["vdim"], 2 * r["groups"] * r["state"]
            out[p + "right.in"] = (2 * inner + bc + r["heads"], W)
            out[p + "right.conv"], out[p + "right.conv.b"] = (inner + bc, r["conv"]), (inner + bc,)
            out[p + "right.A_log"] = out[p + "right.D"] = out[p + "right.dt_bias"] = (r["heads"],)
            out[p + "right.norm"], out[p + "right.o"] = (inner,), (W, inner)
            out[p + "left.out"] = out[p + "right.out"] = (W,)
        if not mlp:
            continue
        q = f"l{l}.mlp."
        out[f"l{l}.norm2"] = (W,)
        E = mlp["router"]["experts"]
        out[q + "router"], out[q + "correction"] = (E, W), (E,)
        for e, ff in [(f"e{i}", mlp["expert"]["ff"]) for i in range(E)] + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else []):
            out[q + e + ".gate"] = out[q + e + ".up"] = (ff, W)
            out[q + e + ".down"] = (W, ff)
    return out


def random_weights(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Seeded bf16 weights: linear weights N(0, 1 / in), norm weights around one, taps of half, decays between fast and slow,
    router logits and corrections that decide most choices clearly."""
    g = torch.Generator().manual_seed(seed)
    out: Dict[str, torch.Tensor] = {}
    for name, shape in tensor_shapes(cfg).items():
        x = torch.randn(tuple(shape), generator=g)
        leaf = name.split(".")[-1]
        if leaf == "A_log":
            x = x - 1.0
        elif leaf == "dt_bias":
            x = x - 2.0
        elif leaf == "D":
            x = 1.0 + 0.3 * x
        elif leaf == "b" and name.endswith("conv.b"):
            x = 0.3 * x
        elif leaf == "correction":
            x = 0.2 * x
        elif leaf == "conv":
            x = 0.5 * x
        elif leaf in ("norm", "norm1", "norm2", "out"):
            x = 1.0 + 0.2 * x
        elif leaf == "router":
            x = 3.0 * x / shape[-1] ** 0.5
        elif name != "embed":
            x = x / shape[-1] ** 0.5
        out[name] = x.to(torch.bfloat16)
    return out
