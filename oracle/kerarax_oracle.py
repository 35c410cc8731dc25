"""Plain, slow restatement of the Kerarax decoder -- TEST INFRASTRUCTURE, NOT PRODUCT CODE.

One function per mechanism, written from the design's equations in torch on the CPU, in one
floating-point type (float64 by default).  It shares nothing with gpustack_b200/: no kernels, no
cache, no scheduler; a sequence is processed whole.

The design: x_0 = LN(embed[token] + s(p)) with a fixed sinusoidal vector s; layers that norm what a sublayer
PUTS OUT and nothing else, x <- x + LN(f(x)); LN is a layer norm with weight and bias.  The mixer is grouped softmax
attention without rotation: q, k and v each pass a short causal convolution per channel, q and k a weighted RMS norm
per head, the scaled score is capped by a tanh and the softmax denominator has one more term of size one.  The
feed-forward routes each token to some experts (weights: a softmax over the chosen logits alone) and adds a shared
expert under a gate of one number per token; an expert is down(relu(up x)^2).  The output logits are capped as the
scores are.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch


# ------------------------------------------------------------------------------ norms
def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w + b


def head_rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """x [T, heads, dim]: every head over its own root mean square, one weight vector for all heads."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


# ------------------------------------------------------------------------------ embedding
def sinusoid(positions: torch.Tensor, width: int, dtype=torch.float64) -> torch.Tensor:
    """[T, width]: entries 2i and 2i + 1 are sine and cosine of p * 10000^(-2i/width)."""
    out = torch.zeros(len(positions), width, dtype=dtype)
    for d in range(width):
        a = positions.to(dtype) * 10000.0 ** (-2.0 * (d // 2) / width)
        out[:, d] = torch.sin(a) if d % 2 == 0 else torch.cos(a)
    return out


# ------------------------------------------------------------------------------ short causal convolution
def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [T, C] from a sequence's first token, w [C, taps] whose LAST column multiplies the current token; zeros
    before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for back in range(taps):
        if back < T:
            y[back:] += w[:, taps - 1 - back] * u[:T - back]
    return y


# ------------------------------------------------------------------------------ capped attention
def soft_cap(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


def softmax_plus_one(s: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum exp(s_j)) along the last dimension."""
    m = torch.clamp(s.max(dim=-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(dim=-1, keepdim=True))


def capped_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, cap: float) -> torch.Tensor:
    """q [T, H, dk], k [T, G, dk], v [T, G, dv] -> [T, H, dv]; head h reads key head h // (H / G), causal."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    later = torch.ones(T, T, dtype=torch.bool).triu(1)
    for h in range(H):
        g = h // (H // G)
        s = soft_cap((q[:, h] @ k[:, g].T) * scale, cap).masked_fill(later, -float("inf"))
        out[:, h] = softmax_plus_one(s) @ v[:, g]
    return out


def attention_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], mx: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, dk, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = causal_conv(h @ w["q"].T, w["q.conv"]).view(T, H, dk)
    k = causal_conv(h @ w["k"].T, w["k.conv"]).view(T, G, dk)
    v = causal_conv(h @ w["v"].T, w["v.conv"]).view(T, G, dv)
    q, k = head_rms_norm(q, w["q.norm"], eps), head_rms_norm(k, w["k.norm"], eps)
    return capped_attention(q, k, v, mx["scale"], mx["softcap"]).reshape(T, H * dv) @ w["o"].T


# ------------------------------------------------------------------------------ routed feed-forward
def relu2_expert(x: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return torch.clamp(x @ up.T, min=0.0) ** 2 @ down.T


def route(z: torch.Tensor, top: int) -> tuple:
    """z [T, E] router logits with their bias: the `top` largest and a softmax over those alone."""
    val, idx = torch.topk(z, top, dim=-1)
    return idx, torch.softmax(val, dim=-1)


def moe_ff(x: torch.Tensor, w: Dict[str, torch.Tensor], mlp: dict) -> torch.Tensor:
    idx, wt = route(x @ w["router"].T + w["router.b"], mlp["router"]["top"])
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for e, p in zip(idx[t].tolist(), wt[t]):
            out[t] += p * relu2_expert(x[t], w[f"e{e}.up"], w[f"e{e}.down"])
    if mlp.get("shared"):
        out = out + torch.sigmoid(x @ w["shared.sg"].T) * relu2_expert(x, w["shared.up"], w["shared.down"])
    return out


# ------------------------------------------------------------------------------ the model
def _part(w: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], trace: Optional[list] = None,
            dtype=torch.float64) -> torch.Tensor:
    """Logits [T, vocab] of one sequence from its first token.  trace: receives the residual after every layer."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]

    def norm(x, name):
        return layer_norm(x, w[name], w[name + ".b"], eps)

    x = w["embed"][torch.tensor(tokens)] + sinusoid(torch.arange(len(tokens)), cfg["width"], dtype)
    x = norm(x, "embed.norm")
    for l, layer in enumerate(cfg["layers"]):
        p = f"l{l}."
        x = x + norm(attention_mixer(x, _part(w, p + "mix."), layer["mixer"], eps), p + "norm1")
        if layer.get("mlp"):
            x = x + norm(moe_ff(x, _part(w, p + "mlp."), layer["mlp"]), p + "norm2")
        if trace is not None:
            trace.append(x.clone())
    return soft_cap(norm(x, "final.norm") @ w["head"].T, cfg["logit_softcap"])


# ------------------------------------------------------------------------------ random checkpoints
def tensor_shapes(cfg: dict) -> Dict[str, tuple]:
    D, V = cfg["width"], cfg["vocab"]
    out: Dict[str, tuple] = {"embed": (V, D), "head": (V, D)}

    def norm(name):
        out[name] = out[name + ".b"] = (D,)

    norm("embed.norm")
    norm("final.norm")
    for l, layer in enumerate(cfg["layers"]):
        p, mx, mlp = f"l{l}.", layer["mixer"], layer.get("mlp")
        norm(p + "norm1")
        for n, rows in (("q", mx["heads"] * mx["dim"]), ("k", mx["kv_heads"] * mx["dim"]), ("v", mx["kv_heads"] * mx["vdim"])):
            out[p + "mix." + n] = (rows, D)
            out[p + f"mix.{n}.conv"] = (rows, mx["conv"])
        out[p + "mix.q.norm"] = out[p + "mix.k.norm"] = (mx["dim"],)
        out[p + "mix.o"] = (D, mx["heads"] * mx["vdim"])
        if not mlp:
            continue
        norm(p + "norm2")
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        out[p + "mlp.router"], out[p + "mlp.router.b"] = (E, D), (E,)
        for e in range(E):
            out[p + f"mlp.e{e}.up"], out[p + f"mlp.e{e}.down"] = (ff, D), (D, ff)
        if mlp.get("shared"):
            fs = mlp["shared"]["ff"]
            out[p + "mlp.shared.up"], out[p + "mlp.shared.down"], out[p + "mlp.shared.sg"] = (fs, D), (D, fs), (1, D)
    return out


def random_weights(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Seeded bf16 weights: linear weights N(0, 1 / in), norm weights around one, biases of a few tenths, convolution taps
    of half."""
    g = torch.Generator().manual_seed(seed)
    out: Dict[str, torch.Tensor] = {}
    for name, shape in tensor_shapes(cfg).items():
        x = torch.randn(tuple(shape), generator=g)
        leaf = name.split(".")[-1]
        if leaf == "b":
            x = 0.3 * x
        elif leaf == "conv":
            x = 0.5 * x
        elif leaf in ("norm", "norm1", "norm2"):
            x = 1.0 + 0.2 * x
        elif name != "embed":
            x = x / shape[-1] ** 0.5
        out[name] = x.to(torch.bfloat16)
    return out
