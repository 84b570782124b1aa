"""A plain, slow restatement of the Ratesun design: one function per mechanism, python loops over tokens and heads,
float64 by default.  It shares no code with ``mdi_llm_b200``; the tests compare the framework with it.

Notation: ``x`` a residual row, ``h`` what a sublayer reads, ``t`` a position counted from 0 in its own sequence,
``W["name"]`` the tensors by checkpoint name.
"""
from __future__ import annotations

import math
from typing import Any, Dict, List, Optional

import torch

DT = torch.float64


def rms(x: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean() + eps)
    return y if w is None else y * w


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean()
    return d / torch.sqrt((d * d).mean() + eps) * w + b


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float) -> torch.Tensor:
    """Three powers of the vector, each divided by its own root mean square, mixed by three numbers, plus a constant."""
    return coef[0] * rms(z, None, eps) + coef[1] * rms(z ** 2, None, eps) + coef[2] * rms(z ** 3, None, eps) + coef[3]


def embed(W: Dict[str, torch.Tensor], cfg: Dict[str, Any], token: int, previous: Optional[int]) -> torch.Tensor:
    b = cfg["embedding"]["bigram"]
    row = b["buckets"] if previous is None else (previous * b["mul_prev"] + token * b["mul_cur"]) % b["buckets"]
    return W["embed"][token] + W["bigram"][row]


def short_conv(w: torch.Tensor, past: List[torch.Tensor]) -> torch.Tensor:
    """``past`` holds h_0 .. h_t; the last column of ``w [C, taps]`` weighs h_t, the one before h_(t-1), and so on."""
    taps = w.shape[1]
    y = torch.zeros_like(past[-1])
    for back in range(min(taps, len(past))):
        y = y + w[:, taps - 1 - back] * past[-1 - back]
    return past[-1] + y


def turn_pairs(v: torch.Tensor, t: int, ndims: int, base: float) -> torch.Tensor:
    """Neighbours (2i, 2i+1) of the first ``ndims`` entries turn by the angle t * base^(-2i/ndims)."""
    out = v.clone()
    for i in range(ndims // 2):
        a = t * base ** (-2.0 * i / ndims)
        out[2 * i] = v[2 * i] * math.cos(a) - v[2 * i + 1] * math.sin(a)
        out[2 * i + 1] = v[2 * i + 1] * math.cos(a) + v[2 * i] * math.sin(a)
    return out


def latent_row(W: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], h: torch.Tensor, t: int, eps: float):
    """What a layer with its own ``dkv`` remembers of a token: the normed latent and the rotated shared key part."""
    z = W[pre + "dkv"] @ h
    L = m["kv_rank"]
    return rms(z[:L], W[pre + "dkv.norm"], eps), turn_pairs(z[L:], t, m["rot"]["dims"], m["rot"]["base"])


def softmax(s: torch.Tensor) -> torch.Tensor:
    e = torch.exp(s - s.max())
    return e / e.sum()


def latent_attention(W: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], h: torch.Tensor, t: int, eps: float,
                     latents: List[torch.Tensor], rotated: List[torch.Tensor]) -> torch.Tensor:
    """``latents`` / ``rotated`` hold positions 0 .. t (this layer's own, or those of the layer it borrows from)."""
    D, R, V = m["dim"], m["rot_dim"], m["vdim"]
    q = W[pre + "uq"] @ rms(W[pre + "dq"] @ h, W[pre + "dq.norm"], eps)
    size = (m.get("mask") or {}).get("size", 0)
    first = max(0, t - size + 1) if size else 0
    C, K = torch.stack(latents[first:t + 1]), torch.stack(rotated[first:t + 1])
    outs = []
    for a in range(m["heads"]):
        qa = q[a * (D + R):(a + 1) * (D + R)]
        qr = turn_pairs(qa[D:], t, m["rot"]["dims"], m["rot"]["base"])
        keys = C @ W[pre + "uk"][a * D:(a + 1) * D].T
        values = C @ W[pre + "uv"][a * V:(a + 1) * V].T
        outs.append(softmax((keys @ qa[:D] + K @ qr) * m["scale"]) @ values)
    return W[pre + "o"] @ torch.cat(outs)


def feed_forward(W: Dict[str, torch.Tensor], pre: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    return W[pre + "down"] @ poly_norm(W[pre + "up"] @ h, W[pre + "act"], eps)


def token_side(W: Dict[str, torch.Tensor], i: int, dim: int, x: torch.Tensor, token: int, eps: float) -> torch.Tensor:
    e = W["side.embed"][token][i * dim:(i + 1) * dim]
    return rms(W[f"l{i}.side.proj"] @ (gelu_tanh(W[f"l{i}.side.gate"] @ x) * e), W[f"l{i}.side.norm"], eps)


def depth_average(weights: torch.Tensor, rows: List[torch.Tensor]) -> torch.Tensor:
    assert len(weights) == len(rows)
    y = torch.zeros_like(rows[0])
    for w, x in zip(weights, rows):
        y = y + w * x
    return y


def forward(cfg: Dict[str, Any], W: Dict[str, torch.Tensor], tokens: List[int], dtype: torch.dtype = DT,
            layers_out: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits ``[len(tokens), vocab]`` of one sequence, token by token.  ``layers_out`` receives the stream every layer
    passes on as ``[layers, tokens, width]``."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps, mult, L = cfg["norm"]["eps"], cfg["residual_mult"], cfg["layers"]
    latents, rotated = [[] for _ in L], [[] for _ in L]
    seen1, seen2 = [[] for _ in L], [[] for _ in L]
    per_layer = [[] for _ in L]
    logits = []
    for t, tok in enumerate(tokens):
        x = embed(W, cfg, tok, tokens[t - 1] if t else None)
        results = [x]
        for i, spec in enumerate(L):
            m, n = spec["mixer"], lambda name, v: layer_norm(v, W[f"l{i}.{name}"], W[f"l{i}.{name}.b"], eps)  # noqa: E731
            seen1[i].append(n("norm1", x))
            h = short_conv(W[f"l{i}.canon1"], seen1[i])
            src = m.get("kv_from")
            if src is None:
                c, k = latent_row(W, f"l{i}.mix.", m, h, t, eps)
                latents[i].append(c)
                rotated[i].append(k)
                src = i
            x = x + mult * n("norm1b", latent_attention(W, f"l{i}.mix.", m, h, t, eps, latents[src], rotated[src]))
            if spec.get("mlp"):
                seen2[i].append(n("norm2", x))
                h = short_conv(W[f"l{i}.canon2"], seen2[i])
                x = x + mult * n("norm2b", feed_forward(W, f"l{i}.mlp.", h, eps))
            if cfg.get("token_side"):
                x = x + mult * token_side(W, i, cfg["token_side"]["dim"], x, tok, eps)
            results.append(x)
            x = depth_average(W[f"l{i}.dwa"], results)
            per_layer[i].append(x)
        logits.append(W["embed"] @ layer_norm(x, W["final.norm"], W["final.norm.b"], eps) * cfg["logit_scale"])
    if layers_out is not None:
        layers_out.append(torch.stack([torch.stack(rows) for rows in per_layer]))
    return torch.stack(logits)


def random_tensors(cfg: Dict[str, Any], seed: int = 0) -> Dict[str, torch.Tensor]:
    """Weights by checkpoint name for ``cfg``, rounded to bfloat16 values (kept in float32)."""
    g = torch.Generator().manual_seed(seed)
    C = cfg["width"]

    def mat(o: int, i: int, gain: float = 1.0) -> torch.Tensor:
        return torch.randn(o, i, generator=g) * gain / math.sqrt(i)

    def vec(n: int, mean: float = 0.0, std: float = 0.3) -> torch.Tensor:
        return mean + torch.randn(n, generator=g) * std

    W = {"embed": torch.randn(cfg["vocab"], C, generator=g),
         "bigram": torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, C, generator=g)}

    def norm(name: str) -> None:
        W[name], W[name + ".b"] = vec(C, 1.0, 0.1), vec(C, 0.0, 0.1)

    norm("final.norm")
    sd = (cfg.get("token_side") or {}).get("dim", 0)
    if sd:
        W["side.embed"] = torch.randn(cfg["vocab"], sd * len(cfg["layers"]), generator=g)
    for i, spec in enumerate(cfg["layers"]):
        m, pre = spec["mixer"], f"l{i}.mix."
        H, D, R, V, L, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
        norm(f"l{i}.norm1")
        norm(f"l{i}.norm1b")
        W[f"l{i}.canon1"] = vec(C * cfg["canon"]["taps"], 0.0, 0.4).view(C, -1)
        W[pre + "dq"], W[pre + "dq.norm"], W[pre + "uq"] = mat(Q, C), vec(Q, 1.0, 0.2), mat(H * (D + R), Q, 2.0)
        if m.get("kv_from") is None:
            W[pre + "dkv"], W[pre + "dkv.norm"] = mat(L + R, C), vec(L, 1.0, 0.2)
        W[pre + "uk"], W[pre + "uv"], W[pre + "o"] = mat(H * D, L, 2.0), mat(H * V, L), mat(C, H * V)
        if spec.get("mlp"):
            norm(f"l{i}.norm2")
            norm(f"l{i}.norm2b")
            W[f"l{i}.canon2"] = vec(C * cfg["canon"]["taps"], 0.0, 0.4).view(C, -1)
            W[f"l{i}.mlp.up"], W[f"l{i}.mlp.down"] = mat(spec["mlp"]["ff"], C), mat(C, spec["mlp"]["ff"])
            W[f"l{i}.mlp.act"] = torch.tensor([0.7, -0.4, 0.5, 0.1]) + vec(4, 0.0, 0.2)
        if sd:
            W[f"l{i}.side.gate"], W[f"l{i}.side.proj"], W[f"l{i}.side.norm"] = mat(sd, C), mat(C, sd), vec(C, 0.8, 0.2)
        w = vec(i + 2, 0.0, 0.3)
        w[-1] += 1.0
        W[f"l{i}.dwa"] = w
    return {k: v.to(torch.bfloat16).float() for k, v in W.items()}
