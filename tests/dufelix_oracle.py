"""A plain, slow restatement of the Dufelix design: one function per mechanism, python loops over tokens and heads,
float64 by default.  It shares no code with ``mdi_llm_b200``; the tests compare the framework with it.

Notation: ``x`` a residual row, ``h`` what a sublayer reads, ``t`` a position counted from 0 in its own sequence,
``W["name"]`` the tensors by checkpoint name.  ``i`` is a layer run, ``src(i)`` the layer whose tensors it uses.
"""
from __future__ import annotations

import math
from typing import Any, Dict, List, Optional

import torch

DT = torch.float64


def rms(x: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean() + eps)
    return y if w is None else y * w


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.maximum(z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- rotary positions ----------------------------------------------------------------------------------------
def frequencies(rot: Dict[str, Any]) -> List[float]:
    """One frequency per rotated pair; with a scaling entry, the low ones (long wavelengths) are divided by the factor
    and a linear ramp over the pair's index joins the two regions."""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not sc:
        return f

    def index_of(turns: float) -> float:  # the pair index that makes `turns` turns over the original length
        return n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(sc["fast"])), 0)
    hi = min(math.ceil(index_of(sc["slow"])), n - 1)
    out = []
    for i in range(n // 2):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f[i] / sc["factor"] * r + f[i] * (1.0 - r))
    return out


def amplitude(rot: Dict[str, Any]) -> float:
    return 0.1 * math.log(rot["scaling"]["factor"]) + 1.0 if rot.get("scaling") else 1.0


def turn(v: torch.Tensor, t: int, rot: Dict[str, Any], neighbours: bool) -> torch.Tensor:
    """The first ``dims`` entries of ``v`` turned for position ``t``: pairs (2i, 2i+1) or (i, i + dims/2)."""
    out, n, amp = v.clone(), rot["dims"], amplitude(rot)
    for i, f in enumerate(frequencies(rot)):
        a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + n // 2)
        c, s = math.cos(t * f) * amp, math.sin(t * f) * amp
        out[a] = v[a] * c - v[b] * s
        out[b] = v[b] * c + v[a] * s
    return out


# ---- mixers --------------------------------------------------------------------------------------------------
def softmax_sum(s: torch.Tensor, values: torch.Tensor, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Softmax-weighted sum; ``sink`` is one more score in the denominator, without a value."""
    top = s.max() if sink is None else torch.maximum(s.max(), sink)
    e = torch.exp(s - top)
    den = e.sum() if sink is None else e.sum() + torch.exp(sink - top)
    return (e / den) @ values


def attention(W: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], h: torch.Tensor, t: int, eps: float, st: Dict[str, Any]) -> torch.Tensor:
    Hh, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v, g = W[pre + "q"] @ h, W[pre + "k"] @ h, W[pre + "v"] @ h, W[pre + "g"] @ h
    st.setdefault("k", []).append(torch.stack([turn(k[a * D:(a + 1) * D], t, m["rot"], False) for a in range(G)]))
    st.setdefault("v", []).append(v.view(G, V))
    K, Vs, outs = torch.stack(st["k"]), torch.stack(st["v"]), []
    for a in range(Hh):
        b = a // (Hh // G)
        s = K[:, b] @ turn(q[a * D:(a + 1) * D], t, m["rot"], False) * m["scale"]
        outs.append(softmax_sum(s, Vs[:, b]) * sigmoid(g[a]))
    return W[pre + "o"] @ torch.cat(outs)


def latent_attention(W: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], h: torch.Tensor, t: int, eps: float, st: Dict[str, Any]) -> torch.Tensor:
    Hh, D, R, V, L = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = W[pre + "uq"] @ rms(W[pre + "dq"] @ h, W[pre + "dq.norm"], eps)
    z = W[pre + "dkv"] @ h
    st.setdefault("c", []).append(rms(z[:L], W[pre + "dkv.norm"], eps))
    st.setdefault("r", []).append(turn(z[L:], t, m["rot"], True))
    C, K, outs = torch.stack(st["c"]), torch.stack(st["r"]), []
    for a in range(Hh):
        qa = q[a * (D + R):(a + 1) * (D + R)]
        keys = C @ W[pre + "uk"][a * D:(a + 1) * D].T
        values = C @ W[pre + "uv"][a * V:(a + 1) * V].T
        s = (keys @ qa[:D] + K @ turn(qa[D:], t, m["rot"], True)) * m["scale"]
        outs.append(softmax_sum(s, values, W[pre + "sink"][a]))
    return W[pre + "o"] @ torch.cat(outs)


def short_conv(w: torch.Tensor, b: torch.Tensor, past: List[torch.Tensor]) -> torch.Tensor:
    """``past`` holds the inputs of positions 0 .. t; the last column of ``w [channels, taps]`` weighs position t."""
    taps, y = w.shape[1], b.clone()
    for back in range(min(taps, len(past))):
        y = y + w[:, taps - 1 - back] * past[-1 - back]
    return y


def state_step(S: torch.Tensor, x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, a_log: torch.Tensor, D: torch.Tensor):
    """One head, one token: the decayed state takes in ``dt B x^T`` and is read by ``C``; ``D x`` passes by it."""
    S = torch.exp(-torch.exp(a_log) * dt) * S + dt * B[:, None] * x[None, :]
    return S, S.T @ C + D * x


def gate_and_norm(y: torch.Tensor, z: torch.Tensor, w: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    y = y * silu(z)
    return torch.cat([rms(p, None, eps) for p in y.chunk(parts)]) * w


def mamba2(W: Dict[str, torch.Tensor], pre: str, m: Dict[str, Any], h: torch.Tensor, t: int, eps: float, st: Dict[str, Any]) -> torch.Tensor:
    Hh, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = Hh * V
    z, xbc, dt = torch.split(W[pre + "in"] @ h, [inner, inner + 2 * G * N, Hh])
    st.setdefault("conv", []).append(xbc)
    x, B, C = torch.split(silu(short_conv(W[pre + "conv"], W[pre + "conv.b"], st["conv"])), [inner, G * N, G * N])
    dt = softplus(dt + W[pre + "dt_bias"])
    S, ys = st.setdefault("S", [torch.zeros(N, V, dtype=h.dtype) for _ in range(Hh)]), []
    for a in range(Hh):
        g = a // (Hh // G)
        S[a], y = state_step(S[a], x[a * V:(a + 1) * V], B[g * N:(g + 1) * N], C[g * N:(g + 1) * N], dt[a], W[pre + "A_log"][a], W[pre + "D"][a])
        ys.append(y)
    return W[pre + "o"] @ gate_and_norm(torch.cat(ys), z, W[pre + "norm"], m["norm_groups"], eps)


MIXERS = {"attention": attention, "latent_attention": latent_attention, "mamba2": mamba2}


def feed_forward(W: Dict[str, torch.Tensor], pre: str, h: torch.Tensor) -> torch.Tensor:
    return W[pre + "down"] @ (gelu_tanh(W[pre + "gate"] @ h) * (W[pre + "up"] @ h))


# ---- the model -----------------------------------------------------------------------------------------------
def src(cfg: Dict[str, Any], i: int) -> int:
    j = cfg["layers"][i].get("weights_of")
    return i if j is None else int(j)


def forward(cfg: Dict[str, Any], W: Dict[str, torch.Tensor], tokens: List[int], dtype: torch.dtype = DT,
            layers_out: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    """Logits ``[len(tokens), vocab]`` of one sequence, token by token.  ``layers_out`` receives the stream after every
    layer as ``[layers, tokens, width]``."""
    W = {k: v.to(dtype) for k, v in W.items()}
    eps, layers = cfg["norm"]["eps"], cfg["layers"]
    states: List[Dict[str, Any]] = [{} for _ in layers]
    per_layer: List[List[torch.Tensor]] = [[] for _ in layers]
    logits = []
    for t, tok in enumerate(tokens):
        x = W["embed"][tok] * cfg["embedding"]["scale"]
        for i, spec in enumerate(layers):
            p = f"l{src(cfg, i)}."
            y = MIXERS[spec["type"]](W, p + "mix.", spec["mixer"], rms(x, W[p + "norm1"], eps), t, eps, states[i])
            x = x + rms(y, W[p + "norm1b"], eps)
            if spec.get("mlp"):
                x = x + rms(feed_forward(W, p + "mlp.", rms(x, W[p + "norm2"], eps)), W[p + "norm2b"], eps)
            per_layer[i].append(x)
        logits.append(W["head"] @ rms(x, W["final.norm"], eps))
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

    W = {"embed": torch.randn(cfg["vocab"], C, generator=g) / cfg["embedding"]["scale"], "head": mat(cfg["vocab"], C),
         "final.norm": vec(C, 1.0, 0.1)}
    for i, spec in enumerate(cfg["layers"]):
        if src(cfg, i) != i:
            continue
        m, pre = spec["mixer"], f"l{i}.mix."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if spec.get("mlp") else ()):
            W[f"l{i}.{n}"] = vec(C, 0.4 if n.endswith("b") else 1.0, 0.1)
        if spec["type"] == "attention":
            Hh, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            W[pre + "q"], W[pre + "k"], W[pre + "v"] = mat(Hh * D, C), mat(G * D, C), mat(G * V, C)
            W[pre + "g"], W[pre + "o"] = mat(Hh, C, 2.0), mat(C, Hh * V)
        elif spec["type"] == "latent_attention":
            Hh, D, R, V, L, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            W[pre + "dq"], W[pre + "dq.norm"], W[pre + "uq"] = mat(Q, C), vec(Q, 1.0, 0.2), mat(Hh * (D + R), Q, 1.5)
            W[pre + "dkv"], W[pre + "dkv.norm"] = mat(L + R, C), vec(L, 1.0, 0.2)
            W[pre + "uk"], W[pre + "uv"], W[pre + "o"] = mat(Hh * D, L, 1.5), mat(Hh * V, L), mat(C, Hh * V)
            W[pre + "sink"] = vec(Hh, 1.0, 1.0)
        else:
            Hh, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            ch = Hh * V + 2 * G * N
            W[pre + "in"], W[pre + "o"] = mat(Hh * V + ch + Hh, C), mat(C, Hh * V)
            W[pre + "conv"], W[pre + "conv.b"] = vec(ch * m["conv"], 0.0, 0.5).view(ch, -1), vec(ch)
            W[pre + "dt_bias"], W[pre + "A_log"], W[pre + "D"] = vec(Hh, -1.5, 1.0), vec(Hh, 0.0, 1.0), vec(Hh, 0.5, 0.5)
            W[pre + "norm"] = vec(Hh * V, 1.0, 0.2)
        if spec.get("mlp"):
            ff = spec["mlp"]["ff"]
            W[f"l{i}.mlp.gate"], W[f"l{i}.mlp.up"], W[f"l{i}.mlp.down"] = mat(ff, C), mat(ff, C), mat(C, ff)
    return {k: v.to(torch.bfloat16).float() for k, v in W.items()}
