"""Plain float64 evaluation of a Vezodra stack, one function per mechanism, whole sequences at a time and nothing cached.
It shares no code with the package: the tests compare the engine (paged cache, carried state, ragged batches, kernels)
with it.

``config`` is the model's ``config.json`` object and ``tensors`` maps checkpoint names to arrays (any float dtype).

The stack: ``x = embed[token]``; a layer adds mixer and feed-forward of the SAME stream, ``x += mixer(c(norm1 x)) +
ff(norm2 x)`` with ``c(h) = h + filter(h)``, a short causal filter per channel; a span of layers runs several times in a
row; final norm, and the embedding table as the head.  Mixers: softmax attention whose values are the keys before their
rotation, and a pair of mixers side by side (windowed attention, delta rule with separate removal and decay vectors)
whose normalised outputs are averaged.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def rms_norm(x: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)
    return y if w is None else y * w


def causal_filter(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``u`` [T, C], ``w`` [C, taps]: ``y[t] = sum_j w[:, j] * u[t - taps + 1 + j]`` with zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[: T - back]
    return y


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------------ rotation
def rotary_angles(T: int, rot: Dict) -> torch.Tensor:
    """``[T, dims / 2]``: the angle of pair i at position p, ``p * base^(-2i / dims) / factor``."""
    dims, base = int(rot["dims"]), float(rot["base"])
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    f = torch.tensor([base ** (-2.0 * i / dims) / factor for i in range(dims // 2)], dtype=F64)
    return torch.arange(T, dtype=F64)[:, None] * f[None, :]


def rotate(x: torch.Tensor, rot: Dict, interleaved: bool) -> torch.Tensor:
    """``x`` [T, heads, n]: the first ``dims`` channels turn in pairs -- (2i, 2i+1) if ``interleaved``, else (i, i + dims/2)
    -- and the channels behind them pass."""
    dims = int(rot["dims"])
    ang = rotary_angles(x.shape[0], rot)[:, None, :]
    c, s = torch.cos(ang), torch.sin(ang)
    first = torch.arange(0, dims, 2) if interleaved else torch.arange(dims // 2)
    second = first + 1 if interleaved else first + dims // 2
    out = x.clone()
    u, v = x[..., first], x[..., second]
    out[..., first] = u * c - v * s
    out[..., second] = v * c + u * s
    return out


# ------------------------------------------------------------------------------------------------ attention
def softmax_rows(s: torch.Tensor, visible: torch.Tensor, extra_one: bool) -> torch.Tensor:
    """Softmax over the visible entries of every row; ``extra_one`` adds 1 to the denominator of the unshifted exponentials."""
    s = s.masked_fill(~visible, float("-inf"))
    top = s.max(dim=-1, keepdim=True).values
    if extra_one:
        top = top.clamp(min=0.0)
    e = torch.exp(s - top)
    den = e.sum(dim=-1, keepdim=True)
    return e / (den + torch.exp(-top) if extra_one else den)


def attend(q, k, v, scale, window: int, extra_one: bool, temp: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``q`` [T, H, d], ``k`` [T, G, d], ``v`` [T, G, dv] -> [T, H, dv]; ``window`` 0 sees every earlier position."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    i = torch.arange(T)
    dist = i[:, None] - i[None, :]
    visible = dist >= 0
    if window > 0:
        visible &= dist < window
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * scale
        if temp is not None:
            s = s * temp[h]
        out[:, h] = softmax_rows(s, visible, extra_one) @ v[:, g]
    return out


def key_value_attention(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict, eps: float) -> torch.Tensor:
    """The values are the projected keys before rotation; one temperature and one sigmoid gate per query head."""
    T = h.shape[0]
    H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q, k = (h @ P["q"].T).view(T, H, d), (h @ P["k"].T).view(T, G, d)
    o = attend(rotate(q, m["rot"], True), rotate(k, m["rot"], True), k, float(m["scale"]), 0, True, P["temp"])
    o = o * torch.sigmoid(h @ P["g"].T)[:, :, None]
    return o.reshape(T, H * d) @ P["o"].T


def windowed_attention(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict, eps: float) -> torch.Tensor:
    """Query and key rows are normalised over ALL heads at once before they are split, then rotated in halves."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms_norm(h @ P["q"].T, P["q.norm"], eps).view(T, H, d)
    k = rms_norm(h @ P["k"].T, P["k.norm"], eps).view(T, G, d)
    v = (h @ P["v"].T).view(T, G, dv)
    o = attend(rotate(q, m["rot"], False), rotate(k, m["rot"], False), v, float(m["scale"]), int(m["mask"]["size"]), False)
    return o.reshape(T, H * dv) @ P["o"].T


# ------------------------------------------------------------------------------------------------ recurrence
def removal_gates(h: torch.Tensor, P: Dict[str, torch.Tensor]):
    """(decay, removal rate) ``[T, heads * dim]``: ``exp(-e^(-1/2) sigmoid(w2 tanh(w1 h) + w0))`` and ``sigmoid(a h + b)``."""
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(h @ P["w1"].T) @ P["w2"].T + P["w0"]))
    return decay, torch.sigmoid(h @ P["a"].T + P["a.b"])


def removal_recurrence(r, k, v, decay, rate, state: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One head, ``[T, n]`` each.  With ``u = k / |k|``: ``S <- diag(decay) S - (rate * u) (u^T S) + k v^T`` (both terms read
    the old ``S`` [key channel, value channel]), ``o = S^T r``."""
    T, n = k.shape
    S = torch.zeros(n, v.shape[1], dtype=F64) if state is None else state
    out = torch.zeros(T, v.shape[1], dtype=F64)
    for t in range(T):
        u = k[t] / torch.sqrt((k[t] * k[t]).sum() + 1e-6)
        S = decay[t][:, None] * S - torch.outer(rate[t] * u, u @ S) + torch.outer(k[t], v[t])
        out[t] = r[t] @ S
    return out


def removal_delta(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, n = int(m["heads"]), int(m["dim"])
    r, k, v = ((h @ P[x].T).view(T, H, n) for x in ("r", "k", "v"))
    decay, rate = (x.view(T, H, n) for x in removal_gates(h, P))
    o = torch.stack([removal_recurrence(r[:, i], k[:, i], v[:, i], decay[:, i], rate[:, i]) for i in range(H)], dim=1)
    o = rms_norm(o, None, eps).reshape(T, H * n) * P["norm"]
    return (o * torch.sigmoid(h @ P["g"].T)) @ P["o"].T


def side_by_side(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict, eps: float) -> torch.Tensor:
    left = windowed_attention(h, sub(P, "left."), m["left"], eps)
    right = removal_delta(h, sub(P, "right."), m["right"], eps)
    return 0.5 * (rms_norm(left, P["left.out"], eps) + rms_norm(right, P["right.out"], eps))


# ------------------------------------------------------------------------------------------------ the stack
def dense_ff(h: torch.Tensor, P: Dict[str, torch.Tensor]) -> torch.Tensor:
    return (silu(h @ P["gate"].T) * (h @ P["up"].T)) @ P["down"].T


def sub(tensors: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(F64) for k, v in tensors.items() if k.startswith(prefix)}


def runs(config: Dict) -> List[int]:
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    a, b = int(loop["start"]), int(loop["stop"])
    return list(range(a)) + list(range(a, b)) * int(loop["times"]) + list(range(b, n))


def layer(x: torch.Tensor, L: Dict, P: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    h = rms_norm(x, P["norm1"], eps)
    h = h + causal_filter(h, P["canon1"])
    mixer = {"attention": key_value_attention, "parallel": side_by_side}[L["type"]]
    y = mixer(h, sub(P, "mix."), L["mixer"], eps)
    if L.get("mlp") is not None:
        y = y + dense_ff(rms_norm(x, P["norm2"], eps), sub(P, "mlp."))
    return x + y


def forward(config: Dict, tensors: Dict[str, torch.Tensor], tokens: List[int], layer_outputs: Optional[list] = None
            ) -> torch.Tensor:
    """float64 logits ``[len(tokens), vocab]`` of one sequence; ``layer_outputs`` collects the stream behind every run."""
    eps = float(config["norm"]["eps"])
    embed = tensors["embed"].to(F64)
    x = embed[torch.tensor(tokens, dtype=torch.long)]
    for i in runs(config):
        x = layer(x, config["layers"][i], sub(tensors, f"l{i}."), eps)
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return rms_norm(x, tensors["final.norm"].to(F64), eps) @ embed.T


# ------------------------------------------------------------------------------------------------ random checkpoints
def random_weights(config: Dict, seed: int = 0, dtype=torch.bfloat16, rank: int = 6) -> Dict[str, torch.Tensor]:
    """A checkpoint of the configuration's shapes; values are rounded to ``dtype`` so that both sides read the same.
    ``rank`` is the inner size of the decay's two-step projection (a tensor shape, not a configuration entry)."""
    gen = torch.Generator().manual_seed(seed)
    W, taps = int(config["width"]), int(config["canon"]["taps"])

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=gen) * std + mean).to(dtype)

    def lin(o, i, gain=1.0):
        return rnd(o, i, std=gain / math.sqrt(i))

    t: Dict[str, torch.Tensor] = {"embed": rnd(int(config["vocab"]), W), "final.norm": rnd(W, std=0.2, mean=1.0)}
    for i, L in enumerate(config["layers"]):
        p, m = f"l{i}.", L["mixer"]
        t[p + "norm1"], t[p + "canon1"] = rnd(W, std=0.2, mean=1.0), rnd(W, taps, std=0.4)
        if L["type"] == "attention":
            H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
            x = p + "mix."
            t[x + "q"], t[x + "k"], t[x + "o"] = lin(H * d, W), lin(G * d, W), lin(W, H * d)
            t[x + "temp"], t[x + "g"] = rnd(H, std=0.4, mean=1.0), lin(H, W, 2.0)
        else:
            a, b = m["left"], m["right"]
            H, G, d, dv = int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"])
            x = p + "mix.left."
            t[x + "q"], t[x + "k"], t[x + "v"] = lin(H * d, W), lin(G * d, W), lin(G * dv, W)
            t[x + "q.norm"], t[x + "k.norm"] = rnd(H * d, std=0.3, mean=1.0), rnd(G * d, std=0.3, mean=1.0)
            t[x + "o"], t[x + "out"] = lin(W, H * dv), rnd(W, std=0.3, mean=1.0)
            H, n = int(b["heads"]), int(b["dim"])
            x = p + "mix.right."
            for name in ("r", "k", "v", "g", "a"):
                t[x + name] = lin(H * n, W)
            t[x + "a.b"], t[x + "w0"] = rnd(H * n), rnd(H * n, std=1.5, mean=-1.0)
            t[x + "w1"], t[x + "w2"] = lin(rank, W), lin(H * n, rank)
            t[x + "norm"], t[x + "o"], t[x + "out"] = rnd(H * n, std=0.3, mean=1.0), lin(W, H * n), rnd(W, std=0.3, mean=1.0)
        if L.get("mlp") is not None:
            ff = int(L["mlp"]["ff"])
            t[p + "norm2"] = rnd(W, std=0.2, mean=1.0)
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = lin(ff, W), lin(ff, W), lin(W, ff)
    return t
