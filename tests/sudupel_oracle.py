"""Plain float64 evaluation of a Sudupel stack, one function per mechanism, whole sequences at a time and nothing cached.
It shares no code with the package: the tests compare the engine (paged cache, carried state, ragged batches, kernels)
with it.

``config`` is the model's ``config.json`` object and ``tensors`` maps checkpoint names to arrays (any float dtype).

The stack: ``x = embed[token] * s``; a layer is ``x += n1b(mixer(n1 x))``, ``x += n2b(ff(n2 x))`` with norms ``n(x) = x / rms(x)
* (1 + w)``; final norm, head, soft cap.  Mixers: lightning attention (a matrix state per head that decays at one fixed rate), and two
pairs of mixers side by side whose outputs are added with one factor each: softmax attention with a unit sink beside a gated linear
recurrent unit, and filtered windowed attention beside gated linear attention.  Feed-forwards: clamped gated, and experts chosen
inside the best groups.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def sub(tensors: Dict[str, torch.Tensor], prefix: str) -> Dict[str, torch.Tensor]:
    return {k[len(prefix):]: v.to(F64) for k, v in tensors.items() if k.startswith(prefix)}


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_filter(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``u`` [T, C], ``w`` [C, taps]: ``y[t] = sum_j w[:, j] * u[t - taps + 1 + j]`` with zeros before the start."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j] * u[: T - back]
    return y


# ------------------------------------------------------------------------------------------------ rotation
def rotary_frequencies(rot: Dict) -> List[float]:
    """Angular frequency of every pair.  With ``scaling``: the pair that makes ``t`` turns over the original context has the index
    ``dims ln(original / (2 pi t)) / (2 ln base)``; pairs below that of ``fast`` turns keep their frequency, pairs above that of
    ``slow`` turns are slowed by ``factor``, a linear ramp lies between."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f

    def pair(turns):
        return dims * math.log(float(sc["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(pair(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair(float(sc["slow"]))), dims - 1)
    out = []
    for i, v in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / float(sc["factor"]) * ramp + v * (1.0 - ramp))
    return out


def rotary_amplitude(rot: Dict) -> float:
    return 0.1 * math.log(float(rot["scaling"]["factor"])) + 1.0 if rot.get("scaling") else 1.0


def rotate(x: torch.Tensor, rot: Dict) -> torch.Tensor:
    """``x`` [T, heads, n]: channels ``i`` and ``i + dims/2`` turn together; the channels behind ``dims`` pass."""
    half = int(rot["dims"]) // 2
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * torch.tensor(rotary_frequencies(rot), dtype=F64)[None, :]
    amp = rotary_amplitude(rot)
    c, s = (torch.cos(ang) * amp)[:, None, :], (torch.sin(ang) * amp)[:, None, :]
    u, v = x[..., :half], x[..., half: 2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


# ------------------------------------------------------------------------------------------------ attention
def attend(q, k, v, scale: float, window: int, unit_sink: bool) -> torch.Tensor:
    """``q`` [T, H, d], ``k`` [T, G, d], ``v`` [T, G, dv] -> [T, H, dv]; ``window`` 0 sees every earlier position; ``unit_sink``
    adds one to the denominator of the (unshifted) exponentials."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    i = torch.arange(T)
    dist = i[:, None] - i[None, :]
    visible = dist >= 0
    if window > 0:
        visible &= dist < window
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T * scale).masked_fill(~visible, float("-inf"))
        top = s.max(dim=-1, keepdim=True).values
        if unit_sink:
            top = top.clamp(min=0.0)
        e = torch.exp(s - top)
        den = e.sum(dim=-1, keepdim=True)
        if unit_sink:
            den = den + torch.exp(-top)
        out[:, h] = e / den @ v[:, g]
    return out


def sink_attention(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict, eps: float) -> torch.Tensor:
    """Query and key rows are normalised over all heads at once, then rotated; every earlier position is visible."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms_norm(h @ P["q"].T, P["q.norm"], eps).view(T, H, d)
    k = rms_norm(h @ P["k"].T, P["k.norm"], eps).view(T, G, d)
    v = (h @ P["v"].T).view(T, G, dv)
    o = attend(rotate(q, m["rot"]), rotate(k, m["rot"]), v, float(m["scale"]), 0, True)
    return o.reshape(T, H * dv) @ P["o"].T


def filtered_window_attention(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict, eps: float) -> torch.Tensor:
    """q, k and v pass a short causal filter; q and k heads are normalised one by one, then rotated; sliding window."""
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (causal_filter(h @ P[n].T, P[n + ".conv"]) for n in ("q", "k", "v"))
    q = rms_norm(q.view(T, H, d), P["q.norm"], eps)
    k = rms_norm(k.view(T, G, d), P["k.norm"], eps)
    o = attend(rotate(q, m["rot"]), rotate(k, m["rot"]), v.view(T, G, dv), float(m["scale"]), int(m["mask"]["size"]), False)
    return o.reshape(T, H * dv) @ P["o"].T


# ------------------------------------------------------------------------------------------------ recurrences
def decayed_outer_products(q, k, v, decay, state: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One head: ``q``, ``k`` [T, n], ``v`` [T, dv], ``decay`` [T, n] (one factor per key channel): ``S <- diag(decay) S + k v^T``,
    ``o = S^T q``."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=F64) if state is None else state
    out = []
    for t in range(k.shape[0]):
        S = decay[t][:, None] * S + torch.outer(k[t], v[t])
        out.append(q[t] @ S)
    return torch.stack(out)


def lightning(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, n, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = silu(h @ P["q"].T).view(T, H, n), silu(h @ P["k"].T).view(T, H, n), silu(h @ P["v"].T).view(T, H, dv)
    o = torch.stack([decayed_outer_products(q[:, i], k[:, i], v[:, i], torch.full((T, n), float(m["decay"][i]), dtype=F64))
                     for i in range(H)], dim=1).reshape(T, H * dv)
    return (rms_norm(o, P["norm"], eps) * torch.sigmoid(h @ P["g"].T)) @ P["o"].T


def gated_linear_attention(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, n, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (h @ P["q"].T * n ** -0.5).view(T, H, n), (h @ P["k"].T).view(T, H, n), (h @ P["v"].T).view(T, H, dv)
    z = (h @ P["a1"].T) @ P["a2"].T + P["a2.b"]
    alpha = (torch.sigmoid(z) ** (1.0 / float(m["tau"]))).view(T, H, n)
    o = torch.stack([decayed_outer_products(q[:, i], k[:, i], v[:, i], alpha[:, i]) for i in range(H)], dim=1)
    o = rms_norm(o, P["norm"], eps).reshape(T, H * dv)
    return (o * silu(h @ P["g"].T)) @ P["o"].T


def lru_gates(u: torch.Tensor, P: Dict[str, torch.Tensor]):
    """(log a, input gate) of the recurrent unit from its filtered input ``u`` [T, width], block by block."""
    blocks, size = P["ra"].shape[0], P["ra"].shape[1]
    r, i = torch.zeros_like(u), torch.zeros_like(u)
    for b in range(blocks):
        part = u[:, b * size: (b + 1) * size]
        r[:, b * size: (b + 1) * size] = torch.sigmoid(part @ P["ra"][b].T + P["ra.b"][b])
        i[:, b * size: (b + 1) * size] = torch.sigmoid(part @ P["ri"][b].T + P["ri.b"][b])
    return -8.0 * r * torch.log1p(torch.exp(P["lam"])), i


def lru_scan(log_a: torch.Tensor, gated: torch.Tensor, state: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``s <- a s + sqrt(1 - a^2) * gated`` per channel."""
    s = torch.zeros(gated.shape[1], dtype=F64) if state is None else state
    out = []
    for t in range(gated.shape[0]):
        s = torch.exp(log_a[t]) * s + torch.sqrt(-torch.expm1(2.0 * log_a[t])) * gated[t]
        out.append(s)
    return torch.stack(out)


def recurrent_block(h: torch.Tensor, P: Dict[str, torch.Tensor], m: Dict) -> torch.Tensor:
    y = gelu_tanh(h @ P["y"].T + P["y.b"])
    u = causal_filter(h @ P["x"].T + P["x.b"], P["conv"]) + P["conv.b"]
    log_a, i = lru_gates(u, P)
    return (lru_scan(log_a, i * u) * y) @ P["o"].T


def parallel(h, P, m, eps):
    return (float(m["left_scale"]) * sink_attention(h, sub(P, "left."), m["left"], eps)
            + float(m["right_scale"]) * recurrent_block(h, sub(P, "right."), m["right"]))


def parallel_2(h, P, m, eps):
    return (float(m["left_scale"]) * filtered_window_attention(h, sub(P, "left."), m["left"], eps)
            + float(m["right_scale"]) * gated_linear_attention(h, sub(P, "right."), m["right"], eps))


# ------------------------------------------------------------------------------------------------ feed-forwards
def dense_ff(h: torch.Tensor, P: Dict[str, torch.Tensor], mlp: Dict) -> torch.Tensor:
    limit = float(mlp["limit"])
    g = (h @ P["gate"].T).clamp(max=limit)
    u = (h @ P["up"].T).clamp(min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ P["down"].T


def choose_experts(scores: torch.Tensor, correction: torch.Tensor, groups: int, keep: int, top: int) -> List[int]:
    """One token: the ``top`` largest ``score + correction`` in the ``keep`` groups whose two largest such sums are largest."""
    choice = (scores + correction).tolist()
    size = len(choice) // groups
    rank = [sum(sorted(choice[g * size: (g + 1) * size], reverse=True)[:2]) for g in range(groups)]
    best = sorted(range(groups), key=lambda g: -rank[g])[:keep]
    open_ = [e for e in range(len(choice)) if e // size in best]
    return sorted(open_, key=lambda e: -choice[e])[:top]


def expert_ff(h: torch.Tensor, P: Dict[str, torch.Tensor], mlp: Dict) -> torch.Tensor:
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    s = torch.sigmoid(h @ P["router"].T)
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in choose_experts(s[t], P["correction"], int(groups["count"]), int(groups["keep"]), int(r["top"])):
            p = f"e{e}."
            y[t] += s[t, e] * (P[p + "down"] @ (silu(P[p + "gate"] @ h[t]) * (P[p + "up"] @ h[t])))
    return y


# ------------------------------------------------------------------------------------------------ the stack
def layer(x: torch.Tensor, L: Dict, P: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    mixer = {"lightning": lightning, "parallel": parallel, "parallel_2": parallel_2}[L["type"]]
    y = mixer(rms_norm(x, 1.0 + P["norm1"], eps), sub(P, "mix."), L["mixer"], eps)
    x = x + rms_norm(y, 1.0 + P["norm1b"], eps)
    if L.get("mlp") is not None:
        ff = {"dense": dense_ff, "moe": expert_ff}[L["mlp"]["kind"]]
        y = ff(rms_norm(x, 1.0 + P["norm2"], eps), sub(P, "mlp."), L["mlp"])
        x = x + rms_norm(y, 1.0 + P["norm2b"], eps)
    return x


def forward(config: Dict, tensors: Dict[str, torch.Tensor], tokens: List[int], layer_outputs: Optional[list] = None
            ) -> torch.Tensor:
    """float64 logits ``[len(tokens), vocab]`` of one sequence; ``layer_outputs`` collects the stream behind every layer."""
    eps = float(config["norm"]["eps"])
    x = tensors["embed"].to(F64)[torch.tensor(tokens, dtype=torch.long)] * float(config["embedding"]["scale"])
    for i, L in enumerate(config["layers"]):
        x = layer(x, L, sub(tensors, f"l{i}."), eps)
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    logits = rms_norm(x, 1.0 + tensors["final.norm"].to(F64), eps) @ tensors["head"].to(F64).T
    cap = float(config["logit_softcap"])
    return cap * torch.tanh(logits / cap)


# ------------------------------------------------------------------------------------------------ random checkpoints
def random_weights(config: Dict, seed: int = 0, dtype=torch.bfloat16, rank: int = 6) -> Dict[str, torch.Tensor]:
    """A checkpoint of the configuration's shapes; values are rounded to ``dtype`` so that both sides read the same.
    ``rank`` is the inner size of the decay's two-step projection (a tensor shape, not a configuration entry)."""
    gen = torch.Generator().manual_seed(seed)
    W, V = int(config["width"]), int(config["vocab"])

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=gen) * std + mean).to(dtype)

    def lin(o, i, gain=1.0):
        return rnd(o, i, std=gain / math.sqrt(i))

    t: Dict[str, torch.Tensor] = {"embed": rnd(V, W, std=0.1), "final.norm": rnd(W, std=0.2), "head": lin(V, W, 2.0)}
    for i, L in enumerate(config["layers"]):
        p, m = f"l{i}.", L["mixer"]
        t[p + "norm1"], t[p + "norm1b"] = rnd(W, std=0.2), rnd(W, std=0.2)
        x = p + "mix."
        if L["type"] == "lightning":
            H, n, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
            t[x + "q"], t[x + "k"], t[x + "v"], t[x + "g"] = lin(H * n, W), lin(H * n, W), lin(H * dv, W), lin(H * dv, W)
            t[x + "norm"], t[x + "o"] = rnd(H * dv, std=0.3, mean=1.0), lin(W, H * dv)
        else:
            a, b = m["left"], m["right"]
            H, G, d, dv = int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"])
            y = x + "left."
            t[y + "q"], t[y + "k"], t[y + "v"], t[y + "o"] = lin(H * d, W), lin(G * d, W), lin(G * dv, W), lin(W, H * dv)
            nq, nk = (H * d, G * d) if L["type"] == "parallel" else (d, d)
            t[y + "q.norm"], t[y + "k.norm"] = rnd(nq, std=0.3, mean=1.0), rnd(nk, std=0.3, mean=1.0)
            if L["type"] == "parallel_2":
                taps = int(a["conv"])
                for name, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                    t[y + name + ".conv"] = rnd(rows, taps, std=0.6)
            y = x + "right."
            if L["type"] == "parallel":
                N, B, taps = int(b["width"]), int(b["blocks"]), int(b["conv"])
                S = N // B
                t[y + "y"], t[y + "x"], t[y + "o"] = lin(N, W), lin(N, W), lin(W, N)
                t[y + "y.b"], t[y + "x.b"], t[y + "conv.b"] = rnd(N, std=0.5), rnd(N, std=0.5), rnd(N, std=0.5)
                t[y + "conv"] = rnd(N, taps, std=0.6)
                for g in ("ra", "ri"):
                    t[y + g], t[y + g + ".b"] = rnd(B, S, S, std=1.0 / math.sqrt(S)), rnd(B, S)
                t[y + "lam"] = rnd(N, std=1.5, mean=-4.0)
            else:
                H, n, dv = int(b["heads"]), int(b["dim"]), int(b["vdim"])
                t[y + "q"], t[y + "k"], t[y + "v"], t[y + "g"] = lin(H * n, W), lin(H * n, W), lin(H * dv, W), lin(H * dv, W)
                t[y + "a1"], t[y + "a2"], t[y + "a2.b"] = lin(rank, W), lin(H * n, rank, 2.0), rnd(H * n, std=1.5)
                t[y + "norm"], t[y + "o"] = rnd(dv, std=0.3, mean=1.0), lin(W, H * dv)
        mlp = L.get("mlp")
        if mlp is not None:
            t[p + "norm2"], t[p + "norm2b"] = rnd(W, std=0.2), rnd(W, std=0.2)
            x = p + "mlp."
            if mlp["kind"] == "dense":
                ff = int(mlp["ff"])
                t[x + "gate"], t[x + "up"], t[x + "down"] = lin(ff, W), lin(ff, W), lin(W, ff)
            else:
                E, ff = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"])
                t[x + "router"], t[x + "correction"] = lin(E, W), rnd(E, std=0.3)
                for e in range(E):
                    y = f"{x}e{e}."
                    t[y + "gate"], t[y + "up"], t[y + "down"] = lin(ff, W), lin(ff, W), lin(W, ff)
    return t
