"""A plain, slow restatement of the Mozetar architecture in float64 PyTorch on the CPU: one function per mechanism, every
request by itself and from its first token.  It shares no code with the engine; the tests compare the engine with it.

Notation: ``h`` a sublayer's input rows, ``p`` / ``i`` / ``j`` positions counted from 0 in a request, ``X`` the streams
``[tokens, streams, width]``.
"""

from __future__ import annotations

import math

import torch

DT = torch.float64


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * weight


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def causal_conv(u: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """``y_t = sum_j weight[:, j] * u_(t - taps + 1 + j)`` per channel, zeros before the first token."""
    tokens, taps = u.shape[0], weight.shape[1]
    y = torch.zeros_like(u)
    for t in range(tokens):
        for j in range(taps):
            source = t - taps + 1 + j
            if source >= 0:
                y[t] = y[t] + weight[:, j] * u[source]
    return y


def frequencies(rot: dict) -> torch.Tensor:
    """One angle per position and pair: ``base ** (-2i / dims)``; with ``scaling`` slow pairs are slowed down further."""
    dims = rot["dims"]
    result = []
    for i in range(dims // 2):
        f = float(rot["base"]) ** (-2.0 * i / dims)
        scaling = rot.get("scaling")
        if scaling:
            length = 2.0 * math.pi / f
            if length > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif length >= scaling["original"] / scaling["high"]:
                s = (scaling["original"] / length - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        result.append(f)
    return torch.tensor(result, dtype=DT)


def rotate_neighbours(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """``x`` [tokens, heads, channels]: channels ``2i`` and ``2i + 1`` of the first ``dims`` turn as a pair."""
    dims = rot["dims"]
    out = x.clone()
    f = frequencies(rot)
    for i in range(dims // 2):
        angle = positions.to(DT) * f[i]
        cos, sin = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * cos - v * sin
        out[..., 2 * i + 1] = v * cos + u * sin
    return out


def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: int | None) -> torch.Tensor:
    """q [tokens, heads, dk], k [tokens, groups, dk], v [tokens, groups, dv]; position i sees itself and what lies before it
    (under a window: up to ``window - 1`` positions back)."""
    tokens, heads, groups = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(tokens, heads, v.shape[2], dtype=DT)
    for i in range(tokens):
        first = 0 if window is None else max(0, i - window + 1)
        for head in range(heads):
            g = head // (heads // groups)
            weight = torch.softmax((k[first : i + 1, g] @ q[i, head]) * scale, dim=0)
            out[i, head] = weight @ v[first : i + 1, g]
    return out


def query_temperature(positions: torch.Tensor, q_temp: dict | None) -> torch.Tensor:
    if not q_temp:
        return torch.ones_like(positions, dtype=DT)
    return torch.tensor([1.0 + q_temp["coef"] * math.log(math.floor((int(p) + 1) / q_temp["every"]) + 1.0) for p in positions], dtype=DT)


def differential_lambda(w: dict, diff: float) -> float:
    return math.exp(float((w["lq1"] * w["lk1"]).sum())) - math.exp(float((w["lq2"] * w["lk2"]).sum())) + diff


def combine_maps(a1: torch.Tensor, a2: torch.Tensor, lam: float, diff: float, gate: torch.Tensor, eps: float) -> torch.Tensor:
    """The two maps' outputs [tokens, heads, dv] as one: ``a1 - lam a2``, each head at unit root mean square, times
    ``1 - diff`` and the head's gate."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff) * torch.sigmoid(gate)[:, :, None]


def differential_attention(h: torch.Tensor, w: dict, cfg: dict, eps: float) -> torch.Tensor:
    heads, groups, dk, dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    tokens = h.shape[0]
    temperature = query_temperature(torch.arange(tokens), cfg.get("q_temp"))
    q = (h @ w["q"].T).reshape(tokens, heads, 2, dk) * temperature[:, None, None, None]
    k = (h @ w["k"].T).reshape(tokens, groups, 2, dk)
    v = (h @ w["v"].T).reshape(tokens, groups, dv)
    maps = [softmax_attention(q[:, :, m], k[:, :, m], v, cfg["scale"], None) for m in (0, 1)]
    o = combine_maps(maps[0], maps[1], differential_lambda(w, cfg["diff"]), cfg["diff"], h @ w["g"].T, eps)
    return o.reshape(tokens, heads * dv) @ w["o"].T


def convolved_attention(h: torch.Tensor, w: dict, cfg: dict, shared: dict, index: int) -> torch.Tensor:
    """Window attention on convolved projections; ``shared`` keeps every layer's keys and values for those that borrow them."""
    heads, groups, dk, dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    tokens = h.shape[0]
    positions = torch.arange(tokens)
    q = rotate_neighbours(causal_conv(h @ w["q"].T, w["q.conv"]).reshape(tokens, heads, dk), positions, cfg["rot"])
    if cfg.get("kv_from") is None:
        k = rotate_neighbours(causal_conv(h @ w["k"].T, w["k.conv"]).reshape(tokens, groups, dk), positions, cfg["rot"])
        v = causal_conv(h @ w["v"].T, w["v.conv"]).reshape(tokens, groups, dv)
        shared[index] = (k, v)
    else:
        k, v = shared[cfg["kv_from"]]
    return softmax_attention(q, k, v, cfg["scale"], cfg["mask"]["size"]).reshape(tokens, heads * dv) @ w["o"].T


def forget_recurrence(q: torch.Tensor, f: torch.Tensor, v: torch.Tensor, state: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """A state ``S[i, j]`` per head becomes ``f[i] S[i, j] + (1 - f[i]) v[j]`` at every token and is read as ``sum_i q[i] S[i, j]``; returns the read-outs and the last state."""
    tokens, heads, dk = q.shape
    state = torch.zeros(heads, dk, v.shape[-1], dtype=DT) if state is None else state.clone()
    out = torch.zeros(tokens, heads, v.shape[-1], dtype=DT)
    for t in range(tokens):
        state = f[t][:, :, None] * state + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", state, q[t])
    return out, state


def forget_gate(z: torch.Tensor, lower: torch.Tensor) -> torch.Tensor:
    return lower + (1.0 - lower) * torch.sigmoid(z)


def hgrn2(h: torch.Tensor, w: dict, cfg: dict, eps: float) -> torch.Tensor:
    heads, dk, dv = cfg["heads"], cfg["dim"], cfg["vdim"]
    tokens = h.shape[0]
    q = silu(h @ w["q"].T).reshape(tokens, heads, dk)
    f = forget_gate(h @ w["f"].T + w["f.b"], w["lower"]).reshape(tokens, heads, dk)
    v = (h @ w["v"].T).reshape(tokens, heads, dv)
    o, _ = forget_recurrence(q, f, v)
    return rms_norm(o, w["norm"], eps).reshape(tokens, heads * dv) @ w["o"].T


def poly_norm(z: torch.Tensor, act: torch.Tensor, eps: float) -> torch.Tensor:
    return act[0] * rms(z, eps) + act[1] * rms(z * z, eps) + act[2] * rms(z * z * z, eps) + act[3]


def dense(h: torch.Tensor, w: dict, eps: float) -> torch.Tensor:
    return poly_norm(h @ w["up"].T + w["up.b"], w["act"], eps) @ w["down"].T + w["down.b"]


def choose_experts(scores: torch.Tensor, router: dict) -> list[int]:
    """The experts of one token (``scores`` [experts]): the largest scores inside the groups with the largest best score."""
    experts, top = router["experts"], router["top"]
    groups = router.get("groups") or {"count": 1, "keep": 1}
    size = experts // groups["count"]
    best = [max(float(scores[g * size + m]) for m in range(size)) for g in range(groups["count"])]
    kept = sorted(range(groups["count"]), key=lambda g: (-best[g], g))[: groups["keep"]]
    open_to = [e for e in range(experts) if e // size in kept]
    return sorted(open_to, key=lambda e: (-float(scores[e]), e))[:top]


def routed_experts(h: torch.Tensor, w: dict, cfg: dict, choice: torch.Tensor | None = None, slack: list | None = None) -> torch.Tensor:
    """``choice`` ([tokens, top], optional): the experts to use instead of the ones this function would choose (for a comparison with
    an implementation whose rounding may turn a close call); ``slack`` then receives, per token, by how much the chosen experts'
    worst score lies below what this function's own choice has at worst (zero where the choices agree), or the kept groups' best
    scores likewise."""
    out = torch.zeros_like(h)
    scores = torch.softmax(h @ w["router"].T, dim=-1)
    groups = cfg["router"].get("groups") or {"count": 1, "keep": 1}
    size = cfg["router"]["experts"] // groups["count"]
    for t in range(h.shape[0]):
        own = order = choose_experts(scores[t], cfg["router"])
        if choice is not None:
            order = [int(e) for e in choice[t]]
            if slack is not None and sorted(order) != sorted(own):
                best = lambda e: float(scores[t, e // size * size : e // size * size + size].max())
                differing = max(float(scores[t, e]) for e in own if e not in order) - min(float(scores[t, e]) for e in order if e not in own)
                group_gap = max(best(e) for e in own) - min(best(e) for e in order)
                slack.append(min(abs(differing), abs(group_gap)) if {e // size for e in own} != {e // size for e in order} else differing)
        weights = scores[t, order] / (scores[t, order].sum() + 1e-20)
        for weight, e in zip(weights, order):
            hidden = silu(h[t] @ w[f"e{e}.gate"].T) * (h[t] @ w[f"e{e}.up"].T)
            out[t] += weight * (hidden @ w[f"e{e}.down"].T)
    return out


def read_streams(X: torch.Tensor, w_in: torch.Tensor) -> torch.Tensor:
    return torch.einsum("s,tsd->td", w_in, X)


def write_streams(X: torch.Tensor, mix: torch.Tensor, w_out: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """``X_to <- sum_from mix[from, to] X_from + out[to] y``."""
    return torch.einsum("fu,tfd->tud", mix, X) + w_out[None, :, None] * y[:, None, :]


def sub(weights: dict, prefix: str) -> dict:
    return {name[len(prefix):]: tensor for name, tensor in weights.items() if name.startswith(prefix)}


def forward(config: dict, weights: dict, tokens: list[int], layers_out: list | None = None, choices: dict | None = None,
            slack: list | None = None) -> torch.Tensor:
    """Logits ``[tokens, vocab]`` of one request read whole; ``weights`` by checkpoint name, in float64.
    ``layers_out`` (a list) receives the sum of the streams after every layer.  ``choices`` (layer -> [tokens, top]) and ``slack``: see
    :func:`routed_experts`."""
    eps = config["norm"]["eps"]
    x = weights["embed"][torch.tensor(tokens, dtype=torch.long)]
    X = x[:, None, :].repeat(1, config["streams"], 1)
    shared: dict = {}
    for index, layer in enumerate(config["layers"]):
        w = sub(weights, f"l{index}.")
        h = rms_norm(read_streams(X, w["hc1.in"]), w["norm1"], eps)
        h = h + causal_conv(h, w["canon1"])
        mix = sub(w, "mix.")
        if layer["type"] == "attention":
            y = differential_attention(h, mix, layer["mixer"], eps)
        elif layer["type"] == "attention_2":
            y = convolved_attention(h, mix, layer["mixer"], shared, index)
        elif layer["type"] == "hgrn2":
            y = hgrn2(h, mix, layer["mixer"], eps)
        else:
            raise ValueError(layer["type"])
        X = write_streams(X, w["hc1.mix"], w["hc1.out"], y)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rms_norm(read_streams(X, w["hc2.in"]), w["norm2"], eps)
            if mlp["kind"] == "dense":
                y = dense(h, sub(w, "mlp."), eps)
            else:
                y = routed_experts(h, sub(w, "mlp."), mlp, None if choices is None else choices.get(index), slack)
            X = write_streams(X, w["hc2.mix"], w["hc2.out"], y)
        if layers_out is not None:
            layers_out.append(X.sum(dim=1))
    return rms_norm(X.sum(dim=1), weights["final.norm"], eps) @ weights["head"].T
