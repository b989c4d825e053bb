"""A plain, slow restatement of the Zevetar architecture in float64 PyTorch on the CPU: one function per mechanism, every request by
itself, every position from the whole prefix.  It shares no code with the engine; the tests compare the engine with it.

Notation: ``h`` a token's normed input row, ``t`` / ``i`` / ``j`` positions counted from 0 in a request.
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


def pair_frequencies(rot: dict) -> tuple[torch.Tensor, float]:
    """``([dims / 2] frequencies, factor on sines and cosines)``: ``base ** (-2m / dims)``, stretched where ``rot`` says so."""
    dims, base = rot["dims"], rot["base"]
    plain = [base ** (-2.0 * m / dims) for m in range(dims // 2)]
    scaling = rot.get("scaling")
    if scaling is None:
        return torch.tensor(plain, dtype=DT), 1.0

    def index_of(turns: float) -> float:
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    low = max(math.floor(index_of(scaling["fast"])), 0)
    high = min(math.ceil(index_of(scaling["slow"])), dims - 1)
    stretched = []
    for m, f in enumerate(plain):
        share = min(max((m - low) / max(high - low, 0.001), 0.0), 1.0)
        stretched.append(f / scaling["factor"] * share + f * (1.0 - share))
    return torch.tensor(stretched, dtype=DT), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_neighbours(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """``x`` [tokens, ..., channels]: channels ``2m`` and ``2m + 1`` of the first ``rot.dims`` are a pair."""
    frequency, factor = pair_frequencies(rot)
    dims = rot["dims"]
    angle = positions.to(DT)[:, None] * frequency[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (dims // 2,)
    cos, sin = (torch.cos(angle) * factor).reshape(shape), (torch.sin(angle) * factor).reshape(shape)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """``x`` [tokens, heads, channels]: channel ``m`` of the first ``rot.dims`` is paired with ``m + dims / 2``."""
    frequency, factor = pair_frequencies(rot)
    half = rot["dims"] // 2
    angle = positions.to(DT)[:, None] * frequency[None, :]
    cos, sin = (torch.cos(angle) * factor)[:, None, :], (torch.sin(angle) * factor)[:, None, :]
    u, v = x[..., :half], x[..., half : 2 * half]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., 2 * half :]], dim=-1)


def latent_rows(h: torch.Tensor, w: dict, cfg: dict, eps: float) -> tuple[torch.Tensor, torch.Tensor]:
    """What a token leaves behind: its normed latent and its rotated key part, ``([tokens, kv_rank], [tokens, rot_dim])``."""
    down = h @ w["dkv"].T
    rank = cfg["kv_rank"]
    return rms_norm(down[:, :rank], w["dkv.norm"], eps), rotate_neighbours(down[:, rank:], torch.arange(h.shape[0]), cfg["rot"])


def latent_attention(h: torch.Tensor, w: dict, cfg: dict, eps: float, rows: tuple[torch.Tensor, torch.Tensor]) -> torch.Tensor:
    """``rows``: the latents and rotated key parts to look at (this layer's own, or another's)."""
    heads, dim, rot_dim, vdim = cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"]
    tokens = h.shape[0]
    positions = torch.arange(tokens)
    latent, key_rot = rows
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).reshape(tokens, heads, dim + rot_dim)
    q_plain, q_rot = q[..., :dim], rotate_neighbours(q[..., dim:], positions, cfg["rot"])
    keys = (latent @ w["uk"].T).reshape(tokens, heads, dim)
    values = (latent @ w["uv"].T).reshape(tokens, heads, vdim)
    size = (cfg.get("mask") or {}).get("size")
    out = torch.zeros(tokens, heads, vdim, dtype=DT)
    for i in range(tokens):
        first = 0 if size is None else max(0, i - size + 1)
        seen = slice(first, i + 1)
        for head in range(heads):
            score = (keys[seen, head] @ q_plain[i, head] + key_rot[seen] @ q_rot[i, head]) * cfg["scale"]
            out[i, head] = torch.softmax(score, dim=0) @ values[seen, head]
    gated = out.reshape(tokens, heads * vdim) * torch.sigmoid(h @ w["g"].T)
    return gated @ w["o"].T


def retention(h: torch.Tensor, w: dict, cfg: dict, eps: float) -> torch.Tensor:
    heads, dk, dv = cfg["heads"], cfg["dim"], cfg["vdim"]
    tokens = h.shape[0]
    positions = torch.arange(tokens)
    q = (h @ w["q"].T).reshape(tokens, heads, dk)
    k = (h @ w["k"].T).reshape(tokens, heads, dk)
    v = (h @ w["v"].T).reshape(tokens, heads, dv)
    if cfg.get("rot") is not None and cfg["rot"]["dims"]:
        q, k = rotate_halves(q, positions, cfg["rot"]), rotate_halves(k, positions, cfg["rot"])
    k = k * dk ** -0.5
    decay = torch.tensor(cfg["decay"], dtype=DT)[:, None, None]
    state = torch.zeros(heads, dk, dv, dtype=DT)
    out = torch.zeros(tokens, heads, dv, dtype=DT)
    for t in range(tokens):
        state = decay * state + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hkv,hk->hv", state, q[t])
    return (rms(out, eps).reshape(tokens, heads * dv) * silu(h @ w["g"].T)) @ w["o"].T


def gated(h: torch.Tensor, w: dict, prefix: str = "") -> torch.Tensor:
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def routed_experts(h: torch.Tensor, w: dict, cfg: dict, choice: torch.Tensor | None = None, slack: list | None = None) -> torch.Tensor:
    """Every chosen expert runs on its score times the token's row.  ``choice`` ([tokens, top], optional): the experts to use instead of
    the ones this function would choose (for a comparison with an implementation whose rounding may turn a close call); ``slack`` then
    receives, per token, by how much the best expert left out beats the worst one taken."""
    experts, top = cfg["router"]["experts"], cfg["router"]["top"]
    scores = torch.sigmoid(h @ w["router"].T)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(experts), key=lambda e: (-float(scores[t, e]), e))[:top]
        if choice is not None:
            order = [int(e) for e in choice[t]]
            others = [float(scores[t, e]) for e in range(experts) if e not in order]
            if slack is not None and others:
                slack.append(max(others) - min(float(scores[t, e]) for e in order))
        for e in order:
            out[t] += gated(scores[t, e] * h[t], w, f"e{e}.")
    if cfg.get("shared") is not None:
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * gated(h, w, "shared.")
    return out


def sub(weights: dict, prefix: str) -> dict:
    return {name[len(prefix):]: tensor for name, tensor in weights.items() if name.startswith(prefix)}


def forward(config: dict, weights: dict, tokens: list[int], layers_out: list | None = None, choices: dict | None = None,
            slack: list | None = None) -> torch.Tensor:
    """Logits ``[tokens, vocab]`` of one request read whole; ``weights`` by checkpoint name, in float64.
    ``layers_out`` (a list) receives the stream after every layer.  ``choices`` (layer -> [tokens, top]) and ``slack``: see
    :func:`routed_experts`."""
    eps = config["norm"]["eps"]
    x = weights["embed"][torch.tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    rows: dict[int, tuple[torch.Tensor, torch.Tensor]] = {}
    for index, layer in enumerate(config["layers"]):
        w = sub(weights, f"l{index}.")
        mix, cfg, mlp = sub(w, "mix."), layer["mixer"], layer.get("mlp")
        h = rms_norm(x, w["norm1"], eps)
        if layer["type"] == "retention":
            y = retention(h, mix, cfg, eps) * w["ls1"]
        elif layer["type"] == "latent_attention":
            if cfg.get("kv_from") is None:
                rows[index] = latent_rows(h, mix, cfg, eps)
                y = latent_attention(h, mix, cfg, eps, rows[index]) * w["ls1"]
            else:
                y = latent_attention(h, mix, cfg, eps, rows[cfg["kv_from"]]) * w["ls1"]
        else:
            raise ValueError(layer["type"])
        if mlp is not None:
            ff = sub(w, "mlp.")
            if mlp["kind"] == "dense":
                y = y + gated(h, ff) * w["ls2"]
            else:
                y = y + routed_experts(h, ff, mlp, None if choices is None else choices[index], slack) * w["ls2"]
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    logits = rms_norm(x, weights["final.norm"], eps) @ weights["embed"].T * config.get("logit_scale", 1.0)
    cap = config.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits
