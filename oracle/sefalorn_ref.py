"""Plain restatement of the Sefalorn layer-list design on the CPU: test infrastructure only.

One function per mechanism, whole sequences at a time, token by token where the design is a recurrence; no cache, no
batching, no padding.  `dtype` is the working precision of the tensors handed in (float64 unless a caller says otherwise).

  layer   x += sigmoid(R1 h + b1) * mixer(h), h = norm1 x;   x += sigmoid(R2 h + b2) * experts(h), h = norm2 x
  out     logits = logit_scale * head norm(x)
"""
from __future__ import annotations

import torch


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def residual_gate(h: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    return torch.sigmoid(h @ w.T + b)


# ------------------------------------------------------------------ attention


def window_mask(T: int, size: int) -> torch.Tensor:
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    return (j <= i) & (i - j < size)


def distance_penalty(T: int, r1: torch.Tensor, r2: torch.Tensor) -> torch.Tensor:
    """[H, T, T]: r1_h ln(1 + r2_h (i - j)) for j <= i, 0 elsewhere."""
    d = (torch.arange(T)[:, None] - torch.arange(T)[None]).clamp(min=0).to(r1.dtype)
    return r1[:, None, None] * torch.log1p(r2[:, None, None] * d[None])


def talking_scores(q, k, scale: float, r1, r2, talk) -> torch.Tensor:
    """q [T, H, d], k [T, G, d] -> scores [H, T, T]: every head's own score less its distance penalty, then mixed."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    own = torch.stack([(q[:, h] @ k[:, h // per].T) * scale for h in range(H)]) - distance_penalty(T, r1, r2)
    return torch.einsum("hg,gij->hij", talk, own)


def window_attention(h, w: dict, m: dict) -> torch.Tensor:
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T + w["q.b"]).view(T, H, d)
    k = (h @ w["k"].T + w["k.b"]).view(T, G, d)
    v = (h @ w["v"].T + w["v.b"]).view(T, G, dv)
    s = talking_scores(q, k, m["scale"], w["r1"], w["r2"], w["talk"])
    p = torch.softmax(s.masked_fill(~window_mask(T, m["mask"]["size"])[None], float("-inf")), -1)
    o = torch.stack([p[a] @ v[:, a // (H // G)] for a in range(H)], 1)
    return o.reshape(T, H * dv) @ w["o"].T + w["o.b"]


# ---------------------------------------------------------------- recurrences


def causal_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x [T, C], w [C, taps]: sum_j w[:, j] x_{t - taps + 1 + j}, zeros before the start."""
    taps = w.shape[1]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                out[t] += w[:, j] * x[t - taps + 1 + j]
    return out


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, g) -> torch.Tensor:
    """One head: q, k [T, d], v [T, dv], beta, g [T] -> o [T, dv]."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = S * g[t]
        S = S + torch.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out.append(S.T @ q[t])
    return torch.stack(out)


def delta_mixer(h, w: dict, m: dict, eps: float) -> torch.Tensor:
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit(silu(causal_conv(h @ w["q"].T, w["q.conv"])).view(T, G, d)) * d ** -0.5
    k = unit(silu(causal_conv(h @ w["k"].T, w["k.conv"])).view(T, G, d))
    v = silu(causal_conv(h @ w["v"].T, w["v.conv"])).view(T, H, dv)
    beta = torch.sigmoid(h @ w["b"].T)
    g = torch.exp(-torch.exp(w["A_log"]) * torch.nn.functional.softplus(h @ w["a"].T + w["dt_bias"]))
    per = H // G
    o = torch.stack([delta_rule(q[:, a // per], k[:, a // per], v[:, a], beta[:, a], g[:, a]) for a in range(H)], 1)
    o = rms_unit(o, eps) * w["norm"] * silu(h @ w["g"].T).view(T, H, dv)
    return o.reshape(T, H * dv) @ w["o"].T


def decay_attention(q, k, v, decay: float) -> torch.Tensor:
    """One head of lightning attention."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = S * decay + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out)


def lightning_mixer(h, w: dict, m: dict, eps: float) -> torch.Tensor:
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k = silu(h @ w["q"].T).view(T, H, d), silu(h @ w["k"].T).view(T, H, d)
    v = silu(h @ w["v"].T).view(T, H, dv)
    o = torch.cat([decay_attention(q[:, a], k[:, a], v[:, a], m["decay"][a]) for a in range(H)], -1)
    return (rms_unit(o, eps) * w["norm"] * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def sub(w: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def parallel_mixer(h, w: dict, m: dict, eps: float) -> torch.Tensor:
    return (m["left_scale"] * window_attention(h, sub(w, "left."), m["left"])
            + m["right_scale"] * delta_mixer(h, sub(w, "right."), m["right"], eps))


# ------------------------------------------------------------------- experts


def route(logits: torch.Tensor, top: int, scale: float):
    """(ids [T, top] by falling score, weights)."""
    s = torch.sigmoid(logits)
    val, ids = torch.topk(s, top, -1)
    return ids, val / (val.sum(-1, keepdim=True) + 1e-20) * scale


def experts(h, w: dict, m: dict) -> torch.Tensor:
    ids, weight = route(h @ w["router"].T, m["router"]["top"], m["router"]["scale"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(ids[t].tolist(), weight[t]):
            out[t] += c * (w[f"e{e}.down"] @ (silu(w[f"e{e}.gate"] @ h[t]) * (w[f"e{e}.up"] @ h[t])))
    return out


def forward(config: dict, tensors: dict, tokens, dtype=torch.float64):
    """(logits [T, vocab], residual stream after every layer [layers, T, width])."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x = t["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    after = []
    for i, layer in enumerate(config["layers"]):
        w = sub(t, f"l{i}.")
        h = layer_norm(x, w["norm1"], eps)
        mixer = {"parallel": parallel_mixer, "lightning": lightning_mixer}[layer["type"]]
        x = x + mixer(h, sub(w, "mix."), layer["mixer"], eps) * residual_gate(h, w["rg1"], w["rg1.b"])
        if layer["mlp"] is not None:
            h = layer_norm(x, w["norm2"], eps)
            x = x + experts(h, sub(w, "mlp."), layer["mlp"]) * residual_gate(h, w["rg2"], w["rg2.b"])
        after.append(x)
    return layer_norm(x, t["final.norm"], eps) @ t["head"].T * config["logit_scale"], torch.stack(after)
