"""Plain restatement of the layer-list decoder designs (Sulepel) on the CPU: test infrastructure only.

One function per mechanism, whole sequences at a time, no cache, no batching, no padding: every position is computed
from all the positions before it, straight from the equations.  `dtype` is the working precision (float64 by
default, so that what a comparison shows is the other side's rounding).

  positions   x_p = embed[token_p] + s_p,  s_p[2i] = sin(p / 10000^(2i/width)),  s_p[2i+1] = cos(same)
  layer       x += mixer(short_conv(norm1 x));  x += ff(norm2 x)          (ff may be absent)
  out         logits = head norm(x)
"""
from __future__ import annotations

import torch


def sinusoid(positions: torch.Tensor, width: int, dtype=torch.float64) -> torch.Tensor:
    i = torch.arange(width, dtype=torch.float64)
    ang = positions.double()[:, None] * torch.pow(torch.tensor(10000.0, dtype=torch.float64), -(2.0 * torch.div(i, 2, rounding_mode="floor")) / width)[None]
    return torch.where((torch.arange(width) % 2 == 0)[None], ang.sin(), ang.cos()).to(dtype)


def group_rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, groups: int) -> torch.Tensor:
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    parts = parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)
    return parts.reshape(x.shape) * w


def short_conv(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """h [T, width], w [width, taps]: h_t + sum_j w[:, j] h_{t - taps + 1 + j}, zeros before the start."""
    T, taps = h.shape[0], w.shape[1]
    out = h.clone()
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] = out[t] + w[:, j] * h[s]
    return out


def visible(T: int, chunk: int) -> torch.Tensor:
    """[T, T] bool: position i sees j <= i, and with chunk > 0 only inside its own chunk of positions."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None]
    ok = j <= i
    return ok & (torch.div(i, chunk, rounding_mode="floor") == torch.div(j, chunk, rounding_mode="floor")) if chunk else ok


def softmax_heads(q, k, v, scale: torch.Tensor, chunk: int) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv], scale [H] -> [T, H, dv]; query head h uses key head h // (H/G)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    mask = visible(T, chunk)
    out = torch.empty(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale[h]
        s = s.masked_fill(~mask, float("-inf"))
        out[:, h] = torch.softmax(s, -1) @ v[:, h // per]
    return out


def head_gate(o: torch.Tensor, h: torch.Tensor, wg: torch.Tensor) -> torch.Tensor:
    return o * torch.sigmoid(h @ wg.T)[..., None]


def attention_mixer(h, w: dict, m: dict) -> torch.Tensor:
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(T, H, d)
    k, v = (h @ w["k"].T).view(T, G, d), (h @ w["v"].T).view(T, G, dv)
    o = softmax_heads(q, k, v, w["temp"] * m["scale"], m["mask"]["size"])
    return head_gate(o, h, w["g"]).reshape(T, H * dv) @ w["o"].T


def latent_mixer(h, w: dict, m: dict, eps: float) -> torch.Tensor:
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(T, H, d)
    c = group_rmsnorm(h @ w["dkv"].T, w["dkv.norm"], eps, 1)
    k, v = (c @ w["uk"].T).view(T, H, d), (c @ w["uv"].T).view(T, H, dv)
    o = softmax_heads(q, k, v, torch.full((H,), m["scale"], dtype=h.dtype), 0)
    return head_gate(o, h, w["g"]).reshape(T, H * dv) @ w["o"].T


def clamped_glu(g: torch.Tensor, u: torch.Tensor, limit: float) -> torch.Tensor:
    g, u = g.clamp(max=limit), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def layered_forward(config: dict, tensors: dict, tokens, dtype=torch.float64):
    """(logits [T, vocab], residual stream after every layer [layers, T, width])."""
    t = {k: v.to(dtype) for k, v in tensors.items()}
    eps, groups, width = config["norm"]["eps"], config["norm"]["groups"], config["width"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = t["embed"][ids] + sinusoid(torch.arange(len(ids)), width, dtype)
    after = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        mix = {k[len(p) + 4:]: v for k, v in t.items() if k.startswith(p + "mix.")}
        h = short_conv(group_rmsnorm(x, t[p + "norm1"], eps, groups), t[p + "canon1"])
        if layer["type"] == "attention":
            x = x + attention_mixer(h, mix, layer["mixer"])
        else:
            x = x + latent_mixer(h, mix, layer["mixer"], eps)
        if layer["mlp"] is not None:
            h = group_rmsnorm(x, t[p + "norm2"], eps, groups)
            a = clamped_glu(h @ t[p + "mlp.gate"].T, h @ t[p + "mlp.up"].T, layer["mlp"]["limit"])
            x = x + a @ t[p + "mlp.down"].T
        after.append(x)
    return group_rmsnorm(x, t["final.norm"], eps, groups) @ t["head"].T, torch.stack(after)
