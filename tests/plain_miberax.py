"""The Miberax architecture written out plainly in float64, one function per mechanism.

A slow oracle for the tests: whole sequences only, no cache, no batching, no kernels; it shares no
code with the engine. Weights come as a dict of tensors under the checkpoint's names and the
configuration as the plain dict of ``config.json``.

Notation: ``x`` is the residual stream ``[n, width]`` of one sequence whose tokens sit at
positions 0 .. n-1, ``h`` a sublayer's input.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


# ----------------------------------------------------------------------------- norms
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def grouped_norm(x, w, groups, eps):
    """Each of ``groups`` equal consecutive parts divided by its own root mean square, times ``w``."""
    n, width = x.shape
    parts = x.reshape(n, groups, width // groups)
    return unit_rms(parts, eps).reshape(n, width) * w


def silu(z):
    return z * torch.sigmoid(z)


# ----------------------------------------------------------------------------- chunked attention
def rotate_neighbours(x, pos, dims, base, factor=1.0):
    """x [n, heads, d]: the pairs (2i, 2i + 1) of the first ``dims`` dims turned by
    ``pos * base^(-2i/dims) / factor``."""
    if dims == 0:
        return x
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=F64) / dims) / factor
    a = pos.to(F64)[:, None] * f[None, :]
    c, s = a.cos()[:, None, :], a.sin()[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def chunk_mask(n, size):
    i = torch.arange(n)[:, None]
    j = torch.arange(n)[None, :]
    seen = j <= i
    return seen & (i // size == j // size) if size else seen


def attend(q, k, v, scale, seen):
    """q [n, H, d], k [n, G, d], v [n, G, dv], seen [n, n] -> [n, H, dv]."""
    group = q.shape[1] // k.shape[1]
    outs = []
    for h in range(q.shape[1]):
        s = (q[:, h] @ k[:, h // group].T * scale).masked_fill(~seen, -math.inf)
        outs.append(s.softmax(-1) @ v[:, h // group])
    return torch.stack(outs, 1)


def chunked_attention(h, w, prefix, m):
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[prefix + "q"].to(F64).T).view(n, H, d)
    k = (h @ w[prefix + "k"].to(F64).T).view(n, G, d)
    v = (h @ w[prefix + "v"].to(F64).T).view(n, G, dv)
    rot = m.get("rot")
    if rot:
        factor = (rot.get("scaling") or {}).get("factor", 1.0)
        pos = torch.arange(n)
        q = rotate_neighbours(q, pos, rot["dims"], rot["base"], factor)
        k = rotate_neighbours(k, pos, rot["dims"], rot["base"], factor)
    o = attend(q, k, v, m["scale"], chunk_mask(n, int((m.get("mask") or {}).get("size", 0))))
    return o.reshape(n, H * dv) @ w[prefix + "o"].to(F64).T


# ----------------------------------------------------------------------------- gated delta rule
def short_conv(x, taps):
    """x [n, channels], taps [channels, K]: y[t] = sum_j taps[:, K-1-j] x[t-j], zeros before the start."""
    K = taps.shape[1]
    y = torch.zeros_like(x)
    for j in range(K):
        y[j:] += taps[:, K - 1 - j] * x[: x.shape[0] - j] if j < x.shape[0] else 0.0
    return y


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, g, S=None):
    """q, k [n, H, d], v [n, H, dv], beta, g [n, H]. Returns outputs [n, H, dv] and the last state
    [H, d, dv]."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64) if S is None else S.to(F64).clone()
    o = torch.zeros(n, H, v.shape[-1], dtype=F64)
    for t in range(n):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o, S


def decay(a, A_log, dt_bias):
    return torch.exp(-torch.exp(A_log) * torch.nn.functional.softplus(a + dt_bias, threshold=1e9))


def delta_inputs(h, w, prefix, m):
    """What enters the recurrence: q, k [n, H, d] (unit vectors, q scaled, heads repeated), v, beta, g."""
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ w[prefix + t].to(F64).T, w[prefix + t + ".conv"].to(F64))) for t in "qkv")
    q = unit_vector(q.view(n, G, d)) * d ** -0.5
    k = unit_vector(k.view(n, G, d))
    beta = torch.sigmoid(h @ w[prefix + "b"].to(F64).T)
    g = decay(h @ w[prefix + "a"].to(F64).T, w[prefix + "A_log"].to(F64), w[prefix + "dt_bias"].to(F64))
    rep = lambda t: t.repeat_interleave(H // G, 1)
    return rep(q), rep(k), v.view(n, H, dv), beta, g


def gated_delta(h, w, prefix, m, eps):
    n = h.shape[0]
    o, _ = delta_rule(*delta_inputs(h, w, prefix, m))
    y = unit_rms(o, eps) * w[prefix + "norm"].to(F64)
    y = y.reshape(n, -1) * silu(h @ w[prefix + "g"].to(F64).T)
    return y @ w[prefix + "o"].to(F64).T


def parallel(h, w, prefix, m, eps):
    a = chunked_attention(h, w, prefix + "left.", m["left"])
    b = gated_delta(h, w, prefix + "right.", m["right"], eps)
    return 0.5 * (unit_rms(a, eps) * w[prefix + "left.out"].to(F64) + unit_rms(b, eps) * w[prefix + "right.out"].to(F64))


# ----------------------------------------------------------------------------- feed-forward
def poly_norm(z, coef, eps):
    a, b, c, e = (coef[i] for i in range(4))
    return a * unit_rms(z, eps) + b * unit_rms(z ** 2, eps) + c * unit_rms(z ** 3, eps) + e


def clamped_glu(gate, up, limit):
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def expert(h, w, prefix, limit):
    a = clamped_glu(h @ w[prefix + "gate"].to(F64).T, h @ w[prefix + "up"].to(F64).T, limit)
    return a @ w[prefix + "down"].to(F64).T


def choose(z, correction, top, groups=1, keep=1, scale=1.0):
    """Router logits z [n, experts + identity] -> chosen [n, top] and their weights. One token at a
    time, ties to the lower index."""
    n, E = z.shape
    size = E // groups
    idx = torch.zeros(n, top, dtype=torch.long)
    wts = torch.zeros(n, top, dtype=F64)
    s = z.softmax(-1)
    for t in range(n):
        c = (s[t] + correction).tolist()
        best = sorted(range(groups), key=lambda g: (-max(c[g * size : (g + 1) * size]), g))[:keep]
        allowed = [e for e in range(E) if e // size in best]
        chosen = sorted(allowed, key=lambda e: (-c[e], e))[:top]
        idx[t] = torch.tensor(chosen)
        val = s[t][chosen]
        wts[t] = val / (val.sum() + 1e-20) * scale
    return idx, wts


def route(h, w, prefix, r):
    g = r.get("groups") or {"count": 1, "keep": 1}
    return choose(h @ w[prefix + "router"].to(F64).T, w[prefix + "correction"].to(F64), r["top"], g["count"], g["keep"],
                  r.get("scale", 1.0))


def moe(h, w, prefix, mlp):
    r = mlp["router"]
    idx, wts = route(h, w, prefix, r)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(idx[t].tolist(), wts[t]):
            y = h[t] if e >= r["experts"] else expert(h[t][None], w, f"{prefix}e{e}.", mlp["expert"]["limit"])[0]
            out[t] += wt * y
    if mlp.get("shared"):
        gate = torch.sigmoid(h @ w[prefix + "shared.sg"].to(F64).T)
        out = out + gate * expert(h, w, prefix + "shared.", mlp["shared"]["limit"])
    return out


def feed_forward(h, w, prefix, mlp, eps):
    if mlp["kind"] == "dense":
        a = poly_norm(h @ w[prefix + "up"].to(F64).T, w[prefix + "act"].to(F64), eps)
        return a @ w[prefix + "down"].to(F64).T
    return moe(h, w, prefix, mlp)


# ----------------------------------------------------------------------------- the model
def forward(tokens, w, cfg, return_layers=False):
    """Logits [n, vocab] of one whole sequence (and the residual stream after every layer)."""
    eps, groups = cfg["norm"]["eps"], cfg["norm"].get("groups", 1)
    x = w["embed"].to(F64)[list(tokens)]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        x = x + parallel(grouped_norm(x, w[pre + "norm1"].to(F64), groups, eps), w, pre + "mix.", layer["mixer"], eps)
        if layer["mlp"] is not None:
            h = grouped_norm(x, w[pre + "norm2"].to(F64), groups, eps)
            x = x + feed_forward(h, w, pre + "mlp.", layer["mlp"], eps)
        after.append(x)
    logits = grouped_norm(x, w["final.norm"].to(F64), groups, eps) @ w["embed"].to(F64).T
    return (logits, torch.stack(after)) if return_layers else logits


def load(folder):
    import json
    from pathlib import Path

    from safetensors.torch import load_file

    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    return cfg, {k: v.to(F64) if v.is_floating_point() else v for k, v in load_file(str(folder / "model.safetensors")).items()}


def model_logits(folder, tokens):
    cfg, w = load(folder)
    return forward(list(tokens), w, cfg).float()


def greedy(folder, prompt, n):
    """n tokens generated greedily after ``prompt`` (the whole sequence is run again each time)."""
    cfg, w = load(folder)
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(forward(tokens, w, cfg)[-1].argmax()))
    return tokens[len(prompt):]
