"""The Tanupel architecture written out plainly in float64, one function per mechanism.

A slow oracle for the tests: whole sequences only, no cache, no batching, no kernels; it shares no
code with the engine. Weights come as a dict of tensors under the checkpoint's names and the
configuration as the plain dict of ``config.json``.

Notation: ``x`` is the residual stream ``[n, width]`` of one sequence whose tokens sit at
positions 0 .. n-1, ``h`` a layer's normed input.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def mat(w, name):
    return w[name].to(F64)


# ----------------------------------------------------------------------------- norms, activations
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def offset_norm(x, w, eps):
    """The weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + w)


def silu(z):
    return z * torch.sigmoid(z)


# ----------------------------------------------------------------------------- attention
def frequencies(rot):
    """float64 [dims / 2]. ``scaling`` with a factor alone divides every frequency; with low, high and
    original it leaves short waves, divides long ones and blends between the two."""
    dims = rot["dims"]
    f = [float(rot["base"]) ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if s and "original" not in s:
        f = [v / s["factor"] for v in f]
    elif s:
        out = []
        for v in f:
            wave = 2.0 * math.pi / v
            if wave < s["original"] / s["high"]:
                out.append(v)
            elif wave > s["original"] / s["low"]:
                out.append(v / s["factor"])
            else:
                t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                out.append((1.0 - t) * v / s["factor"] + t * v)
        f = out
    return torch.tensor(f, dtype=F64)


def rotate_halves(x, pos, rot):
    """x [n, heads, d]: dim i of the first ``dims`` is turned with dim i + dims / 2."""
    if not rot or not rot["dims"]:
        return x
    half = rot["dims"] // 2
    a = pos.to(F64)[:, None] * frequencies(rot)[None, :]
    c, s = a.cos()[:, None, :], a.sin()[:, None, :]
    u, v = x[..., :half], x[..., half : 2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half :]], -1)


def attend(q, k, v, scale, softcap=0.0):
    """q [n, H, d], k [n, G, d], v [n, G, dv]: every query sees itself and what lies before it -> [n, H, dv]."""
    n, H, _ = q.shape
    group = H // k.shape[1]
    hidden = torch.ones(n, n, dtype=torch.bool).triu(1)
    outs = []
    for h in range(H):
        s = q[:, h] @ k[:, h // group].T * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        outs.append(s.masked_fill(hidden, -math.inf).softmax(-1) @ v[:, h // group])
    return torch.stack(outs, 1)


def attention(h, w, prefix, m, eps):
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms(h @ mat(w, prefix + "q").T, eps) * mat(w, prefix + "q.norm")  # over all heads at once
    k = unit_rms(h @ mat(w, prefix + "k").T, eps) * mat(w, prefix + "k.norm")
    v = (h @ mat(w, prefix + "v").T).view(n, G, dv)
    pos = torch.arange(n)
    q = rotate_halves(q.view(n, H, d), pos, m.get("rot"))
    k = rotate_halves(k.view(n, G, d), pos, m.get("rot"))
    o = attend(q, k, v, m["scale"], m.get("softcap") or 0.0)
    return o.reshape(n, H * dv) @ mat(w, prefix + "o").T


# ----------------------------------------------------------------------------- gated delta rule
def short_conv(x, taps):
    """x [n, channels], taps [channels, K]: y[t] = sum_j taps[:, K-1-j] x[t-j], zeros before the start."""
    n, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(n):
        for j in range(min(K, t + 1)):
            y[t] += taps[:, K - 1 - j] * x[t - j]
    return y


def unit_vector(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_decays(z, A_log, dt_bias):
    """z [n, H * d] -> g [n, H, d], one number per head and key channel; A_log per head."""
    n, H = z.shape[0], A_log.shape[0]
    step = torch.nn.functional.softplus(z + dt_bias, threshold=1e9).view(n, H, -1)
    return torch.exp(-torch.exp(A_log)[None, :, None] * step)


def delta_rule(q, k, v, beta, g, S=None):
    """q, k, g [n, H, d], v [n, H, dv], beta [n, H]. Outputs [n, H, dv] and the last state [H, d, dv]."""
    n, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64) if S is None else S.to(F64).clone()
    o = torch.zeros(n, H, v.shape[-1], dtype=F64)
    for t in range(n):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o, S


def delta_inputs(h, w, prefix, m):
    """q, k [n, H, d] (unit vectors, q scaled, key heads repeated), v, beta [n, H], g [n, H, d]."""
    n = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ mat(w, prefix + t).T, mat(w, prefix + t + ".conv"))) for t in "qkv")
    q = unit_vector(q.view(n, G, d)) * d ** -0.5
    k = unit_vector(k.view(n, G, d))
    beta = torch.sigmoid(h @ mat(w, prefix + "b").T)
    z = (h @ mat(w, prefix + "a1").T) @ mat(w, prefix + "a2").T
    g = channel_decays(z, mat(w, prefix + "A_log"), mat(w, prefix + "dt_bias"))
    rep = lambda t: t.repeat_interleave(H // G, 1)
    return rep(q), rep(k), v.view(n, H, dv), beta, g


def gated_delta(h, w, prefix, m, eps):
    n = h.shape[0]
    o, _ = delta_rule(*delta_inputs(h, w, prefix, m))
    y = (unit_rms(o, eps) * mat(w, prefix + "norm")).reshape(n, -1)
    y = y * torch.sigmoid((h @ mat(w, prefix + "g1").T) @ mat(w, prefix + "g2").T)
    return y @ mat(w, prefix + "o").T


def mixer(h, w, prefix, layer, eps):
    m = layer["mixer"]
    if layer["type"] == "attention":
        return attention(h, w, prefix, m, eps)
    return (m["left_scale"] * attention(h, w, prefix + "left.", m["left"], eps)
            + m["right_scale"] * gated_delta(h, w, prefix + "right.", m["right"], eps))


# ----------------------------------------------------------------------------- feed-forward
def gated(h, w, prefix):
    return (silu(h @ mat(w, prefix + "gate").T) * (h @ mat(w, prefix + "up").T)) @ mat(w, prefix + "down").T


def choose(z, correction, top):
    """Router logits z [n, E] -> chosen [n, top] and their weights (not renormalised). Ties to the lower index."""
    s = z.softmax(-1)
    idx = torch.zeros(z.shape[0], top, dtype=torch.long)
    for t in range(z.shape[0]):
        c = (s[t] + correction).tolist()
        idx[t] = torch.tensor(sorted(range(len(c)), key=lambda e: (-c[e], e))[:top])
    return idx, s.gather(1, idx)


def moe(h, w, prefix, mlp):
    idx, wts = choose(h @ mat(w, prefix + "router").T, mat(w, prefix + "correction"), mlp["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        share = (wts * (idx == e)).sum(1)
        rows = share.nonzero()[:, 0]
        if len(rows):
            out[rows] += share[rows, None] * gated(h[rows], w, f"{prefix}e{e}.")
    return out


def feed_forward(h, w, prefix, mlp):
    if mlp is None:
        return torch.zeros_like(h)
    return gated(h, w, prefix) if mlp["kind"] == "dense" else moe(h, w, prefix, mlp)


# ----------------------------------------------------------------------------- the model
def run_order(cfg):
    """(layer, pass or None): layers start .. stop-1 run ``times`` times in a row; the pass is named at its first layer."""
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": n, "stop": n, "times": 1}
    order = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None) for i in range(loop["stop"], n)]


def forward(tokens, w, cfg, return_layers=False):
    """Logits [n, vocab] of one whole sequence (and the residual stream after every run of a layer)."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = mat(w, "embed")[list(tokens)] * cfg["embedding"]["scale"]
    after = []
    for i, t in run_order(cfg):
        layer, pre = cfg["layers"][i], f"l{i}."
        if t is not None:
            x = x + mat(w, "loop.step")[t]
        h = offset_norm(x, mat(w, pre + "norm1"), eps)
        x = x + m * (mixer(h, w, pre + "mix.", layer, eps) + feed_forward(h, w, pre + "mlp.", layer["mlp"]))
        after.append(x)
    logits = offset_norm(x, mat(w, "final.norm"), eps) @ mat(w, "head").T
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
