"""Plain, slow Siparax forward pass: whole sequences, no cache, one function per mechanism.

The oracle of the Siparax tests.  It shares no code with the package under test: it reads a model folder through the
``safetensors`` library, forms every head's keys and values from the latents and every attention as a dense [T, T]
table, takes the short convolution as a loop over tokens and taps and walks the delta rule token by token, head by head.

A layer is x <- x + mixer(N1(x)), then x <- x + ff(N2(x)) where it has a feed-forward, N a layer norm with weight and
bias.  The mixer is a gated delta rule with a decay per key channel, or attention through low-rank latents: rotated in
neighbouring pairs and without a gate ("latent_attention"), or in halves, with a gate per head and possibly over
another layer's latents ("latent_attention_2").  The feed-forward is gated by the tanh form of gelu; the embedding is
normed, and the logits of the untied head are capped.

Everything here is 64-bit, so that what is compared against it is the library's rounding and nothing else.
"""

from __future__ import annotations

import json
import math
from pathlib import Path

import torch
from safetensors import safe_open

F = torch.float64


def read_folder(folder):
    """config.json as a dict and every tensor of the folder's *.safetensors files (floats widened to float64)."""
    folder = Path(folder)
    cfg = json.loads((folder / "config.json").read_text())
    tensors = {}
    for path in sorted(folder.glob("*.safetensors")):
        with safe_open(str(path), framework="pt", device="cpu") as f:
            for name in f.keys():
                t = f.get_tensor(name)
                tensors[name] = t.to(F) if t.is_floating_point() else t
    return cfg, tensors


# ---- norms ------------------------------------------------------------------------------------


def layer_norm(x, weight, bias, eps):
    centred = x - x.mean(dim=-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(dim=-1, keepdim=True) + eps) * weight + bias


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit_length(x):
    """x / sqrt(sum(x^2) + 1e-6) over the last axis."""
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


# ---- the delta rule -----------------------------------------------------------------------------


def short_convolution(u, weight):
    """u [T, C], weight [C, taps]: y_t = sum_j weight[:, j] * u_(t - taps + 1 + j), zeros before the start."""
    T, C = u.shape
    taps = weight.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                y[t] += weight[:, j] * u[src]
    return y


def silu(z):
    return z * torch.sigmoid(z)


def channel_decay(h, w, heads, dim):
    """exp(-exp(A_log) * softplus(a2 (a1 h) + dt_bias)), [T, heads, dim]; A_log one number per head."""
    pre = h @ w["a1"].T @ w["a2"].T + w["dt_bias"]
    softplus = torch.clamp(pre, min=0.0) + torch.log1p(torch.exp(-pre.abs()))
    return torch.exp(-torch.exp(w["A_log"])[None, :, None] * softplus.reshape(-1, heads, dim))


def delta_rule(q, k, v, beta, decay):
    """One head: q, k, decay [T, D], v [T, V], beta [T].  The state decays, is corrected towards v at k, then is read."""
    T, D = q.shape
    S = torch.zeros(D, v.shape[1], dtype=F)
    out = torch.zeros(T, v.shape[1], dtype=F)
    for t in range(T):
        S = decay[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def channel_delta(h, w, m, eps):
    """h [T, width]; w: the mixer's tensors by their last names; m: the mixer's entry of config.json."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(short_convolution(h @ w["q"].T, w["q.conv"])).reshape(T, G, D)
    k = silu(short_convolution(h @ w["k"].T, w["k.conv"])).reshape(T, G, D)
    v = silu(short_convolution(h @ w["v"].T, w["v.conv"])).reshape(T, H, V)
    q, k = unit_length(q) * D ** -0.5, unit_length(k)
    beta = torch.sigmoid(h @ w["b"].T)
    decay = channel_decay(h, w, H, D)
    gate = torch.sigmoid(h @ w["g1"].T @ w["g2"].T).reshape(T, H, V)
    outs = []
    for head in range(H):
        c = head // (H // G)
        o = delta_rule(q[:, c], k[:, c], v[:, head], beta[:, head], decay[:, head])
        outs.append(unit_rms(o, eps) * w["norm"] * gate[:, head])
    return torch.cat(outs, dim=-1) @ w["o"].T


# ---- attention through latents --------------------------------------------------------------------


def stretched_frequencies(rot):
    """(frequency of every pair, what multiplies cosines and sines) from a rotation's entry of config.json."""
    dims, base = int(rot["dims"]), float(rot["base"])
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc is None:
        return plain, 1.0

    def place(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(place(sc["fast"])), 0)
    hi = min(math.ceil(place(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(t, rot, halves):
    """t [T, ..., R] at positions 0 .. T - 1: pair i is columns (i, i + dims / 2) with ``halves``, else (2 i, 2 i + 1)."""
    freqs, magnitude = stretched_frequencies(rot)
    dims = int(rot["dims"])
    out = t.clone()
    pos = torch.arange(t.shape[0]).to(F)
    for i, f in enumerate(freqs):
        a, b = (i, i + dims // 2) if halves else (2 * i, 2 * i + 1)
        c = (torch.cos(pos * f) * magnitude).reshape((-1,) + (1,) * (t.dim() - 2))
        s = (torch.sin(pos * f) * magnitude).reshape((-1,) + (1,) * (t.dim() - 2))
        u, v = t[..., a], t[..., b]
        out[..., a] = u * c - v * s
        out[..., b] = v * c + u * s
    return out


def causal_softmax(s):
    T = s.shape[0]
    s = s.masked_fill(~torch.ones(T, T, dtype=torch.bool).tril(), float("-inf"))
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


def latent_rows(h, w, m, eps, halves):
    """(latent c [T, kv_rank], rotated key part [T, rot_dim]) of a layer with a down-projection of its own."""
    d = h @ w["dkv"].T
    rank = m["kv_rank"]
    return unit_rms(d[:, :rank], eps) * w["dkv.norm"], rotate(d[:, rank:], m["rot"], halves)


def latent_attention(h, w, m, eps, halves, gated, rows=None):
    """``rows``: another layer's (latent, rotated key part) that this layer reads instead of making its own.  Returns
    (output, the rows it read)."""
    T = h.shape[0]
    H, D, R, V = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    if rows is None:
        rows = latent_rows(h, w, m, eps, halves)
    c, k_rot = rows
    q = ((unit_rms(h @ w["dq"].T, eps) * w["dq.norm"]) @ w["uq"].T).reshape(T, H, D + R)
    q_rot = rotate(q[..., D:], m["rot"], halves)
    k = (c @ w["uk"].T).reshape(T, H, D)
    v = (c @ w["uv"].T).reshape(T, H, V)
    outs = []
    for head in range(H):
        s = (q[:, head, :D] @ k[:, head].T + q_rot[:, head] @ k_rot.T) * float(m["scale"])
        o = causal_softmax(s) @ v[:, head]
        if gated:
            o = o * torch.sigmoid(h @ w["g"][head])[:, None]
        outs.append(o)
    return torch.cat(outs, dim=-1) @ w["o"].T, rows


# ---- feed-forward, layers, the model ----------------------------------------------------------------


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def feed_forward(h, gate, up, down):
    return (gelu_tanh(h @ gate.T) * (h @ up.T)) @ down.T


def below(tensors, prefix):
    """{name without the prefix: tensor} of the tensors whose names start with it."""
    return {name[len(prefix):]: t for name, t in tensors.items() if name.startswith(prefix)}


def layer(x, cfg, tensors, i, shared):
    """``shared``: {layer: the latent rows it made}, filled as the layers run."""
    entry, eps, p = cfg["layers"][i], float(cfg["norm"]["eps"]), f"l{i}."
    w, m = below(tensors, p + "mix."), entry["mixer"]
    h = layer_norm(x, tensors[p + "norm1"], tensors[p + "norm1.b"], eps)
    if entry["type"] == "channel_delta":
        y = channel_delta(h, w, m, eps)
    else:
        second = entry["type"] == "latent_attention_2"
        source = m.get("kv_from")
        y, shared[i] = latent_attention(h, w, m, eps, halves=second, gated=second, rows=None if source is None else shared[source])
    x = x + y
    if entry.get("mlp") is not None:
        h = layer_norm(x, tensors[p + "norm2"], tensors[p + "norm2.b"], eps)
        x = x + feed_forward(h, tensors[p + "mlp.gate"], tensors[p + "mlp.up"], tensors[p + "mlp.down"])
    return x


def forward(cfg, tensors, tokens, layers_out=None):
    """Logits [T, vocab] (32-bit) of one sequence; ``layers_out`` receives the residual after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = layer_norm(tensors["embed"][torch.tensor(tokens)], tensors["embed.norm"], tensors["embed.norm.b"], eps)
    shared = {}
    for i in range(len(cfg["layers"])):
        x = layer(x, cfg, tensors, i, shared)
        if layers_out is not None:
            layers_out.append(x.to(torch.float32))
    logits = layer_norm(x, tensors["final.norm"], tensors["final.norm.b"], eps) @ tensors["head"].T
    cap = cfg.get("logit_softcap")
    if cap is not None:
        logits = cap * torch.tanh(logits / cap)
    return logits.to(torch.float32)


def generate(cfg, tensors, prompts, n_new):
    """Greedy continuation of every prompt by ``n_new`` tokens, each from a full forward pass."""
    out = []
    for prompt in prompts:
        seq = list(prompt)
        for _ in range(n_new):
            seq.append(int(forward(cfg, tensors, seq)[-1].argmax()))
        out.append(seq[len(prompt):])
    return out
