"""Plain, slow Nifalorn forward pass: whole sequences, no cache, one function per mechanism.

The oracle of the Nifalorn tests.  It shares no code with the package under test: it reads a model folder through the
``safetensors`` library, builds every attention as a dense [T, T] table per head and map, walks both recurrences token
by token, takes the short convolution as a loop over its taps and runs every expert of a token in a Python loop.

A Nifalorn layer is x <- x + mixer(N1(x)), then x <- x + ff(N2(x)) where it has a feed-forward, with
N(y) = y / sqrt(mean(y^2) + eps) * (1 + w).  A run of layers may repeat with the same weights and nothing in between.
Mixers: lightning attention (a matrix state per head that decays by a constant), a Mamba-2 layer (a matrix state per head
whose decay and step size depend on the token, groups of heads that share keys and queries), and attention with two score
maps per head, rotated in neighbouring pairs, over the query's own chunk of positions.  The feed-forward is dense (up,
squared relu, down) or a mixture of experts with sigmoid scores, chosen inside the best groups of experts, beside a
shared expert with a gate of its own.

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


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def one_plus_norm(x, weight, eps):
    """RMS norm whose weight is stored around zero."""
    return unit_rms(x, eps) * (1.0 + weight)


def silu(z):
    return z / (1.0 + torch.exp(-z))


# ---- lightning attention ---------------------------------------------------------------------


def decayed_memory(q, k, v, decay, step=None, state=None):
    """One head, token by token: S <- decay_t S + step_t k_t v_t^T, o_t = S^T q_t.  q, k [T, D], v [T, V], decay and step
    [T].  Returns (o [T, V], final S)."""
    T = q.shape[0]
    S = torch.zeros(q.shape[1], v.shape[1], dtype=F) if state is None else state.clone()
    o = torch.zeros(T, v.shape[1], dtype=F)
    for t in range(T):
        add = torch.outer(k[t], v[t])
        S = decay[t] * S + (add if step is None else step[t] * add)
        o[t] = S.T @ q[t]
    return o, S


def lightning_attention(h, w, m, eps):
    """h [T, width]; w: the mixer's tensors by short name; m: the mixer's config entry."""
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w["q"].T).reshape(T, H, D)
    k = silu(h @ w["k"].T).reshape(T, H, D)
    v = silu(h @ w["v"].T).reshape(T, H, V)
    heads = []
    for i in range(H):
        heads.append(decayed_memory(q[:, i], k[:, i], v[:, i], torch.full((T,), float(m["decay"][i]), dtype=F))[0])
    o = unit_rms(torch.cat(heads, dim=-1), eps) * w["norm"]
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# ---- Mamba-2 ---------------------------------------------------------------------------------


def causal_convolution(u, weight, bias):
    """u [T, C], weight [C, taps] (the last column meets the current token), bias [C]; zeros before the start."""
    T, taps = u.shape[0], weight.shape[1]
    out = bias[None, :].repeat(T, 1)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += weight[:, j][None, :] * u[:T - back]
    return out


def parts_norm(y, weight, parts, eps):
    """The row in equal consecutive parts, each divided by its own root mean square, times the weight."""
    T = y.shape[0]
    return unit_rms(y.reshape(T, parts, -1), eps).reshape(T, -1) * weight


def mamba2(h, w, m, eps):
    T, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    p = h @ w["in"].T
    z, u, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    u = silu(causal_convolution(u, w["conv"], w["conv.b"]))
    x, B, C = u[:, :inner].reshape(T, H, V), u[:, inner:inner + G * N].reshape(T, G, N), u[:, inner + G * N:].reshape(T, G, N)
    dt = torch.log1p(torch.exp(-(dt + w["dt_bias"]).abs())) + torch.clamp(dt + w["dt_bias"], min=0.0)     # softplus
    heads = []
    for i in range(H):
        g = i // (H // G)
        decay = torch.exp(-torch.exp(w["A_log"][i]) * dt[:, i])
        o, _ = decayed_memory(C[:, g], B[:, g], x[:, i], decay, step=dt[:, i])
        heads.append(o + w["D"][i] * x[:, i])
    y = torch.cat(heads, dim=-1) * silu(z)
    return parts_norm(y, w["norm"], m["norm_groups"], eps) @ w["o"].T


# ---- attention with two score maps over the query's chunk -------------------------------------


def rotary_frequencies(rot):
    """f_i = base^(-2i / dims); with scaling {factor, low, high, original} a frequency whose wavelength 2 pi / f is longer
    than original / low turns ``factor`` times slower, one shorter than original / high stays, a blend between."""
    dims = int(rot["dims"])
    out = []
    for i in range(dims // 2):
        f = float(rot["base"]) ** (-2.0 * i / dims)
        sc = rot.get("scaling")
        if sc:
            length = 2.0 * math.pi / f
            if length > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif length >= sc["original"] / sc["high"]:
                s = (sc["original"] / length - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_pairs(t, positions, rot):
    """t [T, ..., D]: columns (2i, 2i + 1) of the first rot.dims turn by positions * f_i, the rest pass."""
    if not rot:
        return t
    out = t.clone()
    shape = (-1,) + (1,) * (t.dim() - 2)
    for i, f in enumerate(rotary_frequencies(rot)):
        angle = positions.to(F) * f
        c, s = torch.cos(angle).reshape(shape), torch.sin(angle).reshape(shape)
        u, v = t[..., 2 * i], t[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def chunk_table(T, size):
    """[T, T] True where query i sees key j: j <= i, both in one chunk of ``size`` positions (no size: every j <= i)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if size:
        seen &= torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor")
    return seen


def diff_attention(h, w, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    positions = torch.arange(T)
    q = rotate_pairs((h @ w["q"].T).reshape(T, H, 2, D), positions, m.get("rot"))
    k = rotate_pairs((h @ w["k"].T).reshape(T, G, 2, D), positions, m.get("rot"))
    v = (h @ w["v"].T).reshape(T, G, V)
    seen = chunk_table(T, (m.get("mask") or {}).get("size"))
    lam = math.exp(float((w["lq1"] * w["lk1"]).sum())) - math.exp(float((w["lq2"] * w["lk2"]).sum())) + m["diff"]
    heads = []
    for i in range(H):
        g = i // (H // G)
        maps = []
        for which in range(2):
            score = (q[:, i, which] @ k[:, g, which].T) * m["scale"]
            maps.append(torch.softmax(score.masked_fill(~seen, float("-inf")), dim=-1) @ v[:, g])
        heads.append(unit_rms(maps[0] - lam * maps[1], eps) * (1.0 - m["diff"]))
    return torch.cat(heads, dim=-1) @ w["o"].T


# ---- feed-forward ----------------------------------------------------------------------------


def squared_relu(h, up, down):
    return torch.relu(h @ up.T) ** 2 @ down.T


def gated(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(h, router, correction, r):
    """(chosen [T, top], weights [T, top]), one token after another."""
    s = 1.0 / (1.0 + torch.exp(-(h @ router.T)))
    groups = r.get("groups") or {"count": 1, "keep": 1}
    each = s.shape[1] // groups["count"]
    chosen = torch.zeros(h.shape[0], r["top"], dtype=torch.long)
    weights = torch.zeros(h.shape[0], r["top"], dtype=F)
    for t in range(h.shape[0]):
        choice = (s[t] + correction).tolist()
        totals = [sum(sorted(choice[g * each:(g + 1) * each], reverse=True)[:2]) for g in range(groups["count"])]
        kept = sorted(range(groups["count"]), key=lambda g: -totals[g])[:groups["keep"]]
        allowed = [e for g in kept for e in range(g * each, (g + 1) * each)]
        best = sorted(allowed, key=lambda e: -choice[e])[:r["top"]]
        chosen[t] = torch.tensor(best)
        weights[t] = s[t, best] / (s[t, best].sum() + 1e-20) * r.get("scale", 1.0)
    return chosen, weights


def expert_mixture(h, w, mlp):
    """h [T, width]; w: the feed-forward's tensors by short name ('e3.gate', 'router', 'shared.sg', ...)."""
    chosen, weights = route(h, w["router"], w["correction"], mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, wt in zip(chosen[t].tolist(), weights[t]):
            out[t] += wt * gated(h[t:t + 1], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])[0]
    if mlp.get("shared"):
        share = 1.0 / (1.0 + torch.exp(-(h @ w["shared.sg"].T)))
        out = out + share * gated(h, w["shared.gate"], w["shared.up"], w["shared.down"])
    return out


# ---- layers, the model -----------------------------------------------------------------------


MIXERS = {"lightning": lightning_attention, "mamba2": mamba2, "attention": diff_attention}


def below(tensors, prefix):
    """{name without the prefix: tensor} of the tensors whose names start with it."""
    return {name[len(prefix):]: t for name, t in tensors.items() if name.startswith(prefix)}


def layer(x, cfg, tensors, i):
    entry, eps, p = cfg["layers"][i], float(cfg["norm"]["eps"]), f"l{i}."
    x = x + MIXERS[entry["type"]](one_plus_norm(x, tensors[p + "norm1"], eps), below(tensors, p + "mix."), entry["mixer"], eps)
    mlp = entry.get("mlp")
    if mlp is not None:
        h, w = one_plus_norm(x, tensors[p + "norm2"], eps), below(tensors, p + "mlp.")
        x = x + (squared_relu(h, w["up"], w["down"]) if mlp["kind"] == "dense" else expert_mixture(h, w, mlp))
    return x


def layer_runs(cfg):
    """The layers in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if loop is None:
        return list(range(n))
    return (list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n)))


def forward(cfg, tensors, tokens, layers_out=None):
    """Logits [T, vocab] (32-bit) of one sequence; ``layers_out`` receives the residual after every layer run."""
    x = tensors["embed"][torch.tensor(tokens)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    for i in layer_runs(cfg):
        x = layer(x, cfg, tensors, i)
        if layers_out is not None:
            layers_out.append(x.to(torch.float32))
    x = one_plus_norm(x, tensors["final.norm"], float(cfg["norm"]["eps"]))
    return ((x @ tensors["head"].T) * float(cfg.get("logit_scale", 1.0))).to(torch.float32)


def generate(cfg, tensors, prompts, n_new):
    """Greedy continuation of every prompt by ``n_new`` tokens, each from a full forward pass."""
    out = []
    for prompt in prompts:
        seq = list(prompt)
        for _ in range(n_new):
            seq.append(int(forward(cfg, tensors, seq)[-1].argmax()))
        out.append(seq[len(prompt):])
    return out
