"""Tagulix, stated plainly: one function per mechanism, float64, a Python loop over the positions wherever one position
depends on the ones before it. Nothing here is shared with the engine; the tests compare the engine with it.

A model is a dict of tensors by checkpoint name and the config.json dict. Notation: h [T, D] is a mixer's input, rows are
the positions 0 .. T - 1 of ONE sequence. The stream is s rows x_1 .. x_s of width D per position (`hyper`): a sublayer reads a
weighted sum of them, and its output joins all of them.
"""

from __future__ import annotations

import math

import torch

F64 = torch.float64


def lin(w, h, b=None):
    """Matrices are stored [out, in]."""
    y = h @ w.to(F64).T
    return y if b is None else y + b.to(F64)


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, gain, eps):
    return unit_rms(x, eps) * gain.to(F64)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


# A test may set this to a function that disturbs the rows on their way into every sublayer (and into the head): how far the
# logits of a position move under small disturbances says how well-conditioned the position is.
DISTURB = None
# A test may set this to a list: every router then appends, per position, how narrowly its choice was made (the smallest gap
# between something chosen and something not, among experts and among groups).
MARGINS = None


# ---- attention -----------------------------------------------------------------------------------
def rotate_pairs(x, positions, dims, base):
    """x [T, heads, d]: of each head the pairs (2i, 2i + 1), i < dims / 2, turn by position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = torch.tensor([p * base ** (-2.0 * i / dims) for p in positions], dtype=F64)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def distance_bucket(n: int, buckets: int, bias_max: int) -> int:
    """The row of the bias table for a key n positions back: the first half of the rows are distances of their own, the rest
    cover the distances up to bias_max in equal steps of the logarithm; everything farther shares the last row."""
    half = buckets // 2
    if n < half:
        return n
    return min(buckets - 1, half + math.floor(math.log(n / half) / math.log(bias_max / half) * (buckets - half)))


def distance_bias(table, n_positions: int, bias_max: int):
    """table [B, H] -> [H, n_positions]: head h's bias for a key n positions back."""
    rows = [distance_bucket(n, table.shape[0], bias_max) for n in range(n_positions)]
    return table.to(F64)[rows].T.contiguous()


def query_temperature(position: int, coef: float, every: int) -> float:
    return 1.0 + coef * math.log(math.floor((position + 1) / every) + 1)


def attend(q, k, v, scale, window=0, bias=None, sink=None, positions=None):
    """q [T, H, d], k [J, G, d], v [J, G, dv] of one sequence; positions[t] is row t's place (default t). A row at position i sees
    the keys j <= i with i - j < window (window 0: all of them). bias [H, >= J] by distance, added after the scale; sink [H]: one
    more term exp(sink) in the denominator."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    k_of, v_of = k.repeat_interleave(per, dim=1), v.repeat_interleave(per, dim=1)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        i = t if positions is None else positions[t]
        j0 = max(0, i - window + 1) if window else 0
        s = torch.einsum("hd,jhd->hj", q[t], k_of[j0: i + 1]) * scale
        if bias is not None:
            s = s + bias[:, : i - j0 + 1].flip(-1)        # key j stands i - j back
        top = s.max(dim=-1).values
        if sink is not None:
            top = torch.maximum(top, sink)
        e = torch.exp(s - top[:, None])
        total = e.sum(dim=-1)
        if sink is not None:
            total = total + torch.exp(sink - top)
        out[t] = torch.einsum("hj,jhv->hv", e / total[:, None], v_of[j0: i + 1])
    return out


def window_attention(h, w, p, cfg, eps):
    """Rotated queries and keys, then each head's divided by its root mean square; a sliding window; biases everywhere."""
    T, H, d = h.shape[0], cfg["heads"], cfg["dim"]
    G, dv = cfg.get("kv_heads", H), cfg.get("vdim", d)
    pos = list(range(T))
    q, k = lin(w[p + "q"], h, w[p + "q.b"]).view(T, H, d), lin(w[p + "k"], h, w[p + "k.b"]).view(T, G, d)
    v = lin(w[p + "v"], h, w[p + "v.b"]).view(T, G, dv)
    if cfg.get("rot"):
        q, k = (rotate_pairs(x, pos, cfg["rot"]["dims"], float(cfg["rot"]["base"])) for x in (q, k))
    out = attend(unit_rms(q, eps), unit_rms(k, eps), v, cfg["scale"], window=(cfg.get("mask") or {}).get("size", 0))
    return lin(w[p + "o"], out.reshape(T, H * dv), w[p + "o.b"])


def biased_attention(h, w, p, cfg, eps):
    """No rotation: a learned bias by distance, queries that grow with the position, a sink; every earlier position is seen."""
    T, H, d = h.shape[0], cfg["heads"], cfg["dim"]
    G, dv = cfg.get("kv_heads", H), cfg.get("vdim", d)
    q = rms_norm(lin(w[p + "q"], h).view(T, H, d), w[p + "q.norm"], eps)
    k = rms_norm(lin(w[p + "k"], h).view(T, G, d), w[p + "k.norm"], eps)
    v = lin(w[p + "v"], h).view(T, G, dv)
    if cfg.get("q_temp"):
        q = q * torch.tensor([query_temperature(t, cfg["q_temp"]["coef"], cfg["q_temp"]["every"]) for t in range(T)], dtype=F64)[:, None, None]
    out = attend(q, k, v, cfg["scale"], bias=distance_bias(w[p + "rel"], T, cfg["bias_max"]), sink=w[p + "sink"].to(F64))
    return lin(w[p + "o"], out.reshape(T, H * dv))


# ---- linear attention with a fixed decay per head ----------------------------------------------------
def decay_core(q, k, v, decay, state=None):
    """q, k [T, H, d], v [T, H, dv], decay [H] -> (o [T, H, dv], state [H, d, dv])."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = decay[:, None, None] * S + torch.einsum("hd,hv->hdv", k[t], v[t])
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def lightning(h, w, p, cfg, eps):
    """silu on queries, keys and values; all heads normed together; a gate per number."""
    T, H, d = h.shape[0], cfg["heads"], cfg["dim"]
    dv = cfg.get("vdim", d)
    q, k = (silu(lin(w[p + s], h)).view(T, H, d) for s in "qk")
    v = silu(lin(w[p + "v"], h)).view(T, H, dv)
    o, _ = decay_core(q, k, v, torch.tensor([float(x) for x in cfg["decay"]], dtype=F64))
    o = rms_norm(o.reshape(T, H * dv), w[p + "norm"], eps) * torch.sigmoid(lin(w[p + "g"], h))
    return lin(w[p + "o"], o)


# ---- the mixture -------------------------------------------------------------------------------------
def route(z, correction, top, groups, keep, scale):
    """z [n] logits of one position over experts and identity outputs -> [n] weights, zero for those not chosen."""
    n = z.shape[0]
    s = torch.softmax(z, dim=0)
    c = s + correction
    size = n // groups
    marks = [float(c[g * size: (g + 1) * size].max()) for g in range(groups)]
    kept = sorted(range(groups), key=lambda g: (-marks[g], g))[:keep]
    open_to = [e for e in range(n) if e // size in kept]
    chosen = sorted(open_to, key=lambda e: (-float(c[e]), e))[:top]
    total = sum(float(s[e]) for e in chosen) + 1e-20
    out = torch.zeros(n, dtype=F64)
    for e in chosen:
        out[e] = s[e] / total * scale
    gap = math.inf
    if keep < groups:
        gap = min(marks[g] for g in kept) - max(marks[g] for g in range(groups) if g not in kept)
    left = [float(c[e]) for e in open_to if e not in chosen]
    if left:
        gap = min(gap, min(float(c[e]) for e in chosen) - max(left))
    return out, gap


def mixture(h, w, p, cfg):
    r = cfg["router"]
    n_experts, n_identity = r["experts"], r.get("identity") or 0
    groups = r.get("groups") or {"count": 1, "keep": 1}
    correction = w[p + "correction"].to(F64)
    z = lin(w[p + "router"], h)
    weights, gaps = torch.zeros(h.shape[0], n_experts + n_identity, dtype=F64), []
    for t in range(h.shape[0]):
        weights[t], gap = route(z[t], correction, r["top"], groups["count"], groups["keep"], float(r.get("scale", 1.0)))
        gaps.append(gap)
    if MARGINS is not None:
        MARGINS.append(gaps)
    y = weights[:, n_experts:].sum(-1, keepdim=True) * h          # the identity outputs give the input back
    for e in range(n_experts):
        y = y + weights[:, e: e + 1] * lin(w[f"{p}e{e}.down"], gelu_erf(lin(w[f"{p}e{e}.up"], h)))
    return y


# ---- several streams ---------------------------------------------------------------------------------
def hyper(x, w, p, sublayer, m):
    """x [T, s, D]; u = sum_a in[a] x_a is what the sublayer reads; x_b <- sum_a mix[a, b] x_a + m out[b] y. A model that says nothing of
    streams has one, and no weights for it: x <- x + m y."""
    if p + "in" not in w:
        return x + m * sublayer(x[:, 0])[:, None, :]
    u = torch.einsum("a,tad->td", w[p + "in"].to(F64), x)
    y = sublayer(u)
    return torch.einsum("ab,tad->tbd", w[p + "mix"].to(F64), x) + m * w[p + "out"].to(F64)[None, :, None] * y[:, None, :]


def forward(config, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; `layers_out` (a list) receives the sum of the streams after every layer."""
    def read(rows):
        return DISTURB(rows) if DISTURB is not None else rows

    eps, m = config["norm"]["eps"], float(config.get("residual_mult", 1.0))
    x = w["embed"].to(F64)[torch.tensor(tokens)]
    x = x[:, None, :].repeat(1, config.get("streams") or 1, 1)
    for i, layer in enumerate(config["layers"]):
        own = layer.get("weights_of")
        p, mix = f"l{i if own is None else own}.", layer["mixer"]

        def mixer(u):
            h = read(rms_norm(u, w[p + "norm1"], eps))
            if layer["type"] == "attention":
                return window_attention(h, w, p + "mix.", mix, eps)
            return mix["left_scale"] * biased_attention(h, w, p + "mix.left.", mix["left"], eps) \
                + mix["right_scale"] * lightning(h, w, p + "mix.right.", mix["right"], eps)

        x = hyper(x, w, p + "hc1.", mixer, m)
        if layer.get("mlp") is not None:
            x = hyper(x, w, p + "hc2.", lambda u: mixture(read(rms_norm(u, w[p + "norm2"], eps)), w, p + "mlp.", layer["mlp"]), m)
        if layers_out is not None:
            layers_out.append(x.sum(1))
    return lin(w["head"], read(rms_norm(x.sum(1), w["final.norm"], eps)))


def read_model(folder):
    """(config.json as a dict, tensors by name in float64)."""
    import json
    from pathlib import Path

    from safetensors.torch import load_file

    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), {n: t.to(F64) for n, t in load_file(str(folder / "model.safetensors")).items()}


def generate(config: dict, w: dict, prompt: list[int], n_new: int) -> list[int]:
    """Greedy continuation, recomputing the whole sequence for every token (first index on ties)."""
    seq = list(prompt)
    for _ in range(n_new):
        seq.append(int(forward(config, w, seq)[-1].argmax()))
    return seq[len(prompt):]
