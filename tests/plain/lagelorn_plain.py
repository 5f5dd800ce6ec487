"""Lagelorn, stated plainly: one function per mechanism, float64, a Python loop over the positions wherever one position
depends on the ones before it. Nothing here is shared with the engine; the tests compare the engine with it.

A model is a dict of tensors by checkpoint name and the config.json dict. Notation: h [T, D] is a mixer's input, rows are
the positions 0 .. T - 1 of ONE sequence. The stream is normalised AFTER every sum: x <- norm1(alpha x + mixer(x)),
x <- norm2(alpha x + feed_forward(x)); then the token's own side input joins it: x <- x + normed(proj(gelu(gate x) * e)).
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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# A test may set this to a function that disturbs the stream's rows on their way into every sublayer (and into the head):
# how far the logits of a position move under small disturbances says how well-conditioned the position is.
DISTURB = None


# ---- attention by chunks -------------------------------------------------------------------------
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


def softmax_with_sink(s, sink):
    """s [H, J] -> weights [H, J] whose denominator also holds exp(sink[h]), a term without key or value."""
    top = torch.maximum(s.max(dim=-1).values, sink)
    e = torch.exp(s - top[:, None])
    return e / (e.sum(dim=-1) + torch.exp(sink - top))[:, None]


def chunk_attention_core(q, k, v, scale, bias, sink, chunk, positions=None):
    """q [T, H, d] (already normed), k [J, G, d], v [J, G, dv] of one sequence; positions[t] is row t's place (default t). Row at
    position i sees the keys of its own chunk up to i. bias [H, >= J] by distance; sink [H]. chunk 0: one chunk."""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    k_of, v_of = k.repeat_interleave(per, dim=1), v.repeat_interleave(per, dim=1)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        i = t if positions is None else positions[t]
        j0 = i // chunk * chunk if chunk else 0
        s = torch.einsum("hd,jhd->hj", q[t], k_of[j0: i + 1]) * scale
        s = s + bias[:, : i - j0 + 1].flip(-1)        # key j stands i - j back
        out[t] = torch.einsum("hj,jhv->hv", softmax_with_sink(s, sink), v_of[j0: i + 1])
    return out


def chunk_attention(h, w, p, cfg, eps):
    T = h.shape[0]
    H, d = cfg["heads"], cfg["dim"]
    G = cfg.get("kv_heads", H)
    q = rms_norm(lin(w[p + "q"], h, w[p + "q.b"]), w[p + "q.norm"], eps).view(T, H, d)      # one norm over all heads
    k_raw = lin(w[p + "k"], h, w[p + "k.b"])
    k = rms_norm(k_raw, w[p + "k.norm"], eps).view(T, G, d)
    chunk = (cfg.get("mask") or {}).get("size", 0)
    out = chunk_attention_core(q, k, k_raw.view(T, G, d), cfg["scale"], distance_bias(w[p + "rel"], T, cfg["bias_max"]),
                               w[p + "sink"].to(F64), chunk)
    return lin(w[p + "o"], out.reshape(T, H * d))


# ---- the gated delta rule --------------------------------------------------------------------------
def short_conv(x, taps):
    """x [T, C], taps [C, n], the last column the current row's -> silu of the causal convolution."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=F64), x])
    return silu(sum(padded[i: i + x.shape[0]] * taps[:, i].to(F64) for i in range(n)))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_core(q, k, v, g, beta, state=None):
    """q, k [T, H, d], v [T, H, dv], g, beta [T, H] -> (o [T, H, dv], state [H, d, dv])."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + torch.einsum("hd,hv->hdv", k[t], u)
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out, S


def delta(h, w, p, cfg, eps):
    T = h.shape[0]
    H, d = cfg["heads"], cfg["dim"]
    G, dv = cfg.get("kv_heads", H), cfg.get("vdim", d)
    per = H // G
    q = unit(short_conv(lin(w[p + "q"], h), w[p + "q.conv"]).view(T, G, d)) * d ** -0.5
    k = unit(short_conv(lin(w[p + "k"], h), w[p + "k.conv"]).view(T, G, d))
    v = short_conv(lin(w[p + "v"], h), w[p + "v.conv"]).view(T, H, dv)
    beta = torch.sigmoid(lin(w[p + "b"], h))
    g = torch.exp(-torch.exp(w[p + "A_log"].to(F64)) * torch.nn.functional.softplus(lin(w[p + "a"], h) + w[p + "dt_bias"].to(F64)))
    o, _ = delta_core(q.repeat_interleave(per, dim=1), k.repeat_interleave(per, dim=1), v, g, beta)
    o = rms_norm(o, w[p + "norm"], eps).reshape(T, H * dv)
    return lin(w[p + "o"], o * silu(lin(w[p + "g"], h)))


# ---- time mixing with a decay per channel ------------------------------------------------------------
def shifted(h):
    """The row before each row; zeros before the first."""
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def time_mix_core(r, k, v, decay, bonus, state=None):
    """r, k, decay [T, H, d], v [T, H, d], bonus [H, d] -> (o [T, H, d], state [H, d, d])."""
    T, H, d = r.shape
    S = torch.zeros(H, d, d, dtype=F64) if state is None else state.clone()
    out = torch.zeros(T, H, d, dtype=F64)
    for t in range(T):
        write = torch.einsum("hi,hj->hij", k[t], v[t])
        out[t] = torch.einsum("hij,hi->hj", S + bonus[:, :, None] * write, r[t])
        S = decay[t][:, :, None] * S + write
    return out, S


def time_mix(h, w, p, cfg, eps):
    T, H, d = h.shape[0], cfg["heads"], cfg["dim"]
    prev = shifted(h)
    mix = {s: h + (prev - h) * w[f"{p}mu.{s}"].to(F64) for s in "rkvgw"}
    r, k, v = (lin(w[p + s], mix[s]).view(T, H, d) for s in "rkv")
    decay = torch.exp(-torch.exp(lin(w[p + "w2"], torch.tanh(lin(w[p + "w1"], mix["w"]))) + w[p + "w0"].to(F64))).view(T, H, d)
    o, _ = time_mix_core(r, k, v, decay, w[p + "u"].to(F64))
    o = unit_rms(o, eps).reshape(T, H * d) * w[p + "norm"].to(F64)
    return lin(w[p + "o"], o * silu(lin(w[p + "g"], mix["g"])))


# ---- the rest of a layer -----------------------------------------------------------------------------
def feed_forward(h, w, p):
    inner = gelu_tanh(lin(w[p + "gate"], h, w[p + "gate.b"])) * lin(w[p + "up"], h, w[p + "up.b"])
    return lin(w[p + "down"], inner, w[p + "down.b"])


def side_input(x, e, w, p, eps):
    """e [T, dim]: the tokens' own rows for this layer -> what joins the stream."""
    g = gelu_tanh(lin(w[p + "gate"], x)) * e
    return rms_norm(lin(w[p + "proj"], g), w[p + "norm"], eps)


def forward(config, w, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; `layers_out` (a list) receives the stream after every layer."""
    def read(rows):
        return DISTURB(rows) if DISTURB is not None else rows

    eps, alpha = config["norm"]["eps"], float(config.get("postln_alpha", 1.0))
    ids = torch.tensor(tokens)
    x = w["embed"].to(F64)[ids] + w["pos"].to(F64)[: len(tokens)]
    side = config.get("token_side")
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = read(x)
        if layer["type"] == "delta":
            y = delta(h, w, p + "mix.", m, eps)
        else:
            y = m["left_scale"] * chunk_attention(h, w, p + "mix.left.", m["left"], eps) \
                + m["right_scale"] * time_mix(h, w, p + "mix.right.", m["right"], eps)
        x = rms_norm(alpha * x + y, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = rms_norm(alpha * x + feed_forward(read(x), w, p + "mlp."), w[p + "norm2"], eps)
        if side:
            n = side["dim"]
            x = x + side_input(read(x), w["side.embed"].to(F64)[ids, i * n: (i + 1) * n], w, p + "side.", eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    logits = lin(w["head"], read(rms_norm(x, w["final.norm"], eps)))
    cap = config.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits


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
