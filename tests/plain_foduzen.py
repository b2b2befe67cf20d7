"""A plain, slow implementation of the Foduzen decoder in dense 64-bit torch operations over whole sequences: one
function per mechanism, each written from the mechanism's equations (stated in its docstring) and sharing no code
with the package.

The design: x = embed[token] * embedding.scale + a sinusoidal vector of the position.  A layer normalises what its
sublayers give, never what they read: x <- x + g1 rms(mixer(x)), then x <- x + g2 rms(feed_forward(x)), g1 and g2
single numbers.  The mixer is a gated linear recurrent unit behind a short convolution (`rglru`), or windowed softmax
attention with an output gate beside a Mamba-2 recurrence (`parallel`), each side normed and half their sum taken.  The
feed-forward is dense with the xIELU activation, or absent.  logits = head (g rms(x))."""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def gelu_tanh(z):
    """z/2 (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))."""
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    """log(1 + e^z), for every z without overflow."""
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def position_vectors(positions, width):
    """[T, width]: column c holds, with i = c // 2, sin(p 10000^(-2i/width)) for even c and the cosine for odd c."""
    out = torch.zeros(len(positions), width, dtype=F64)
    for c in range(width):
        angle = positions.to(F64) * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.sin(angle) if c % 2 == 0 else torch.cos(angle)
    return out


def embedding(tokens, positions, table, scale):
    """table[token] * scale + the position's vector."""
    return table.to(F64)[tokens] * scale + position_vectors(positions, table.shape[1])


def causal_conv(x, taps, bias):
    """y_t[c] = bias[c] + sum_j taps[c, j] x_(t - n + 1 + j)[c], n taps, zeros before the first token."""
    T, n = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=F64), x])
    y = bias.to(F64)[None, :].repeat(T, 1)
    for j in range(n):
        y = y + taps[:, j].to(F64)[None, :] * padded[j:j + T]
    return y


def block_linear(u, matrices, bias):
    """u [T, blocks * s] in `blocks` parts, part b through the square matrix b [out, in], plus bias [blocks, s]."""
    blocks, size = matrices.shape[0], matrices.shape[1]
    parts = u.view(u.shape[0], blocks, size)
    return (torch.einsum("tbi,boi->tbo", parts, matrices.to(F64)) + bias.to(F64)[None]).reshape(u.shape[0], -1)


def gated_recurrence(u, r, i, lam, state=None):
    """log a = -8 r softplus(lam), a = e^(log a);  S_t = a S_(t-1) + sqrt(1 - a^2) i u per channel, S before the first
    token zero or `state`.  Returns (S of every token, the last S)."""
    log_a = -8.0 * r * softplus(lam.to(F64))[None, :]
    a, inflow = torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a)) * i * u
    S = torch.zeros(u.shape[1], dtype=F64) if state is None else state.to(F64).clone()
    out = torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + inflow[t]
        out[t] = S
    return out, S


def rglru(h, w):
    """y = gelu(W_y h + b), u = conv(W_x h + b); in every block r = sigmoid(ra u + b), i = sigmoid(ri u + b); the gated
    recurrence over u; W_o (S * y)."""
    y = gelu_tanh(h @ w["y"].to(F64).T + w["y.b"].to(F64))
    u = causal_conv(h @ w["x"].to(F64).T + w["x.b"].to(F64), w["conv"], w["conv.b"])
    r = torch.sigmoid(block_linear(u, w["ra"], w["ra.b"]))
    i = torch.sigmoid(block_linear(u, w["ri"], w["ri.b"]))
    S, _ = gated_recurrence(u, r, i, w["lam"])
    return (S * y) @ w["o"].to(F64).T


def window_mask(positions, size):
    """[T, T] True where key j is visible to query i: 0 <= p_i - p_j < size (size None: every j <= i)."""
    delta = positions[:, None] - positions[None, :]
    visible = delta >= 0
    if size is not None:
        visible &= delta < int(size)
    return visible


def gated_attention(h, positions, w, m, eps):
    """q = W_q h + b, k = W_k h + b, v = W_v h + b; every q head and every k head over its root mean square, times a
    weight of the head's size for all heads; no rotation.  Query head a reads key/value head a // (H / G); softmax of
    scale * (q . k) over the window; the heads side by side times sigmoid(W_g h); W_o and its bias."""
    H, d = m["heads"], m["dim"]
    G, dv = m.get("kv_heads", H), m.get("vdim", d)
    T = h.shape[0]
    q = (h @ w["q"].to(F64).T + w["q.b"].to(F64)).view(T, H, d)
    k = (h @ w["k"].to(F64).T + w["k.b"].to(F64)).view(T, G, d)
    v = (h @ w["v"].to(F64).T + w["v.b"].to(F64)).view(T, G, dv)
    q, k = rms(q, eps) * w["q.norm"].to(F64), rms(k, eps) * w["k.norm"].to(F64)
    visible = window_mask(positions, (m.get("mask") or {}).get("size"))
    out = torch.zeros(T, H, dv, dtype=F64)
    for a in range(H):
        g = a // (H // G)
        scores = (q[:, a] @ k[:, g].T) * float(m["scale"])
        out[:, a] = torch.softmax(scores.masked_fill(~visible, float("-inf")), dim=-1) @ v[:, g]
    gated = out.reshape(T, H * dv) * torch.sigmoid(h @ w["g"].to(F64).T)
    return gated @ w["o"].to(F64).T + w["o.b"].to(F64)


def head_recurrence(x, B, C, dt, A_log, D, state=None):
    """x [T, heads, P], B and C [T, groups, N], dt [T, heads] (positive).  Head h reads group h // (heads / groups):
    S_t = exp(-exp(A_log_h) dt) S_(t-1) + dt B_t x_t^T  (N x P),  y_t = S_t^T C_t + D_h x_t.  Returns (y, last S)."""
    T, heads, P = x.shape
    groups, N = B.shape[1], B.shape[2]
    of = torch.arange(heads) // (heads // groups)
    S = torch.zeros(heads, N, P, dtype=F64) if state is None else state.to(F64).clone()
    y = torch.zeros(T, heads, P, dtype=F64)
    rate = -torch.exp(A_log.to(F64))
    for t in range(T):
        decay = torch.exp(rate * dt[t])[:, None, None]
        S = decay * S + dt[t][:, None, None] * B[t, of][:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnp,hn->hp", S, C[t, of]) + D.to(F64)[:, None] * x[t]
    return y, S


def grouped_gated_norm(y, z, weight, groups, eps):
    """y * silu(z), cut into `groups` equal parts, each over its own root mean square, times weight."""
    v = (y * silu(z)).view(y.shape[0], groups, -1)
    return rms(v, eps).reshape(y.shape[0], -1) * weight.to(F64)


def mamba2(h, w, m, eps):
    """[z | x | B | C | dt] = W_in h; x, B and C through the convolution and SiLU; dt <- softplus(dt + dt_bias); the
    heads' recurrence; the gated norm in groups; W_o."""
    heads, P, N, G = m["heads"], m["vdim"], m["state"], m.get("groups", 1)
    inner, T = heads * P, h.shape[0]
    rows = h @ w["in"].to(F64).T
    z, xbc, dt = rows[:, :inner], rows[:, inner:2 * inner + 2 * G * N], rows[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    dt = softplus(dt + w["dt_bias"].to(F64))
    x = xbc[:, :inner].reshape(T, heads, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    y, _ = head_recurrence(x, B, C, dt, w["A_log"], w["D"])
    y = grouped_gated_norm(y.reshape(T, inner), z, w["norm"], m.get("norm_groups", 1), eps)
    return y @ w["o"].to(F64).T


def _under(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def parallel(h, positions, w, m, eps):
    """(rms(attention(h)) * left.out + rms(mamba2(h)) * right.out) / 2."""
    left = gated_attention(h, positions, _under(w, "left."), m["left"], eps)
    right = mamba2(h, _under(w, "right."), m["right"], eps)
    return 0.5 * (rms(left, eps) * w["left.out"].to(F64) + rms(right, eps) * w["right.out"].to(F64))


def xielu(z, p, q):
    """z > 0: softplus(p) z^2 + z/2;  z <= 0: (1/2 + softplus(q)) (e^z - 1 - z) + z/2."""
    low = torch.clamp(z, max=0.0)
    return torch.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (torch.expm1(low) - low)) + 0.5 * z


def dense_mlp(h, w):
    """down xielu(up h) with the two numbers of `act`."""
    act = w["act"].to(F64)
    return xielu(h @ w["up"].to(F64).T, act[0], act[1]) @ w["down"].to(F64).T


def forward(config: dict, tensors: dict, tokens, layer_outputs=None):
    """Logits [T, vocab] (64-bit) of one sequence from position 0.  `layer_outputs`: a list that receives the residual
    stream after every layer."""
    eps = float(config["norm"]["eps"])
    positions = torch.arange(len(tokens))
    x = embedding(torch.tensor(list(tokens), dtype=torch.long), positions, tensors["embed"], float((config.get("embedding") or {}).get("scale", 1.0)))
    for n, layer in enumerate(config["layers"]):
        w = _under(tensors, f"l{n}.")
        mixer = _under(w, "mix.")
        y = rglru(x, mixer) if layer["type"] == "rglru" else parallel(x, positions, mixer, layer["mixer"], eps)
        x = x + rms(y, eps) * w["norm1"].to(F64)
        if layer.get("mlp"):
            x = x + rms(dense_mlp(x, _under(w, "mlp.")), eps) * w["norm2"].to(F64)
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return (rms(x, eps) * tensors["final.norm"].to(F64)) @ tensors["head"].to(F64).T


def greedy(config, weights, prompt, count):
    """`count` tokens after `prompt`, each the largest logit's id (the largest id among equals)."""
    tokens, out = list(prompt), []
    for _ in range(count):
        row = forward(config, weights, tokens)[-1]
        best = row.max()
        token = max(i for i in range(len(row)) if row[i] == best)
        out.append(token)
        tokens.append(token)
    return out
