"""A plain, slow implementation of the Botuvik decoder in dense 64-bit torch operations over whole sequences: one
function per mechanism, each written from the mechanism's equations (stated in its docstring) and sharing no code
with the package.

The design: x = embed[token].  Every layer does x <- x + N1b(mixer(N1(x))) and, where it has a feed-forward,
x <- x + N2b(ff(N2(x))), N(.) an RMS norm with a plain weight.  The mixer is grouped-query softmax attention (biases,
interleaved rotation, a weightless norm per head behind it, a tanh cap on the scores, a learned sink per head) or the
matrix memory of xLSTM (`mlstm`).  The feed-forward is a dense squared ReLU, a mixture of gated SiLU experts (sigmoid
scores, groups judged by their two largest, a shared expert), or absent.  A run of layers may be gone through several
times: the embedding output comes in again ahead of every pass but the first, and a stored vector ahead of every pass.
logits = head N(x)."""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis, eps inside the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rotate_interleaved(x, positions, base, dims):
    """x [T, heads, d]: for i < dims/2 the pair (u, v) = (x[2i], x[2i+1]) at position p becomes
    (u cos a - v sin a, v cos a + u sin a), a = p base^(-2i/dims); elements from dims on pass unchanged."""
    freq = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    angle = positions.to(F64)[:, None] * freq[None, :]
    c, s = torch.cos(angle)[:, None, :], torch.sin(angle)[:, None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def attend(q, k, v, scale, cap, sink):
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head a reads head a // (H / G).  s = scale q.k, then cap tanh(s / cap)
    (cap None: s itself); token i weighs every j <= i with exp(s_ij) / (exp(sink_a) + sum_j exp(s_ij)) (sink None: without
    that term).  Returns [T, H, dv]."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    k, v = k.repeat_interleave(group, dim=1), v.repeat_interleave(group, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * float(scale)
    if cap:
        s = float(cap) * torch.tanh(s / float(cap))
    s = s.masked_fill(torch.arange(T)[None, :] > torch.arange(T)[:, None], -math.inf)
    top = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        sink = sink.to(F64)[:, None, None]
        top = torch.maximum(top, sink)
    e = torch.exp(s - top)
    total = e.sum(dim=-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink - top)
    return torch.einsum("hij,jhd->ihd", e / total, v)


def attention(h, positions, w, m, eps):
    """q, k, v = W h + b; q and k turned in interleaved pairs over their first rot.dims elements, then each head of q and
    of k over its root mean square (no weight); `attend`; the heads side by side through W_o."""
    T, H, d = h.shape[0], m["heads"], m["dim"]
    G, dv = m.get("kv_heads", H), m.get("vdim", d)
    q = (h @ w["q"].to(F64).T + w["q.b"].to(F64)).view(T, H, d)
    k = (h @ w["k"].to(F64).T + w["k.b"].to(F64)).view(T, G, d)
    v = (h @ w["v"].to(F64).T + w["v.b"].to(F64)).view(T, G, dv)
    if m.get("rot") and m["rot"]["dims"]:
        q = rotate_interleaved(q, positions, m["rot"]["base"], m["rot"]["dims"])
        k = rotate_interleaved(k, positions, m["rot"]["base"], m["rot"]["dims"])
    o = attend(rms(q, eps), rms(k, eps), v, m["scale"], m.get("softcap"), w["sink"])
    return o.reshape(T, H * dv) @ w["o"].to(F64).T


def mlstm_recurrence(q, k, v, i, f, state=None, fragile=None):
    """q, k [T, H, d], v [T, H, dv], log gates i, f [T, H].  With S [H, d, dv], n [H, d] and m [H] (all zero at the start, or
    `state`): m_t = max(f_t + m_(t-1), i_t), S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T, n_t the same
    with k_t alone, o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6).  Returns (o [T, H, dv], (S, n, m)).  `fragile` [T]:
    marked where a head's query lies almost across everything its memory holds, so that S_t^T q_t is what rounding leaves of it
    (the norm behind it raises that to full size)."""
    T, H, d = q.shape
    S, n, m = (torch.zeros(H, d, v.shape[2], dtype=F64), torch.zeros(H, d, dtype=F64), torch.zeros(H, dtype=F64)) \
        if state is None else tuple(t.clone() for t in state)
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        m = new
        below = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        read = torch.einsum("hdv,hd->hv", S, q[t])
        if fragile is not None:
            most = S.flatten(1).norm(dim=1) * q[t].norm(dim=1)
            fragile[t] |= bool((read.norm(dim=1) < 3e-2 * most).any())
        out[t] = read / below[:, None]
    return out, (S, n, m)


def mlstm(h, w, m, eps, state=None, fragile=None):
    """q = W_q h dim^(-1/2), k = W_k h, v = W_v h; log gates i = cap tanh((W_i h + b_i) / cap) and
    f = log sigmoid(cap tanh((W_f h + b_f) / cap)); `mlstm_recurrence`; each head's o over its root mean square; heads side
    by side times a weight, times sigmoid(W_g h), through W_o.  Returns (output, the state behind the last token)."""
    T, H, d, dv, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    q = (h @ w["q"].to(F64).T).view(T, H, d) * d ** -0.5
    k = (h @ w["k"].to(F64).T).view(T, H, d)
    v = (h @ w["v"].to(F64).T).view(T, H, dv)
    i = cap * torch.tanh((h @ w["i"].to(F64).T + w["i.b"].to(F64)) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w["f"].to(F64).T + w["f.b"].to(F64)) / cap))
    o, state = mlstm_recurrence(q, k, v, i, f, state, fragile)
    y = rms(o, eps).reshape(T, H * dv) * w["norm"].to(F64) * torch.sigmoid(h @ w["g"].to(F64).T)
    return y @ w["o"].to(F64).T, state


def squared_relu_mlp(h, up, down):
    """down relu(up h)^2."""
    return (torch.relu(h @ up.to(F64).T) ** 2) @ down.to(F64).T


def gated_silu_mlp(h, gate, up, down):
    """down (silu(gate h) * (up h)), silu(z) = z sigmoid(z)."""
    z = h @ gate.to(F64).T
    return (z * torch.sigmoid(z) * (h @ up.to(F64).T)) @ down.to(F64).T


def route(h, w, router, fragile=None):
    """s = sigmoid(W_router h).  The experts form groups.count groups of neighbours; a group's score is the sum of its two
    largest s (of its only one where a group is one expert); experts outside the groups.keep best groups are out.  The `top`
    largest s are chosen; weights: the chosen s over their sum (+ 1e-20).  Returns (indices [T, top], weights [T, top]).
    `fragile` [T]: marked where a choice is close enough for 16-bit rounding to turn it."""
    s = torch.sigmoid(h @ w["router"].to(F64).T)
    total, top = s.shape[1], int(router["top"])
    c, groups = s.clone(), router.get("groups")
    if groups and int(groups["count"]) > 1:
        count, keep = int(groups["count"]), int(groups["keep"])
        size = total // count
        judged = torch.topk(c.view(-1, count, size), min(2, size), dim=-1).values.sum(-1)
        kept = torch.topk(judged, keep, dim=-1).indices
        allowed = torch.zeros_like(judged, dtype=torch.bool).scatter_(1, kept, True)
        c = c.masked_fill(~allowed.repeat_interleave(size, dim=1), -math.inf)
        if fragile is not None and keep < count:
            ranked = torch.sort(judged, dim=-1, descending=True).values
            fragile |= (ranked[:, keep - 1] - ranked[:, keep]) < 2.5e-2
    chosen = torch.topk(c, top, dim=-1).indices
    if fragile is not None and top < total:
        ranked = torch.sort(c, dim=-1, descending=True).values
        fragile |= (ranked[:, top - 1] - ranked[:, top]) < 1.5e-2
    picked = torch.gather(s, 1, chosen)
    return chosen, picked / (picked.sum(dim=-1, keepdim=True) + 1e-20)


def expert_mixture(h, w, mlp, fragile=None):
    """sum over the chosen e of weight_e * expert_e(h), each a `gated_silu_mlp`, plus shared(h) where there is a shared
    expert of the same form."""
    chosen, weights = route(h, w, mlp["router"], fragile)
    out = torch.zeros(h.shape[0], h.shape[1], dtype=F64)
    for t in range(h.shape[0]):
        for weight, e in zip(weights[t], chosen[t]):
            e = f"e{int(e)}."
            out[t] += weight * gated_silu_mlp(h[t:t + 1], w[e + "gate"], w[e + "up"], w[e + "down"])[0]
    if mlp.get("shared"):
        out = out + gated_silu_mlp(h, w["shared.gate"], w["shared.up"], w["shared.down"])
    return out


def layer_order(config):
    """[(layer, pass, whether it is the first layer of its pass)] in the order in which layers run; pass None outside the
    repeated run."""
    loop, order = config.get("loop"), []
    n = len(config["layers"])
    if not loop:
        return [(i, None, False) for i in range(n)]
    for i in range(loop["start"]):
        order.append((i, None, False))
    for t in range(loop["times"]):
        for i in range(loop["start"], loop["stop"]):
            order.append((i, t, i == loop["start"]))
    return order + [(i, None, False) for i in range(loop["stop"], n)]


def forward(config: dict, tensors: dict, tokens, layer_outputs=None, fragile=None):
    """Logits [T, vocab] (64-bit) of one sequence from position 0.  `layer_outputs`: a list that receives the residual
    stream after every layer run.  `fragile`: a boolean tensor [T] in which the rows are marked whose result rests on a
    router's close call that 16-bit rounding may turn, or on what rounding leaves of a memory's answer."""
    eps = float(config["norm"]["eps"])
    positions = torch.arange(len(tokens))
    norm = lambda x, name: rms(x, eps) * tensors[name].to(F64)
    first = tensors["embed"].to(F64)[torch.tensor(list(tokens), dtype=torch.long)]
    x = first
    for i, t, opens in layer_order(config):
        if opens:
            if t > 0:
                x = x + first
            x = x + tensors["loop.step"][t].to(F64)
        layer, p = config["layers"][i], f"l{i}."
        w = {k[len(p) + 4:]: v for k, v in tensors.items() if k.startswith(p + "mix.")}
        h = norm(x, p + "norm1")
        if layer["type"] == "attention":
            y = attention(h, positions, w, layer["mixer"], eps)
        else:
            y = mlstm(h, w, layer["mixer"], eps, fragile=fragile)[0]
        x = x + norm(y, p + "norm1b")
        mlp = layer.get("mlp")
        if mlp:
            w = {k[len(p) + 4:]: v for k, v in tensors.items() if k.startswith(p + "mlp.")}
            h = norm(x, p + "norm2")
            y = squared_relu_mlp(h, w["up"], w["down"]) if mlp["kind"] == "dense" else expert_mixture(h, w, mlp, fragile)
            x = x + norm(y, p + "norm2b")
        if layer_outputs is not None:
            layer_outputs.append(x.clone())
    return norm(x, "final.norm") @ tensors["head"].to(F64).T


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
