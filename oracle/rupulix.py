"""CPU oracle for the Rupulix decoder -- TEST INFRASTRUCTURE ONLY (plain, slow, one function per mechanism).

Rupulix is a decoder-only model whose layer list comes from config.json.  The residual is `streams` parallel copies of the stream
x_1 .. x_n, all the embedding row at the start.  Around sublayer q of a layer (1: mixer, 2: feed-forward), with small learned tables
a (in), b (out), M (mix, [from, to]):

  y = sublayer(rms(sum_s a_s x_s) w);   x_t <- sum_s M[s, t] x_s + b_t y      (all streams at once);   head: E (rms(sum_s x_s) w) * logit_scale

Notation (weights W are [out, in], applied as W x):
  rms(y)        = y / sqrt(mean(y^2) + eps)
  rotation      : dimensions are turned in pairs by pos * base^(-2i / dims); pairs (2i, 2i + 1), or (i, i + dims / 2)
  latent        : c | k_r = W_dkv h, c <- rms(c) w;  per head  q_u | q_r = (W_q h)_head, score = (q_u . U_k c + rot(q_r) . rot(k_r)) scale,
                  over the last `size` tokens, exp(sink) in the denominator;  W_o of the heads' U_v c sums
  parallel      : left_scale * left + right_scale * right
    left        : q, k = rot(rms(per head) w), scores of all heads mixed by T[to, from] ahead of the softmax; W_o
    right       : y = gelu_tanh(W_y h + b), u = conv(W_x h + b) + b;  per equal part of u: r, i = sigmoid(R u + b), sigmoid(I u + b);
                  log a = -8 r softplus(lam);  S <- a S + sqrt(1 - a^2) i u;  W_o (S * y)
  feed-forward  : W_down relu(W_up h)^2

A span of the layer list may run several times in a row with the same weights; every run has its own cache and state.
Everything runs in the dtype of the weights handed in (float64 in the tests), whole prompts or token by token; `State` makes the
two forms comparable.
"""
from __future__ import annotations

import math

import numpy as np
import torch


# ---------------------------------------------------------------------------------------------- mechanisms
def rms(y, eps):
    return y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def rotate(x, pos, dims, base, halves):
    """x [S, heads, d]: the first `dims` dimensions turn in pairs, the rest pass."""
    out = x.clone()
    for i in range(dims // 2):
        a, b = (i, i + dims // 2) if halves else (2 * i, 2 * i + 1)
        ang = pos.to(x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        out[:, :, a] = x[:, :, a] * c - x[:, :, b] * s
        out[:, :, b] = x[:, :, b] * c + x[:, :, a] * s
    return out


def visible(pos, size):
    """Positions that a token at `pos` sees: itself and the size - 1 before it (size 0: all before it)."""
    return torch.arange(max(0, pos - size + 1) if size else 0, pos + 1)


def softmax_with_sink(s, sink=None):
    """s [heads, keys]; sink [heads]: one more term in the denominator."""
    m = s.max(-1, keepdim=True).values
    if sink is not None:
        m = torch.maximum(m, sink[:, None])
    e = torch.exp(s - m)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink[:, None] - m)
    return e / den


def causal_conv(u, w, b, before):
    """u [S, C] the new inputs, before [taps - 1, C] the ones ahead of them (zeros at the start), w [C, taps]: its last column weighs
    the current token.  -> (outputs, the new `before`)."""
    taps = w.shape[1]
    full = torch.cat([before, u])
    y = torch.zeros_like(u)
    for j in range(taps):
        y = y + full[j:j + u.shape[0]] * w[:, j]
    return y + b, full[full.shape[0] - (taps - 1):]


def block_linear(u, w, b):
    """u [S, C] in equal parts, w [parts, n, n] ([out, in]), b [parts, n]."""
    parts, n = b.shape
    return torch.cat([u[:, k * n:(k + 1) * n] @ w[k].T + b[k] for k in range(parts)], 1)


def linear_recurrence(log_a, gated, S):
    """S <- a S + sqrt(1 - a^2) * gated, token by token."""
    out = []
    for t in range(log_a.shape[0]):
        a = torch.exp(log_a[t])
        S = a * S + torch.sqrt(-torch.expm1(2.0 * log_a[t])) * gated[t]
        out.append(S)
    return torch.stack(out), S


def stream_in(xs, a):
    """xs [streams, S, W]"""
    return (a[:, None, None] * xs).sum(0)


def stream_out(xs, M, b, y):
    n = xs.shape[0]
    return torch.stack([sum(M[s, t] * xs[s] for s in range(n)) + b[t] * y for t in range(n)])


def feed_forward(h, p, pre):
    return torch.relu(h @ p[pre + "up"].T).pow(2) @ p[pre + "down"].T


# ---------------------------------------------------------------------------------------------- state and mixers
class State:
    """What every run of a layer carries from token to token: cached rows, windows, recurrent states."""

    def __init__(self, config):
        self.len = 0
        n = len(run_order(config))
        self.rows = [{} for _ in range(n)]
        self.win = [None] * n
        self.mem = [None] * n

    def extend(self, ri, name, new):
        old = self.rows[ri].get(name)
        self.rows[ri][name] = new if old is None else torch.cat([old, new])
        return self.rows[ri][name]


def run_order(config):
    n = len(config["layers"])
    lp = config.get("loop")
    if not lp:
        return list(range(n))
    a, b = lp["start"], lp["stop"]
    return list(range(a)) + list(range(a, b)) * lp["times"] + list(range(b, n))


def latent_attention(h, pos, p, pre, m, eps, state, ri):
    H, du, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot, size = m["rot"], (m.get("mask") or {}).get("size", 0)
    S = h.shape[0]
    q = (h @ p[pre + "q"].T).reshape(S, H, du + dr)
    qu, qr = q[:, :, :du], rotate(q[:, :, du:], pos, rot["dims"], rot["base"], False)
    low = h @ p[pre + "dkv"].T
    c = state.extend(ri, "c", rms(low[:, :r], eps) * p[pre + "dkv.norm"])
    kr = state.extend(ri, "kr", rotate(low[:, None, r:], pos, rot["dims"], rot["base"], False)[:, 0])
    k = (c @ p[pre + "uk"].T).reshape(-1, H, du)
    v = (c @ p[pre + "uv"].T).reshape(-1, H, dv)
    out = torch.zeros(S, H, dv, dtype=h.dtype)
    for t in range(S):
        see = visible(int(pos[t]), size)
        s = (torch.einsum("hd,jhd->hj", qu[t], k[see]) + qr[t] @ kr[see].T) * m["scale"]
        out[t] = torch.einsum("hj,jhd->hd", softmax_with_sink(s, p[pre + "sink"]), v[see])
    return out.reshape(S, H * dv) @ p[pre + "o"].T


def talking_attention(h, pos, p, pre, m, eps, state, ri):
    H, G, d, dv, rot = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    S = h.shape[0]
    q = rms((h @ p[pre + "q"].T).reshape(S, H, d), eps) * p[pre + "q.norm"]
    k = rms((h @ p[pre + "k"].T).reshape(S, G, d), eps) * p[pre + "k.norm"]
    q = rotate(q, pos, rot["dims"], rot["base"], True)
    k = state.extend(ri, "k", rotate(k, pos, rot["dims"], rot["base"], True))
    v = state.extend(ri, "v", (h @ p[pre + "v"].T).reshape(S, G, dv))
    out = torch.zeros(S, H, dv, dtype=h.dtype)
    kv_of = torch.arange(H) // (H // G)
    for t in range(S):
        see = visible(int(pos[t]), 0)
        s = torch.einsum("hd,jhd->hj", q[t], k[see][:, kv_of]) * m["scale"]
        out[t] = torch.einsum("hj,jhd->hd", softmax_with_sink(p[pre + "talk"] @ s), v[see][:, kv_of])
    return out.reshape(S, H * dv) @ p[pre + "o"].T


def recurrent_block(h, p, pre, m, state, ri):
    C, taps = m["width"], m["conv"]
    if state.win[ri] is None:
        state.win[ri] = torch.zeros(taps - 1, C, dtype=h.dtype)
        state.mem[ri] = torch.zeros(C, dtype=h.dtype)
    y = gelu_tanh(h @ p[pre + "y"].T + p[pre + "y.b"])
    u, state.win[ri] = causal_conv(h @ p[pre + "x"].T + p[pre + "x.b"], p[pre + "conv"], p[pre + "conv.b"], state.win[ri])
    r = torch.sigmoid(block_linear(u, p[pre + "ra"], p[pre + "ra.b"]))
    i = torch.sigmoid(block_linear(u, p[pre + "ri"], p[pre + "ri.b"]))
    mem, state.mem[ri] = linear_recurrence(-8.0 * r * softplus(p[pre + "lam"]), i * u, state.mem[ri])
    return (mem * y) @ p[pre + "o"].T


def forward(config, p, tokens, state=None, trace=None):
    """tokens: the next tokens of one sequence -> logits [S, vocab].  `p`: name -> tensor.  `trace`, a list, receives the sum of
    the streams after every run of a layer."""
    state = state or State(config)
    eps = config["norm"]["eps"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    pos = torch.arange(state.len, state.len + ids.numel())
    xs = torch.stack([p["embed"][ids]] * config["streams"])
    for ri, li in enumerate(run_order(config)):
        lc, pre = config["layers"][li], f"l{li}."
        m = lc["mixer"]
        h = rms(stream_in(xs, p[pre + "hc1.in"]), eps) * p[pre + "norm1"]
        if lc["type"] == "latent_attention":
            y = latent_attention(h, pos, p, pre + "mix.", m, eps, state, ri)
        elif lc["type"] == "parallel":
            y = m["left_scale"] * talking_attention(h, pos, p, pre + "mix.left.", m["left"], eps, state, ri) \
                + m["right_scale"] * recurrent_block(h, p, pre + "mix.right.", m["right"], state, ri)
        else:
            raise ValueError(lc["type"])
        xs = stream_out(xs, p[pre + "hc1.mix"], p[pre + "hc1.out"], y)
        if lc.get("mlp"):
            h = rms(stream_in(xs, p[pre + "hc2.in"]), eps) * p[pre + "norm2"]
            xs = stream_out(xs, p[pre + "hc2.mix"], p[pre + "hc2.out"], feed_forward(h, p, pre + "mlp."))
        if trace is not None:
            trace.append(xs.sum(0))
    state.len += ids.numel()
    return (rms(xs.sum(0), eps) * p["final.norm"]) @ p["embed"].T * config["logit_scale"]


# ---------------------------------------------------------------------------------------------- random models for tests
def tensor_shapes(config):
    W, n = config["width"], config["streams"]
    out = {"embed": (config["vocab"], W), "final.norm": (W,)}
    for i, lc in enumerate(config["layers"]):
        m, pre = lc["mixer"], f"l{i}."
        for q in (1, 2) if lc.get("mlp") else (1,):
            out.update({f"{pre}norm{q}": (W,), f"{pre}hc{q}.in": (n,), f"{pre}hc{q}.out": (n,), f"{pre}hc{q}.mix": (n, n)})
        if lc["type"] == "latent_attention":
            H, d, dv, r, dr = m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["rot_dim"]
            M = pre + "mix."
            out.update({M + "q": (H * (d + dr), W), M + "dkv": (r + dr, W), M + "dkv.norm": (r,), M + "uk": (H * d, r), M + "uv": (H * dv, r),
                        M + "sink": (H,), M + "o": (W, H * dv)})
        else:
            a, b = m["left"], m["right"]
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            L, R = pre + "mix.left.", pre + "mix.right."
            out.update({L + "q": (H * d, W), L + "k": (G * d, W), L + "v": (G * dv, W), L + "q.norm": (d,), L + "k.norm": (d,), L + "talk": (H, H),
                        L + "o": (W, H * dv)})
            C, k = b["width"], b["blocks"]
            s = C // k
            out.update({R + "y": (C, W), R + "y.b": (C,), R + "x": (C, W), R + "x.b": (C,), R + "conv": (C, b["conv"]), R + "conv.b": (C,),
                        R + "ra": (k, s, s), R + "ra.b": (k, s), R + "ri": (k, s, s), R + "ri.b": (k, s), R + "lam": (C,), R + "o": (W, C)})
        if lc.get("mlp"):
            F = lc["mlp"]["ff"]
            out.update({pre + "mlp.up": (F, W), pre + "mlp.down": (W, F)})
    return out


def random_weights(config, seed=0):
    """bf16-representable float64 tensors: projections ~ 1/sqrt(in), norms around one, stream tables near pass-through, decays spread
    from a few tokens to hundreds."""
    g = torch.Generator().manual_seed(seed)
    p = {}
    for name, shape in tensor_shapes(config).items():
        last = name.rsplit(".", 1)[-1]
        noise = torch.randn(shape, generator=g)
        if name == "embed":
            t = noise
        elif last in ("norm1", "norm2", "norm"):
            t = 1.0 + noise * 0.1
        elif last == "in":
            t = (1.0 + noise * 0.3) / shape[0]
        elif last == "out":
            t = 1.0 + noise * 0.4
        elif last == "mix":
            t = torch.eye(shape[0]) * 0.9 + noise * 0.15
        elif last == "talk":
            t = torch.eye(shape[0]) + noise * 0.4
        elif last == "conv":
            t = noise * 0.4
            t[:, -1] += 0.7
        elif last == "lam":
            t = torch.log(torch.expm1(torch.exp(torch.rand(shape, generator=g) * 5.0 - 6.5)))
        elif last in ("b", "sink"):
            t = noise * 0.3
        else:
            t = noise / math.sqrt(shape[-1])
        p[name] = t.to(torch.bfloat16).to(torch.float64)
    return p


def to_numpy_bf16_bits(t):
    return t.to(torch.bfloat16).view(torch.int16).numpy().view(np.uint16)
