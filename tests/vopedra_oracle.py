"""Vopedra in float64, one plain function per mechanism, written from the equations; it shares no code with the package.

Notation: T tokens, W width.  unit(x) = x / sqrt(mean(x^2) + eps) over the last axis.  Everything runs token after token
with explicit states.

  embedding     x = g_e * unit(E[token]);  x0 denotes this x
  runs          the layer list with the slice [start, stop) repeated `times` times in a row, every repetition with a state
                of its own; ahead of repetition t: x <- x + x0 (t > 0 only), then x <- x + step[t]
  layer         x <- x + mixer(g1 * unit(x)) + ff(g2 * unit(x)), both of the same x
  mlstm         q = W_q h / sqrt(d), k = W_k h, v = W_v h per head; a = c tanh((W_i h + b_i) / c),
                b = log sigmoid(c tanh((W_f h + b_f) / c)), c = gate_cap;  u' = max(b + u, a)  (u = 0 ahead of the first token)
                S <- e^(b + u - u') S + e^(a - u') k v^T,  n <- e^(b + u - u') n + e^(a - u') k,
                o = S^T q / (max(|n . q|, e^(-u')) + 1e-6);  y = W_o (sigmoid(W_g h) * g * concat(unit(o)))
  mamba1        [x | z] = W_in h;  x <- silu(bias + causal convolution);  [dt | B | C] = W_x x;  D = softplus(W_dt dt + b);
                S[c, n] <- exp(-D_c e^(A_log[c, n])) S[c, n] + D_c x_c B_n;  y_c = S[c, :] . C + skip_c x_c;  W_o (y * silu(z))
  parallel      (g_l * unit(left(h)) + g_r * unit(right(h))) / 2
    left        q, k, v = projections; q <- g_q * unit(q), k <- g_k * unit(k) over ALL heads' columns; rotary (pairs i, i + n/2)
                on the first n = rot.dims of every head; p_h = causal softmax(scale q_h . k_c(h)), c(h) = h // (H / G);
                p'_h = sum_g talk[h][g] p_g;  o_h = sum_j p'_h,j v_c(h),j;  W_o concat(o)
    right       q = silu(W_q h), v = W_v h, f = l + (1 - l) sigmoid(W_f h + b) per head and channel;
                S <- diag(f) S + (1 - f) v^T;  o = S^T q;  W_o concat(g * unit(o)), g of one head's size
  ff            W_down (gelu(W_gate h) * W_up h), gelu(z) = z/2 (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))
  output        logits = W_head (g * unit(x))
"""
import math

import torch

F64 = torch.float64


def unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x / (1 + torch.exp(-x))


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp(min=0)


def log_sigmoid(x):
    return -softplus(-x)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_half_pairs(x, positions, base, n):
    """x [T, heads, size]: dimension i < n / 2 turns with i + n / 2 by position * base^(-2 i / n); the rest passes."""
    i = torch.arange(n // 2, dtype=F64)
    a = positions.to(F64)[:, None] * torch.pow(torch.tensor(float(base), dtype=F64), -2.0 * i / max(n, 1))[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], -1)


def softmax_then_mix_rows(q, k, v, scale, talk, first=0):
    """q [T, H, d] and k [S, G, d] as they meet, v [S, G, dv]; query row t sits at position first + t and sees keys
    0 .. first + t.  The heads' softmax weights are mixed by talk [H, H] before they meet the values."""
    T, H, _ = q.shape
    G, dv = v.shape[1:]
    rep = H // G
    out = torch.zeros(T, H, dv, dtype=F64)
    for t in range(T):
        n = first + t + 1
        p = torch.stack([torch.softmax(k[:n, h // rep] @ q[t, h] * scale, -1) for h in range(H)])
        p = talk @ p
        for h in range(H):
            out[t, h] = p[h] @ v[:n, h // rep]
    return out


def attention_branch(t, p, m, h, eps):
    T = h.shape[0]
    H, G, d, dv, rot = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    pos = torch.arange(T)
    q = (t[p + "q.norm"] * unit(h @ t[p + "q"].T, eps)).reshape(T, H, d)
    k = (t[p + "k.norm"] * unit(h @ t[p + "k"].T, eps)).reshape(T, G, d)
    q, k = rotate_half_pairs(q, pos, rot["base"], rot["dims"]), rotate_half_pairs(k, pos, rot["base"], rot["dims"])
    o = softmax_then_mix_rows(q, k, (h @ t[p + "v"].T).reshape(T, G, dv), m["scale"], t[p + "talk"])
    return o.reshape(T, H * dv) @ t[p + "o"].T


def gated_rows(q, k, v, f, S=None):
    """q, k, f [T, H, d], v [T, H, dv]:  S <- diag(f) S + k v^T,  o = S^T q.  Returns (o [T, H, dv], S)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64) if S is None else S.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for i in range(T):
        S = f[i][:, :, None] * S + k[i][:, :, None] * v[i][:, None, :]
        out[i] = torch.einsum("hdv,hd->hv", S, q[i])
    return out, S


def hgrn2_branch(t, p, m, h, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    low = t[p + "lower"]
    f = (low + (1 - low) / (1 + torch.exp(-(h @ t[p + "f"].T + t[p + "f.b"])))).reshape(T, H, d)
    q, v = silu(h @ t[p + "q"].T).reshape(T, H, d), (h @ t[p + "v"].T).reshape(T, H, dv)
    o, _ = gated_rows(q, 1 - f, v, f)
    return (t[p + "norm"] * unit(o, eps)).reshape(T, H * dv) @ t[p + "o"].T


def parallel_mixer(t, p, m, h, eps):
    left, right = attention_branch(t, p + "left.", m["left"], h, eps), hgrn2_branch(t, p + "right.", m["right"], h, eps)
    return (t[p + "left.out"] * unit(left, eps) + t[p + "right.out"] * unit(right, eps)) / 2


def mlstm_gates(zi, zf, cap):
    """(log input gate, log forget gate) from the gates' projections, bias included."""
    return cap * torch.tanh(zi / cap), log_sigmoid(cap * torch.tanh(zf / cap))


def mlstm_rows(q, k, v, a, b, state=None):
    """q (scaled), k [T, H, d], v [T, H, dv], log gates a (input), b (forget) [T, H].  Returns (o, (S, n, u))."""
    T, H, d = q.shape
    dv = v.shape[-1]
    S, n, u = state if state is not None else (torch.zeros(H, d, dv, dtype=F64), torch.zeros(H, d, dtype=F64), torch.zeros(H, dtype=F64))
    out = torch.zeros(T, H, dv, dtype=F64)
    for i in range(T):
        u_new = torch.maximum(b[i] + u, a[i])
        keep, put = torch.exp(b[i] + u - u_new), torch.exp(a[i] - u_new)
        S = keep[:, None, None] * S + put[:, None, None] * k[i][:, :, None] * v[i][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[i]
        u = u_new
        den = torch.maximum((n * q[i]).sum(-1).abs(), torch.exp(-u)) + 1e-6
        out[i] = torch.einsum("hdv,hd->hv", S, q[i]) / den[:, None]
    return out, (S, n, u)


def mlstm_mixer(t, p, m, h, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ t[p + "q"].T).reshape(T, H, d) * d ** -0.5, (h @ t[p + "k"].T).reshape(T, H, d), (h @ t[p + "v"].T).reshape(T, H, dv)
    a, b = mlstm_gates(h @ t[p + "i"].T + t[p + "i.b"], h @ t[p + "f"].T + t[p + "f.b"], m["gate_cap"])
    o, _ = mlstm_rows(q, k, v, a, b)
    return (unit(o, eps).reshape(T, H * dv) * t[p + "norm"] / (1 + torch.exp(-(h @ t[p + "g"].T)))) @ t[p + "o"].T


def causal_conv_rows(x, w, bias):
    """x [T, C], w [C, taps]: tap j meets the input taps - 1 - j tokens back, nothing ahead of the first token."""
    T, taps = x.shape[0], w.shape[1]
    pad = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=F64), x], 0)
    return bias + sum(w[:, j] * pad[j:j + T] for j in range(taps))


def selective_rows(x, step, A, B, C, S=None):
    """x, step [T, c], A [c, n], B, C [T, n]:  S <- exp(step A) S + step x B^T;  y = S C.  Returns (y, S)."""
    T, c = x.shape
    S = torch.zeros(c, A.shape[1], dtype=F64) if S is None else S.clone()
    y = torch.zeros(T, c, dtype=F64)
    for i in range(T):
        S = torch.exp(step[i][:, None] * A) * S + (step[i] * x[i])[:, None] * B[i][None, :]
        y[i] = S @ C[i]
    return y, S


def mamba1_mixer(t, p, m, h):
    inner, r, n = m["inner"], m["dt_rank"], m["state"]
    xz = h @ t[p + "in"].T
    x, z = silu(causal_conv_rows(xz[:, :inner], t[p + "conv"], t[p + "conv.b"])), xz[:, inner:]
    s = x @ t[p + "x"].T
    step = softplus(s[:, :r] @ t[p + "dt"].T + t[p + "dt.b"])
    y, _ = selective_rows(x, step, -torch.exp(t[p + "A_log"]), s[:, r:r + n], s[:, r + n:])
    return ((y + t[p + "D"] * x) * silu(z)) @ t[p + "o"].T


def gated_ff(t, p, h):
    return (gelu_tanh(h @ t[p + "gate"].T) * (h @ t[p + "up"].T)) @ t[p + "down"].T


def run_order(n_layers, loop):
    """[(layer, repetition or None if it opens none)] in the order the layers run."""
    if not loop:
        return [(i, None) for i in range(n_layers)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n_layers)]


def mixer_out(t, p, l, h, eps):
    m = l["mixer"]
    if l["type"] == "mlstm":
        return mlstm_mixer(t, p, m, h, eps)
    if l["type"] == "mamba1":
        return mamba1_mixer(t, p, m, h)
    return parallel_mixer(t, p, m, h, eps)


def model_logits(tensors, cfg, tokens, residual_out=None):
    t = {k: v.to(F64) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = x0 = t["embed.norm"] * unit(t["embed"][torch.tensor(tokens)], eps)
    for i, opens in run_order(len(cfg["layers"]), cfg.get("loop")):
        l, p = cfg["layers"][i], f"l{i}."
        if opens is not None:
            if opens > 0:
                x = x + x0
            x = x + t["loop.step"][opens]
        y = mixer_out(t, p + "mix.", l, t[p + "norm1"] * unit(x, eps), eps)
        if l.get("mlp"):
            y = y + gated_ff(t, p + "mlp.", t[p + "norm2"] * unit(x, eps))
        x = x + y
        if residual_out is not None:
            residual_out.append(x.clone())
    return (t["final.norm"] * unit(x, eps)) @ t["head"].T


def logit_error(got, want):
    """Per row: root mean square of the difference with its mean taken off, over the root mean square of the wanted row."""
    d = got.to(F64) - want.to(F64)
    d = d - d.mean(-1, keepdim=True)
    w = want.to(F64) - want.to(F64).mean(-1, keepdim=True)
    return torch.sqrt((d * d).mean(-1)) / torch.sqrt((w * w).mean(-1))
