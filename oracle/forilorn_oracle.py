"""Plain, slow restatement of the Forilorn decoder-only language model (test infrastructure only).

Torch on the CPU, one function per mechanism, whole sequences at once, no cache and no carried state: every position
is recomputed from the start of its sequence.  Nothing here is imported by the product path and nothing of the product
path is imported here.  The arithmetic type is the type of the tensors handed in (float64 gives a reference whose own
rounding is negligible).

Notation: matrices are ``[out, in]`` and applied as ``W @ x``; ``p`` maps the short tensor names of one mixer or
feed-forward (``q``, ``dkv.norm``, ``g``, ``up`` ...) to tensors, ``m`` is the matching dictionary of the configuration.

The model: x = s embed[token] + bigram[row(previous token, token)]; per layer x += r n_1(mixer(x)), x += r n_2(ff(x)) with
n(y) = y / rms(y) (1 + w) - the sublayers read x itself; logits = embed @ n_f(x).
"""

from __future__ import annotations

import math

import torch


# ---- elementwise pieces ---------------------------------------------------------------------------------------------
def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def zero_norm(x, w, eps):
    """The model's norm: the stored weight is the distance from one."""
    return rms_unit(x, eps) * (1.0 + w)


def gelu(z):
    """The tanh form."""
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- embedding --------------------------------------------------------------------------------------------------------
def bigram_rows(tokens, b):
    """The row of the pair table for every token of a sequence: the pair (previous, current) hashed into the buckets, the
    row behind the buckets for the first token."""
    rows = [b["buckets"]]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((int(prev) * b["mul_prev"] + int(cur) * b["mul_cur"]) % b["buckets"])
    return rows


def embedding(cfg, w, tokens):
    tokens = [int(t) for t in tokens]
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    b = cfg["embedding"].get("bigram")
    if b:
        x = x + w["bigram"][torch.tensor(bigram_rows(tokens, b), dtype=torch.long)]
    return x


# ---- rotary positions -------------------------------------------------------------------------------------------------
def rotate(x, positions, rot):
    """Turns the first ``dims`` channels of x [T, heads, n] (pairs 2i, 2i + 1) by position x base^(-2i/dims)."""
    if not rot or rot["dims"] == 0:
        return x
    dims = int(rot["dims"])
    f = torch.tensor([float(rot["base"]) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64).to(x.dtype)
    ang = positions.to(x.dtype)[:, None, None] * f[None, None, :]
    cs, sn = torch.cos(ang), torch.sin(ang)
    out = x.clone()
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = a * cs - b * sn
    out[..., 1:dims:2] = b * cs + a * sn
    return out


# ---- which keys a position sees ------------------------------------------------------------------------------------------
def in_chunk(i, j, size):
    """Key j is seen from query i when it is not in the future and lies in the same block of ``size`` positions."""
    return j <= i and i // size == j // size


def in_window(i, j, size):
    """Key j is seen from query i when it is not in the future and less than ``size`` tokens back."""
    return 0 <= i - j < size


def seen_mask(positions, rule, size):
    """[T, T] of ``rule`` over all pairs (no size: every earlier key)."""
    pos = [int(v) for v in positions]
    return torch.tensor([[(j <= i if size is None else rule(i, j, size)) for j in pos] for i in pos], dtype=torch.bool)


def softmax_rows(s, seen):
    s = torch.where(seen, s, torch.full_like(s, -math.inf))
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


# ---- mixers -----------------------------------------------------------------------------------------------------------
def attention(h, p, m, eps, positions=None):
    """Grouped-query softmax attention inside chunks: the values are the projected keys; q and k are turned, then divided by
    their root mean square per head; the heads' outputs are multiplied by the sigmoid of a projection of h."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(T) if positions is None else positions
    size = m["mask"]["size"] if m.get("mask") else None
    raw = (h @ p["k"].T).reshape(T, G, d)
    q = rms_unit(rotate((h @ p["q"].T).reshape(T, H, d), pos, m.get("rot")), eps)
    k = rms_unit(rotate(raw, pos, m.get("rot")), eps)
    seen = seen_mask(pos, in_chunk, size)
    out = torch.zeros((T, H, d), dtype=h.dtype)
    for hh in range(H):
        g = hh // (H // G)
        out[:, hh] = softmax_rows((q[:, hh] @ k[:, g].T) * m["scale"], seen) @ raw[:, g]
    return (out.reshape(T, H * d) * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


def latent_attention(h, p, m, eps, positions=None):
    """Softmax attention in a window whose keys and values are up-projections of one normed latent per token, with a turned key
    part shared by all heads; every head's output is multiplied by one sigmoid number."""
    T = h.shape[0]
    H, d, r, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    pos = torch.arange(T) if positions is None else positions
    size = m["mask"]["size"] if m.get("mask") else None
    cq = rms_unit(h @ p["dq"].T, eps) * p["dq.norm"]
    q = (cq @ p["uq"].T).reshape(T, H, d + r)
    down = h @ p["dkv"].T
    R = down.shape[1] - r
    c = rms_unit(down[:, :R], eps) * p["dkv.norm"]
    q_turned = rotate(q[..., d:], pos, m.get("rot"))
    k_turned = rotate(down[:, None, R:], pos, m.get("rot"))[:, 0]
    k = (c @ p["uk"].T).reshape(T, H, d)
    v = (c @ p["uv"].T).reshape(T, H, dv)
    seen = seen_mask(pos, in_window, size)
    out = torch.zeros((T, H, dv), dtype=h.dtype)
    for hh in range(H):
        s = (q[:, hh, :d] @ k[:, hh].T + q_turned[:, hh] @ k_turned.T) * m["scale"]
        out[:, hh] = softmax_rows(s, seen) @ v[:, hh]
    out = out * torch.sigmoid(h @ p["g"].T)[:, :, None]
    return out.reshape(T, H * dv) @ p["o"].T


# ---- feed-forward -------------------------------------------------------------------------------------------------------
def dense_ff(h, p):
    return gelu(h @ p["up"].T) @ p["down"].T


# ---- the model --------------------------------------------------------------------------------------------------------
MIXERS = {"attention": attention, "latent_attention": latent_attention}


def part(p, prefix):
    return {k[len(prefix):]: v for k, v in p.items() if k.startswith(prefix)}


def forward(cfg: dict, w: dict, tokens, keep_layers: bool = False, dtype=torch.float64):
    """Logits [T, vocab] of one whole sequence (and the residual stream after every layer)."""
    eps, r = cfg["norm"]["eps"], cfg["residual_mult"]
    w = {k: v.to(dtype) for k, v in w.items()}
    x = embedding(cfg, w, tokens)
    kept = []
    for i, lc in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + r * zero_norm(MIXERS[lc["type"]](x, part(w, p + "mix."), lc["mixer"], eps), w[p + "norm1"], eps)
        if lc.get("mlp"):
            x = x + r * zero_norm(dense_ff(x, part(w, p + "mlp.")), w[p + "norm2"], eps)
        kept.append(x)
    logits = zero_norm(x, w["final.norm"], eps) @ w["embed"].T
    return (logits, torch.stack(kept)) if keep_layers else logits


def greedy(cfg: dict, w: dict, prompt, n_new: int):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


def random_weights(cfg: dict, seed: int, spread: float = 1.0) -> dict:
    """Random float32 tensors that bfloat16 holds exactly, under the checkpoint's names."""
    g = torch.Generator().manual_seed(seed)
    D, w = cfg["width"], {}

    def mat(n_out, n_in, gain=1.0):
        return (torch.randn((n_out, n_in), generator=g) * (gain * spread / math.sqrt(n_in))).to(torch.bfloat16).float()

    def vec(n, mean=0.0, dev=0.1):
        return (mean + dev * torch.randn((n,), generator=g)).to(torch.bfloat16).float()

    emb = cfg["embedding"]
    w["embed"] = (torch.randn((cfg["vocab"], D), generator=g) * (spread / math.sqrt(D))).to(torch.bfloat16).float()
    w["final.norm"] = vec(D)
    if emb.get("bigram"):
        w["bigram"] = (torch.randn((emb["bigram"]["buckets"] + 1, D), generator=g) * (0.7 * spread)).to(torch.bfloat16).float()
    for i, lc in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lc["mixer"]
        q, H, d, dv = p + "mix.", m["heads"], m["dim"], m["vdim"]
        w[p + "norm1"] = vec(D, 0.0, 0.3)
        if lc["type"] == "attention":
            G = m["kv_heads"]
            w[q + "q"], w[q + "k"], w[q + "g"], w[q + "o"] = mat(H * d, D), mat(G * d, D), mat(H * d, D, 1.5), mat(D, H * d)
        else:
            r, Rq, R = m["rot_dim"], m["q_rank"], m["kv_rank"]
            w[q + "dq"], w[q + "dq.norm"], w[q + "uq"] = mat(Rq, D), vec(Rq, 1.0, 0.3), mat(H * (d + r), Rq, 1.5)
            w[q + "dkv"], w[q + "dkv.norm"] = mat(R + r, D), vec(R, 1.0, 0.3)
            w[q + "uk"], w[q + "uv"] = mat(H * d, R, 1.5), mat(H * dv, R)
            w[q + "g"], w[q + "o"] = mat(H, D, 1.5), mat(D, H * dv)
        f = lc.get("mlp")
        if f:
            w[p + "norm2"] = vec(D, 0.0, 0.3)
            w[p + "mlp.up"], w[p + "mlp.down"] = mat(f["ff"], D, 1.5), mat(D, f["ff"])
    return w
