"""A plain, slow implementation of the Gipinex decoder: whole sequences, no cache, no batching, one function for each
mechanism, float64. It shares no code with the engine and is what the engine's Gipinex results are compared with.

The design in this file's notation (x: residual stream [T, d], x0: the embedding rows, a: a constant):

    layer:      x <- x + a mixer(N1(x));   x <- x + a ff(N2(x))       (N: RMS norm whose weight is stored as w - 1; a layer
                                                                       may have no ff)
    loop:       layers start .. stop-1 run several times with the same tensors; ahead of each pass x <- W [x; x0]
    mixers:     'attention'         queries and keys of unit root mean square; the values are the keys before that; a score
                                    loses slope_h times the distance, and the heads' scores are mixed BEFORE the softmax;
                                    a sigmoid gate per channel
                'latent_attention'  keys and values made from one small vector per token and one rotated key part that
                                    all heads share; queries through a latent of their own; a sigmoid gate per head
    ff:         dense (clamped gated activation, biases), or routed experts whose weights are a softmax over the chosen
                logits, plus an optional expert that every token uses
    output:     RMS norm, the embedding table
"""
import math

import torch

F64 = torch.float64


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def offset_norm(x, w, eps):
    """The weight is stored around zero."""
    return rms_unit(x, eps) * (1.0 + w)


# ------------------------------------------------------------------------------------------------ attention
def distance_slopes(H):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=F64)


def biased_scores(q, k, scale):
    """q [H, T, d], k [H, T, d]: q . k * scale - slope_h (i - j)."""
    H, T, _ = q.shape
    i = torch.arange(T, dtype=F64)
    dist = i[:, None] - i[None, :]
    return torch.einsum("hid,hjd->hij", q, k) * scale - distance_slopes(H)[:, None, None] * dist[None]


def mix_heads(talk, s):
    """s'_h = sum_g talk[h, g] s_g."""
    return torch.einsum("hg,gij->hij", talk, s)


def causal_softmax(s):
    T = s.shape[-1]
    seen = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    return torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1)


def mixed_score_attention(q, k, scale, talk, eps):
    """q [T, H, d], k [T, G, d] as projected. Returns [T, H, d]: query head h uses key/value head h // (H / G)."""
    T, H, d = q.shape
    per = H // k.shape[1]
    keys = rms_unit(k, eps).repeat_interleave(per, dim=1).permute(1, 0, 2)
    vals = k.repeat_interleave(per, dim=1).permute(1, 0, 2)
    s = biased_scores(rms_unit(q, eps).permute(1, 0, 2), keys, scale)
    p = causal_softmax(mix_heads(talk, s))
    return torch.einsum("hij,hjd->ihd", p, vals)


def attention_mixer(h, w, c, eps):
    T = h.shape[0]
    H, G, d = c["heads"], c["kv_heads"], c["dim"]
    q = (h @ w["q"].T).view(T, H, d)
    k = (h @ w["k"].T).view(T, G, d)
    o = mixed_score_attention(q, k, c["scale"], w["talk"], eps).reshape(T, H * d)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# ------------------------------------------------------------------------------------------------ latent attention
def rotate_pairs(x, positions, dims, base):
    """x [..., T, n]: neighbours (x_2i, x_2i+1) = (u, v), i < dims / 2, become (u cos a - v sin a, v cos a + u sin a) with
    a = position * base^(-2i / dims); the rest pass unchanged."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    a = positions.to(F64)[:, None] * f[None, :]
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * torch.cos(a) - v * torch.sin(a)
    out[..., 1:dims:2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def latent_attention_mixer(h, w, c, eps, positions):
    T = h.shape[0]
    H, dn, dr, dv, r = c["heads"], c["dim"], c["rot_dim"], c["vdim"], c["kv_rank"]
    base, dims = c["rot"]["base"], c["rot"].get("dims", dr)
    cq = rms_norm(h @ w["dq"].T, w["dq.norm"], eps)
    q = (cq @ w["uq"].T).view(T, H, dn + dr).permute(1, 0, 2)
    z = h @ w["dkv"].T
    lat = rms_norm(z[:, :r], w["dkv.norm"], eps)
    k_rot = rotate_pairs(z[:, r:], positions, dims, base)
    q_rot = rotate_pairs(q[:, :, dn:], positions, dims, base)
    k = (lat @ w["uk"].T).view(T, H, dn).permute(1, 0, 2)
    v = (lat @ w["uv"].T).view(T, H, dv).permute(1, 0, 2)
    s = (torch.einsum("hid,hjd->hij", q[:, :, :dn], k) + torch.einsum("hid,jd->hij", q_rot, k_rot)) * c["scale"]
    o = torch.einsum("hij,hjd->ihd", causal_softmax(s), v)
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w["o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def clamped_glu(g, u, limit):
    g = torch.clamp(g, max=limit)
    u = torch.clamp(u, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(h, w, limit):
    return clamped_glu(h @ w["gate"].T + w["gate.b"], h @ w["up"].T + w["up.b"], limit) @ w["down"].T + w["down.b"]


def expert(h, w, name, limit):
    return clamped_glu(h @ w[name + ".gate"].T, h @ w[name + ".up"].T, limit) @ w[name + ".down"].T


def choose_experts(z, top):
    """(ids, weights): the `top` largest logits (ties: the lower index), weighted by the softmax over them alone."""
    ids = torch.tensor([sorted(range(z.shape[1]), key=lambda e: (-float(row[e]), e))[:top] for row in z])
    return ids, torch.softmax(torch.gather(z, 1, ids), dim=-1)


def routed_experts(h, w, c, forced=None, info=None):
    """`forced` [T, top]: take these experts instead of the own choice; `info` (a list) receives the logits and the choice."""
    z = h @ w["router"].T + w["router.b"]
    ids, wts = choose_experts(z, c["router"]["top"])
    if info is not None:
        info.append({"logits": z, "own": ids})
    if forced is not None:
        ids = forced.to(torch.int64)
        wts = torch.softmax(torch.gather(z, 1, ids), dim=-1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(ids[t].tolist(), wts[t]):
            out[t] += p * expert(h[t:t + 1], w, f"e{e}", c["expert"]["limit"])[0]
    if c.get("shared"):
        out = out + expert(h, w, "shared", c["shared"]["limit"])
    return out


# ------------------------------------------------------------------------------------------------ the model
def run_order(config):
    """[(layer, first of a pass)]: the layers in the order in which they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    body = [(i, i == a) for i in range(a, b)]
    return [(i, False) for i in range(a)] + body * loop["times"] + [(i, False) for i in range(b, n)]


def _sub(tensors, prefix):
    return {k[len(prefix):]: v.to(F64) for k, v in tensors.items() if k.startswith(prefix)}


def forward(config: dict, tensors: dict, tokens, streams: bool = False, forced=None, info=None):
    """Logits [T, vocab] of one sequence from its start; `streams`: also the stream behind every layer run. `forced`:
    {place in the run order: ids [T, top]}; `info` (a dict) receives each routed run's logits and choice."""
    eps, a = config["norm"]["eps"], config["residual_mult"]
    tokens = torch.as_tensor(tokens, dtype=torch.int64)
    positions = torch.arange(tokens.shape[0])
    x0 = tensors["embed"].to(F64)[tokens]
    x, kept = x0, []
    for n, (i, enters) in enumerate(run_order(config)):
        layer, p = config["layers"][i], f"l{i}."
        if enters:
            x = torch.cat([x, x0], dim=1) @ tensors["loop.in"].to(F64).T
        h = offset_norm(x, tensors[p + "norm1"].to(F64), eps)
        w, c = _sub(tensors, p + "mix."), layer["mixer"]
        if layer["type"] == "attention":
            y = attention_mixer(h, w, c, eps)
        elif layer["type"] == "latent_attention":
            y = latent_attention_mixer(h, w, c, eps, positions)
        else:
            raise ValueError(layer["type"])
        x = x + a * y
        m = layer.get("mlp")
        if m is not None:
            h = offset_norm(x, tensors[p + "norm2"].to(F64), eps)
            wf = _sub(tensors, p + "mlp.")
            if m["kind"] == "dense":
                y = dense_ff(h, wf, m["limit"])
            else:
                rec = [] if info is not None else None
                y = routed_experts(h, wf, m, None if forced is None else forced.get(n), rec)
                if info is not None:
                    info[n] = rec[0]
            x = x + a * y
        kept.append(x.clone())
    logits = offset_norm(x, tensors["final.norm"].to(F64), eps) @ tensors["embed"].to(F64).T
    return (logits, kept) if streams else logits
