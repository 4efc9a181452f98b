"""A plain, slow implementation of the Zuvevik decoder: whole sequences, no cache, no batching, one function for each
mechanism, float64. It shares no code with the engine and is what the engine's Zuvevik results are compared with.

The design in this file's notation (X: the streams [S, T, d]):

    start:      x0 = E[token] + B[pair of neighbouring tokens]; every stream starts as x0
    sublayer:   u = sum_s a_s X_s;  y = f(N(u));  X'_t = sum_s M[s, t] X_s + b_t y       (a, b, M: the sublayer's own)
    mixer:      windowed attention; q and k normed over the whole projection and rotated in halves; the values blended with
                those of the first blending layer; a sigmoid gate per channel
    ff:         dense (silu gate), or routed experts whose weight scales what the expert READS
    output:     the sum of the streams, RMS norm, a head of its own, a constant factor
"""
import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------------ embedding
def pair_rows(tokens, mul_prev, mul_cur, buckets):
    """The row of the pair table for every token: a hash of (previous, current), or the last row without a previous one."""
    rows, prev = [], None
    for t in (int(v) for v in tokens):
        rows.append(buckets if prev is None else (prev * mul_prev + t * mul_cur) % buckets)
        prev = t
    return torch.tensor(rows)


def embed(tokens, table, pairs, c):
    return table[tokens] + pairs[pair_rows(tokens, c["mul_prev"], c["mul_cur"], c["buckets"])]


# ------------------------------------------------------------------------------------------------ norm, streams
def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def read_streams(X, a):
    return torch.einsum("s,std->td", a, X)


def write_streams(X, M, b, y):
    """M is indexed [from, to]."""
    return torch.einsum("st,snd->tnd", M, X) + b[:, None, None] * y[None]


# ------------------------------------------------------------------------------------------------ attention
def rotate_halves(x, positions, dims, base):
    """x [T, heads, n]: (x_i, x_(i + dims/2)) = (u, v) become (u cos a - v sin a, v cos a + u sin a), a = position *
    base^(-2i / dims); dimensions from `dims` on pass unchanged."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    a = (positions.to(F64)[:, None] * f[None, :])[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a), x[..., dims:]], dim=-1)


def visible(T, window):
    """[query, key]: the key is the query or one of the window - 1 tokens before it."""
    i = torch.arange(T)
    back = i[:, None] - i[None, :]
    return (back >= 0) & (back < window if window else back >= 0)


def attend(q, k, v, scale, window):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; query head h uses key/value head h // (H / G)."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    k, v = k.repeat_interleave(per, dim=1), v.repeat_interleave(per, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    p = torch.softmax(s.masked_fill(~visible(T, window), float("-inf")), dim=-1)
    return torch.einsum("hij,jhe->ihe", p, v)


def blend_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def channel_gate(o, h, wg):
    return o * torch.sigmoid(h @ wg.T)


def attention_mixer(h, w, c, eps, positions, first_values):
    """(output, the projected values as the first blending layer hands them on)."""
    T = h.shape[0]
    H, G, d, e = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    dims, base = c["rot"]["dims"], c["rot"]["base"]
    q = rotate_halves(rms_norm(h @ w["q"].T, w["q.norm"], eps).view(T, H, d), positions, dims, base)
    k = rotate_halves(rms_norm(h @ w["k"].T, w["k.norm"], eps).view(T, G, d), positions, dims, base)
    own = h @ w["v"].T
    v = own if first_values is None else blend_values(own, first_values, w["vmix"])
    window = (c.get("mask") or {}).get("size", 0)
    o = attend(q, k, v.view(T, G, e), c["scale"], window).reshape(T, H * e)
    return channel_gate(o, h, w["g"]) @ w["o"].T, own


# ------------------------------------------------------------------------------------------------ feed-forward
def dense_ff(h, w):
    g = h @ w["gate"].T
    return (g * torch.sigmoid(g) * (h @ w["up"].T)) @ w["down"].T


def clamped_glu(g, u, limit):
    g = torch.clamp(g, max=limit)
    u = torch.clamp(u, min=-limit, max=limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def expert(h, w, name, limit):
    return clamped_glu(h @ w[name + ".gate"].T, h @ w[name + ".up"].T, limit) @ w[name + ".down"].T


def choose_experts(z, top):
    """(ids, weights): the `top` largest sigmoid scores (ties: the lower index), which are the weights as they are."""
    s = torch.sigmoid(z)
    ids = torch.tensor([sorted(range(z.shape[1]), key=lambda e: (-float(row[e]), e))[:top] for row in s])
    return ids, torch.gather(s, 1, ids)


def routed_experts(h, w, c, forced=None, info=None):
    """`forced` [T, top]: take these experts instead of the own choice; `info` (a list) receives the logits and the choice."""
    z = h @ w["router"].T
    ids, wts = choose_experts(z, c["router"]["top"])
    if info is not None:
        info.append({"logits": z, "own": ids})
    if forced is not None:
        ids = forced.to(torch.int64)
        wts = torch.gather(torch.sigmoid(z), 1, ids)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, p in zip(ids[t].tolist(), wts[t]):
            out[t] += expert(p * h[t:t + 1], w, f"e{e}", c["expert"]["limit"])[0]
    return out


# ------------------------------------------------------------------------------------------------ the model
def _sub(tensors, prefix):
    return {k[len(prefix):]: v.to(F64) for k, v in tensors.items() if k.startswith(prefix)}


def forward(config: dict, tensors: dict, tokens, streams: bool = False, forced=None, info=None):
    """Logits [T, vocab] of one sequence from its start; `streams`: also the sum of the streams behind every layer.
    `forced`: {layer: ids [T, top]}; `info` (a dict) receives each routed layer's logits and choice."""
    eps, S = config["norm"]["eps"], config["streams"]
    tokens = torch.as_tensor(tokens, dtype=torch.int64)
    positions = torch.arange(tokens.shape[0])
    get = lambda name: tensors[name].to(F64)
    x0 = embed(tokens, get("embed"), get("bigram"), config["embedding"]["bigram"])
    X = x0[None].repeat(S, 1, 1)
    first, kept = None, []
    for i, layer in enumerate(config["layers"]):
        p, c, m = f"l{i}.", layer["mixer"], layer.get("mlp")
        if layer["type"] != "attention":
            raise ValueError(layer["type"])
        h = rms_norm(read_streams(X, get(p + "hc1.in")), get(p + "norm1"), eps)
        blends = bool(c.get("v_mix"))
        y, own = attention_mixer(h, _sub(tensors, p + "mix."), c, eps, positions, first if blends else None)
        if blends and first is None:
            first = own
        X = write_streams(X, get(p + "hc1.mix"), get(p + "hc1.out"), y)
        if m is not None:
            h = rms_norm(read_streams(X, get(p + "hc2.in")), get(p + "norm2"), eps)
            wf = _sub(tensors, p + "mlp.")
            if m["kind"] == "dense":
                y = dense_ff(h, wf)
            else:
                rec = [] if info is not None else None
                y = routed_experts(h, wf, m, None if forced is None else forced.get(i), rec)
                if info is not None:
                    info[i] = rec[0]
            X = write_streams(X, get(p + "hc2.mix"), get(p + "hc2.out"), y)
        kept.append(X.sum(0))
    logits = rms_norm(X.sum(0), get("final.norm"), eps) @ get("head").T * config["logit_scale"]
    return (logits, kept) if streams else logits
