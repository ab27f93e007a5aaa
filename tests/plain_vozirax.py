"""Vozirax, plainly: whole sequences, no cache, no batching, one function per mechanism.

Everything here is written from the design's equations for the tests to compare the engine
with; it shares no code with the package.  ``tensors`` maps checkpoint names to tensors,
``config`` is the parsed config.json.  Arithmetic runs in ``dtype`` (float64 unless told
otherwise).

Notation: T tokens, W the model's width, H heads, G key/value heads or groups, d a head's
query/key size, e its value size, N the numbers of a state row, p_t the position of token t
(0 for the first token of a sequence).
"""

import json
import math
import os
import struct

import numpy as np
import torch


# ------------------------------------------------------------------------------- norms, activations
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """A gain that is stored as its distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


def unit_rms_in_parts(x, parts, eps):
    """The last axis cut into ``parts`` equal runs, each divided by its own root mean square."""
    return unit_rms(x.reshape(*x.shape[:-1], parts, -1), eps).reshape(x.shape)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0.0)


def linear(tensors, name, h):
    return h @ tensors[name].to(h.dtype).T


# ------------------------------------------------------------------------------- positions
def position_rows(positions, width, dtype=torch.float64):
    """Number 2i of position p's row is sin(p / 10000^(2i / width)), number 2i + 1 the cosine of the same angle."""
    rows = torch.zeros(len(positions), width, dtype=dtype)
    for c in range(width):
        angle = positions.to(dtype) * 10000.0 ** (-2.0 * (c // 2) / width)
        rows[:, c] = torch.sin(angle) if c % 2 == 0 else torch.cos(angle)
    return rows


# ------------------------------------------------------------------------------- state space
def causal_convolution(u, weight, bias):
    """u [T, C], weight [C, taps], newest row last; rows before the first are zeros."""
    taps = weight.shape[1]
    rows = torch.cat([u.new_zeros(taps - 1, u.shape[1]), u])
    out = bias[None].expand_as(u).clone()
    for j in range(taps):
        out = out + weight[:, j] * rows[j:j + u.shape[0]]
    return out


def state_space(x, b, c, dt, a_log, d):
    """x [T, H, e], b and c [T, G, N], dt [T, H] (positive): one H x N x e state, token by token."""
    T, H, e = x.shape
    share = H // b.shape[1]
    rate = -torch.exp(a_log)
    state = x.new_zeros(H, b.shape[2], e)
    rows = []
    for t in range(T):
        keep = torch.exp(rate * dt[t])
        b_t, c_t = b[t].repeat_interleave(share, 0), c[t].repeat_interleave(share, 0)
        state = keep[:, None, None] * state + (dt[t][:, None] * b_t)[:, :, None] * x[t][:, None, :]
        rows.append(torch.einsum("hn,hne->he", c_t, state) + d[:, None] * x[t])
    return torch.stack(rows)


def mamba(tensors, prefix, m, h, eps):
    """One projection, convolved parts, the state, the gate and then the norm in parts."""
    t = lambda name: tensors[prefix + name].to(h.dtype)
    H, e, N, G, T = m["heads"], m["vdim"], m["state"], m["groups"], h.shape[0]
    inner = H * e
    z, xbc, dt = torch.split(linear(tensors, prefix + "in", h), [inner, inner + 2 * G * N, H], dim=-1)
    x, b, c = torch.split(silu(causal_convolution(xbc, t("conv"), t("conv.b"))), [inner, G * N, G * N], dim=-1)
    y = state_space(x.reshape(T, H, e), b.reshape(T, G, N), c.reshape(T, G, N), softplus(dt + t("dt_bias")), t("A_log"),
                    t("D"))
    y = unit_rms_in_parts(y.reshape(T, inner) * silu(z), m["norm_groups"], eps) * t("norm")
    return linear(tensors, prefix + "o", y)


# ------------------------------------------------------------------------------- attention
def causal_softmax(scores):
    """scores [T, T] (query, key)."""
    T = scores.shape[-1]
    return torch.softmax(scores.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf")), dim=-1)


def temperature(positions, q_temp, dtype=torch.float64):
    """What the queries of a position are multiplied by."""
    if not q_temp:
        return torch.ones(len(positions), dtype=dtype)
    runs = torch.div(positions + 1, q_temp["every"], rounding_mode="floor").to(dtype)
    return 1.0 + q_temp["coef"] * torch.log(runs + 1.0)


def keys_and_values(tensors, prefix, m, h, eps):
    """[T, G, 2, d] normed keys of both maps, [T, G, e] values."""
    G, T = m["kv_heads"], h.shape[0]
    k = linear(tensors, prefix + "k", h).reshape(T, G, 2, m["dim"])
    return (unit_rms(k, eps) * tensors[prefix + "k.norm"].to(h.dtype),
            linear(tensors, prefix + "v", h).reshape(T, G, m["vdim"]))


def map_share(tensors, prefix, m, dtype=torch.float64):
    """How much of the second map is taken off the first."""
    dot = lambda a, b: (tensors[prefix + a].to(dtype) * tensors[prefix + b].to(dtype)).sum()
    return torch.exp(dot("lq1", "lk1")) - torch.exp(dot("lq2", "lk2")) + m["diff"]


def differential_attention(tensors, prefix, m, h, positions, eps, kv):
    """Two softmax maps per head over the same values, subtracted; head norm without a gain; a gate per head."""
    H, G, d, T = m["heads"], m["kv_heads"], m["dim"], h.shape[0]
    q = linear(tensors, prefix + "q", h).reshape(T, H, 2, d)
    q = unit_rms(q, eps) * tensors[prefix + "q.norm"].to(h.dtype)
    q = q * temperature(positions, m.get("q_temp"), h.dtype)[:, None, None, None]
    k, v = kv
    share = map_share(tensors, prefix, m, h.dtype)
    gates = torch.sigmoid(linear(tensors, prefix + "g", h))
    rows = []
    for head in range(H):
        group = head // (H // G)
        a1, a2 = (causal_softmax((q[:, head, i] @ k[:, group, i].T) * m["scale"]) @ v[:, group] for i in (0, 1))
        rows.append(unit_rms(a1 - share * a2, eps) * (1.0 - m["diff"]) * gates[:, head:head + 1])
    return linear(tensors, prefix + "o", torch.cat(rows, dim=-1))


# ------------------------------------------------------------------------------- feed-forward
def gated_ff(tensors, prefix, h):
    return linear(tensors, prefix + "down", silu(linear(tensors, prefix + "gate", h)) * linear(tensors, prefix + "up", h))


def expert(tensors, prefix, h):
    return linear(tensors, prefix + "down", torch.relu(linear(tensors, prefix + "up", h)) ** 2)


def election(scores, correction, router):
    """One token's scores: ({expert: weight}, how clear the election was)."""
    E, top = router["experts"], router["top"]
    choice = scores + correction
    standing = list(range(E))
    margin = float("inf")
    groups = router.get("groups")
    if groups:
        per = E // groups["count"]
        marks = []
        for g in range(groups["count"]):
            best = sorted((float(choice[e]) for e in range(g * per, (g + 1) * per)), reverse=True)[:2]
            marks.append((sum(best), g))
        marks.sort(key=lambda item: (-item[0], item[1]))
        if groups["keep"] < groups["count"]:
            margin = marks[groups["keep"] - 1][0] - marks[groups["keep"]][0]
        kept = {g for _, g in marks[:groups["keep"]]}
        standing = [e for e in standing if e // per in kept]
    order = sorted(standing, key=lambda e: (-float(choice[e]), e))
    if top < len(order):
        margin = min(margin, float(choice[order[top - 1]] - choice[order[top]]))
    total = sum(scores[e] for e in order[:top]) + 1e-20
    return {e: scores[e] / total * router.get("scale", 1.0) for e in order[:top]}, margin


def routed_experts(tensors, prefix, mlp, h, margins=None):
    scores = torch.sigmoid(linear(tensors, prefix + "router", h))
    correction = tensors[prefix + "correction"].to(h.dtype)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        weights, margin = election(scores[t], correction, mlp["router"])
        if margins is not None:
            margins[t] = min(margins[t], margin)
        for e, weight in weights.items():
            out[t] = out[t] + weight * expert(tensors, f"{prefix}e{e}.", h[t])
    return out


# ------------------------------------------------------------------------------- the model
def forward(tensors, config, tokens, dtype=torch.float64, layers_out=None, margins=None):
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: a list that receives the residual rows behind
    every layer; ``margins``: a list of T numbers that receives how clear each token's closest election was."""
    eps = config["norm"]["eps"]
    t = lambda name: tensors[name].to(dtype)
    ids = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(len(ids))
    x = t("embed")[ids] + position_rows(positions, config["width"], dtype)
    if margins is not None and not margins:
        margins.extend([float("inf")] * len(ids))
    cached = {}
    for index, layer in enumerate(config["layers"]):
        p, m = f"l{index}.", layer["mixer"]
        h = centred_norm(x, t(p + "norm1"), eps)
        if layer["type"] == "mamba2":
            y = mamba(tensors, p + "mix.", m, h, eps)
        else:
            lender = m.get("kv_from")
            if lender is None:
                cached[index] = keys_and_values(tensors, p + "mix.", m, h, eps)
            y = differential_attention(tensors, p + "mix.", m, h, positions, eps,
                                       cached[index if lender is None else lender])
        y = y * t(p + "ls1")
        mlp = layer.get("mlp")
        if mlp is not None:
            h = centred_norm(x, t(p + "norm2"), eps)
            ff = gated_ff(tensors, p + "mlp.", h) if mlp["kind"] == "dense" else \
                routed_experts(tensors, p + "mlp.", mlp, h, margins)
            y = y + ff * t(p + "ls2")
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    return centred_norm(x, t("final.norm"), eps) @ t("head").T * config["logit_scale"]


def read_folder(folder, dtype=torch.float64):
    """(tensors, config) of a model folder, with a small safetensors reader of its own."""
    with open(os.path.join(folder, "config.json")) as handle:
        config = json.load(handle)
    with open(os.path.join(folder, "model.safetensors"), "rb") as handle:
        length = struct.unpack("<Q", handle.read(8))[0]
        header = json.loads(handle.read(length))
        data = handle.read()
    tensors = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        begin, end = entry["data_offsets"]
        raw = data[begin:end]
        if entry["dtype"] == "BF16":
            bits = np.frombuffer(raw, dtype=np.uint16).astype(np.uint32) << 16
            array = torch.from_numpy(bits.view(np.float32).copy())
        elif entry["dtype"] == "F32":
            array = torch.from_numpy(np.frombuffer(raw, dtype=np.float32).copy())
        elif entry["dtype"] == "F16":
            array = torch.from_numpy(np.frombuffer(raw, dtype=np.float16).astype(np.float32))
        else:
            raise ValueError(f"{name}: {entry['dtype']}")
        tensors[name] = array.reshape(entry["shape"]).to(dtype)
    return tensors, config


# ------------------------------------------------------------------------------- random models for the tests
def tensor_shapes(config):
    """{checkpoint name: shape} of a model of ``config``."""
    W, V = config["width"], config["vocab"]
    shapes = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for index, layer in enumerate(config["layers"]):
        p, m = f"l{index}.", layer["mixer"]
        shapes.update({p + "norm1": (W,), p + "ls1": (W,)})
        mix = lambda name: p + "mix." + name
        H, e = m["heads"], m["vdim"]
        if layer["type"] == "mamba2":
            inner, channels = H * e, H * e + 2 * m["groups"] * m["state"]
            shapes.update({mix("in"): (inner + channels + H, W), mix("conv"): (channels, m["conv"]), mix("conv.b"): (channels,),
                           mix("dt_bias"): (H,), mix("A_log"): (H,), mix("D"): (H,), mix("norm"): (inner,),
                           mix("o"): (W, inner)})
        else:
            d, G = m["dim"], m["kv_heads"]
            shapes.update({mix("q"): (2 * H * d, W), mix("q.norm"): (d,), mix("g"): (H, W), mix("o"): (W, H * e)})
            shapes.update({mix(name): (d,) for name in ("lq1", "lk1", "lq2", "lk2")})
            if m.get("kv_from") is None:
                shapes.update({mix("k"): (2 * G * d, W), mix("k.norm"): (d,), mix("v"): (G * e, W)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        shapes.update({p + "norm2": (W,), p + "ls2": (W,)})
        ff = lambda name: p + "mlp." + name
        if mlp["kind"] == "dense":
            shapes.update({ff("gate"): (mlp["ff"], W), ff("up"): (mlp["ff"], W), ff("down"): (W, mlp["ff"])})
        else:
            E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
            shapes.update({ff("router"): (E, W), ff("correction"): (E,)})
            for index_e in range(E):
                shapes.update({ff(f"e{index_e}.up"): (F, W), ff(f"e{index_e}.down"): (W, F)})
    return shapes


def random_model(config, seed):
    """Random tensors (rounded to bfloat16, stored as such) that keep activations of order one: states that remember from a
    few to hundreds of tokens, second maps that take a good part off the first, corrections that turn elections and make
    choice scores negative."""
    g = torch.Generator().manual_seed(seed)
    tensors = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".")[-1]
        if name == "embed":
            value = torch.randn(shape, generator=g)
        elif name.endswith(("q.norm", "k.norm")):
            value = 1.3 + 0.2 * torch.randn(shape, generator=g)
        elif name.endswith("mix.norm"):
            value = 1.0 + 0.2 * torch.randn(shape, generator=g)
        elif leaf in ("norm", "norm1", "norm2"):
            value = 0.2 * torch.randn(shape, generator=g)
        elif leaf in ("ls1", "ls2"):
            value = 0.6 + 0.2 * torch.randn(shape, generator=g)
        elif leaf == "conv":
            value = torch.randn(shape, generator=g) / math.sqrt(shape[1])
        elif leaf == "b":
            value = 0.3 * torch.randn(shape, generator=g)
        elif leaf == "dt_bias":
            value = torch.randn(shape, generator=g) - 1.0
        elif leaf == "A_log":
            value = 5.0 * torch.rand(shape, generator=g) - 4.0
        elif leaf == "D":
            value = torch.randn(shape, generator=g)
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            value = 0.6 * torch.randn(shape, generator=g) / math.sqrt(shape[0]) ** 0.5
        elif leaf == "correction":
            value = 0.5 * torch.randn(shape, generator=g) - 0.6
        elif leaf == "router":
            value = 2.0 * torch.randn(shape, generator=g) / math.sqrt(shape[1])
        else:
            value = torch.randn(shape, generator=g) / math.sqrt(shape[1])
        tensors[name] = value.to(torch.bfloat16)
    return tensors


def dense_mlp(ff=48):
    return {"kind": "dense", "ff": ff}


def moe_mlp(experts=6, top=2, ff=24, groups=(3, 2), scale=1.5):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def mamba_layer(heads=4, vdim=16, state=24, groups=2, norm_groups=2, conv=3, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups,
                                                    "norm_groups": norm_groups, "conv": conv}}


def diff_layer(heads=4, kv_heads=2, dim=12, vdim=20, scale=0.3, diff=0.4, q_temp=(0.2, 16), kv_from=None, mlp=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if q_temp is not None:
        mixer["q_temp"] = {"coef": q_temp[0], "every": q_temp[1]}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mlp": mlp, "mixer": mixer}


def make_config(layers, width=64, vocab=97, eps=1e-5, logit_scale=0.7):
    return {"architecture": "Vozirax", "layers": layers, "logit_scale": logit_scale, "norm": {"eps": eps}, "vocab": vocab,
            "width": width}
