"""Tiny Nuzulorn configurations of the tests' own, and a folder of random weights shaped so that faults show.

Sizes differ from layer to layer and between the configurations: query heads over 1, 2 or as many key/value heads, value
heads smaller and larger than the keys', rotations of a whole head, of a part and of nothing, windows of one token, of less
than a block, of less and of more than a page; blocks of one token, of sizes that divide a page, that do not and that are
longer than one; temperatures that step at every position, often and never; experts in one group, in groups of one, two and
more, of which one, some or all stay; layers without a feed-forward; orders of their own; residual constants of one, small
and negative; hashes whose products leave 32 bits; widths that are no multiple of 8.
"""

import json
from pathlib import Path

import torch


def attn(heads, kv_heads, dim, vdim, window, pool, scale, base, dims):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=window, pool=pool), rot=dict(base=base, dims=dims),
                scale=scale)


def capped(heads, kv_heads, dim, vdim, scale, softcap, coef, every):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, softcap=softcap, q_temp=dict(coef=coef, every=every))


def hgrn(heads, dim, vdim):
    return dict(heads=heads, dim=dim, vdim=vdim)


ATT = attn(6, 2, 24, 16, 21, 8, 0.5, 300.0, 16)
ATT_LONG_BLOCK = attn(4, 4, 16, 24, 30, 20, 0.6, 10000.0, 16)   # blocks longer than a page of 8 or 16, no divisor of one
ATT_ODD = attn(3, 1, 20, 28, 33, 7, 0.45, 1000000.0, 6)        # blocks that straddle pages of every size
ATT_SHORT = attn(5, 5, 12, 10, 5, 12, 0.7, 500.0, 4)           # a window shorter than a block
ATT_SELF = attn(2, 1, 10, 6, 1, 3, 0.9, 100.0, 0)              # every token itself, and blocks; no rotation
ATT_ONES = attn(4, 2, 8, 8, 9, 1, 0.8, 70.0, 8)                # every block is one token: plain attention after all
ATT_WIDE = attn(2, 2, 16, 12, 1000, 16, 0.6, 10000.0, 8)       # a window longer than any prompt here
ATT_MID = attn(8, 2, 64, 48, 90, 16, 0.2, 10000.0, 32)
ATT_MID2 = attn(4, 4, 32, 64, 40, 4, 0.35, 500000.0, 32)
CAP = capped(6, 2, 24, 16, 0.6, 4.0, 0.5, 11)
CAP_STEP = capped(5, 5, 12, 20, 0.9, 2.5, 0.3, 1)
CAP_NEVER = capped(3, 1, 10, 6, 0.7, 30.0, 1.5, 5000)
CAP_NEG = capped(4, 2, 16, 8, 0.5, 6.0, -0.2, 40)
CAP_MID = capped(8, 2, 64, 80, 0.3, 8.0, 0.4, 50)
HG = hgrn(3, 12, 10)
HG_WIDE = hgrn(2, 20, 36)
HG_MID = hgrn(4, 64, 48)


def moe(ff, experts, top, groups=1, keep=1, scale=1.0):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, groups=dict(count=groups, keep=keep), scale=scale))


def layer(mixer, mlp):
    kind = "attention" if "mask" in mixer else "attention_2" if "q_temp" in mixer else "hgrn2"
    return dict(type=kind, mixer=json.loads(json.dumps(mixer)), mlp=mlp)


def model(width, vocab, layers, buckets=97, mul_prev=31, mul_cur=7, mult=0.6, eps=1e-5):
    return dict(architecture="Nuzulorn", width=width, vocab=vocab, norm=dict(eps=eps), residual_mult=mult, layers=layers,
                embedding=dict(bigram=dict(buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur)))


CONFIGS = {
    "mix": model(80, 200, [
        layer(ATT, moe(24, 6, 2, groups=3, keep=2, scale=1.7)),
        layer(HG, moe(16, 8, 3, groups=2, keep=1, scale=0.8)),
        layer(CAP, None),
        layer(ATT_SHORT, moe(12, 5, 1, scale=2.0)),
        layer(CAP_STEP, moe(20, 4, 2, groups=4, keep=3)),
    ]),
    "odd": model(52, 90, [layer(CAP_NEG, moe(20, 6, 2, groups=2, keep=2, scale=0.5)), layer(HG_WIDE, None), layer(ATT_ODD, moe(12, 7, 3)),
                          layer(ATT_LONG_BLOCK, None), layer(HG, moe(10, 9, 4, groups=3, keep=2, scale=1.2))],
                 buckets=13, mul_prev=1000003, mul_cur=99991, mult=1.0, eps=1e-6),
    # sizes that are multiples of nothing much: rows of 50 and 77
    "ragged": model(50, 77, [layer(ATT_SELF, moe(10, 3, 2)), layer(CAP_NEVER, None), layer(ATT_ONES, moe(14, 4, 1, groups=2, keep=1))],
                    buckets=1, mul_prev=5, mul_cur=3, mult=-0.4, eps=1e-3),
    "alone": model(48, 120, [layer(HG, moe(24, 6, 2, groups=2, keep=1, scale=1.5)), layer(ATT_WIDE, None), layer(ATT_LONG_BLOCK, moe(16, 4, 4))],
                   buckets=500, mul_prev=3000000019, mul_cur=2000000011, mult=0.35),
    # sizes that the tensor-core kernels take
    "mid": model(128, 300, [layer(ATT_MID, moe(64, 8, 2, groups=4, keep=2, scale=1.4)), layer(CAP_MID, moe(136, 4, 1)),
                            layer(HG_MID, moe(64, 6, 3, groups=2, keep=2)), layer(ATT_MID2, None)], mult=0.5, eps=1e-6),
}
PAGE = {"mix": 8, "odd": 16, "ragged": 32, "alone": 64, "mid": 64}
LENGTHS = {"mix": [1, 45, 2, 97, 33, 130, 64], "odd": [70, 3, 41, 100], "ragged": [75, 2, 140], "alone": [90, 1, 150],
           "mid": [330, 129, 64]}
# Largest |difference| over largest |reference logit|. (Scores of these weights are several units large, so what bfloat16
# makes of q and k moves softmax weights by a few percent here.)
TOL = {"float32": 3e-5, "bfloat16": 4e-2}


def make_folder(config, seed, folder, std=0.08):
    """A model folder with random weights of deviation ``std`` (a wide model wants a smaller one), biases, norm weights and
    averages that are not small, gates that forget slowly and fast, and routing that is rarely a close call: the
    embeddings hold a handful of orthogonal directions in an order of their own per token, with sizes that are well
    apart, and every router's rows point along them (undoing its norm's weights)."""
    from safetensors.torch import save_file

    from akas_b200.config import config_from_dict
    from akas_b200.weights import random_tensors

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    tensors = random_tensors(config_from_dict(config), seed=seed, std=std, dtype="float32")
    g = torch.Generator().manual_seed(seed + 1)
    c = config["width"]
    for name in list(tensors):
        shape = tensors[name].shape
        if name.endswith(("norm1", "norm2", "final.norm", "mix.norm")):
            tensors[name] = 1.0 + torch.randn(shape, generator=g) * 0.25
        elif name.endswith("f.b"):
            tensors[name] = torch.randn(shape, generator=g) * 2.0
        elif name.endswith(".b"):
            tensors[name] = torch.randn(shape, generator=g) * 0.3
        elif name.endswith("lower"):
            tensors[name] = torch.rand(shape, generator=g) ** 0.5 * 0.99
        elif name.endswith("sink"):
            tensors[name] = torch.randn(shape, generator=g) * 1.5
        elif name.endswith("correction"):
            tensors[name] = torch.randn(shape, generator=g) * 0.25
        elif name.endswith("dwa"):
            # the last result counts most and the embedding's output little: the head is the embedding, whose own token's
            # logit would otherwise dwarf what the layers do
            tensors[name] = torch.randn(shape, generator=g) * 0.25
            tensors[name][0] *= 0.2
            tensors[name][-1] += 0.8
        elif name.endswith(("mix.o", ".down", "mix.v")):
            tensors[name] = tensors[name] * 3.0
        elif name == "bigram":
            tensors[name] = torch.randn(shape, generator=g) * 0.5
    most = max([entry["mlp"]["router"]["experts"] for entry in config["layers"] if entry["mlp"]] + [1])
    directions = torch.linalg.qr(torch.randn(c, most, generator=g))[0].T
    sizes = torch.linspace(-1.0, 1.0, most) if most > 1 else torch.zeros(1)
    orders = torch.stack([sizes[torch.randperm(most, generator=g)] for _ in range(config["vocab"])])
    apart = 1.5 * c ** 0.5 * (3.0 / most) ** 0.5
    tensors["embed"] = torch.randn(tensors["embed"].shape, generator=g) + apart * orders @ directions
    for name in list(tensors):
        if name.endswith("mlp.router"):
            rows = directions[torch.randperm(most, generator=g)[: tensors[name].shape[0]]]
            tensors[name] = rows * (most / c ** 0.5) / tensors[name.replace("mlp.router", "norm2")]
    tensors = {k: v.to(torch.bfloat16).contiguous() for k, v in tensors.items()}  # stored as a checkpoint stores them
    save_file(tensors, str(folder / "model.safetensors"))
    (folder / "config.json").write_text(json.dumps(config))
    return folder, {k: v.to(torch.float64) for k, v in tensors.items()}


def plant(folder, config, key_token, query_token, strength=0.7, value=4.0):
    """Rewrites a folder so that in layer 0 (an attention layer) ``query_token``'s queries and ``key_token``'s keys are long
    along one channel that a rotation leaves alone: wherever the two stand, the query's score for that key is far above
    the others', so the key is felt among hundreds. The two tokens' embeddings are two orthogonal vectors of +-1 (layer
    0's first norm weighs all channels alike here, and the second table is empty); the channel's row of every query head
    points along the query token's, of every key head along the key token's."""
    from safetensors.torch import load_file, save_file

    m = config["layers"][0]["mixer"]
    channel, c = m["dim"] - 1, config["width"]
    assert m.get("rot", dict(dims=0))["dims"] <= channel
    u, u2 = torch.ones(c), torch.ones(c)
    u[1::2] = -1.0
    u2[2::4] = u2[3::4] = -1.0
    path = str(Path(folder) / "model.safetensors")
    t = load_file(path)
    t["embed"][key_token], t["embed"][query_token] = u.to(torch.bfloat16), u2.to(torch.bfloat16)
    t["bigram"] = torch.zeros_like(t["bigram"])
    t["l0.norm1"] = torch.ones_like(t["l0.norm1"])
    for a in range(m["heads"]):
        t["l0.mix.q"][a * m["dim"] + channel] = (strength * u2 / c ** 0.5).to(torch.bfloat16)
        t["l0.mix.q.b"][a * m["dim"] + channel] = 0.0
    for a in range(m["kv_heads"]):
        t["l0.mix.k"][a * m["dim"] + channel] = (strength * u / c ** 0.5).to(torch.bfloat16)
        t["l0.mix.k.b"][a * m["dim"] + channel] = 0.0
    t["l0.mix.v"] = (t["l0.mix.v"].float() * value).to(torch.bfloat16)
    save_file(t, path)
    return {k: v.to(torch.float64) for k, v in t.items()}


def prompts(vocab, lengths, seed):
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, vocab, (n,), generator=g).tolist() for n in lengths]
