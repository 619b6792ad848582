"""Small Bulidra configurations and weights for tests. Heads are given loud scores and the branches weights of order one, so that a key
too many, a wrong history row or a missing factor shows in the logits."""
import torch

from neuralfn_b200.models.bulidra import BulidraConfig, random_tensors


def layer(*, heads=4, kv_heads=2, dim=32, vdim=48, conv=3, window=0, temp=None, kv_from=None, ff=64, scale=0.4):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale}
    if window:
        m["mask"] = {"size": window}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(layers, *, side=16, vocab=96, width=64, embed_scale=8.0, eps=1e-5, seed=0):
    cfg = {"architecture": "Bulidra", "vocab": vocab, "width": width, "embedding": {"scale": embed_scale}, "norm": {"eps": eps}, "layers": layers}
    if side:
        cfg["token_side"] = {"dim": side}
    w = random_tensors(BulidraConfig.from_dict(cfg), seed)
    return cfg, w


def tokens_of(cfg, n, *, seed, below=None):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, below or cfg["vocab"], (n,), generator=g).tolist()


def boost_needle(cfg, w, *, query, key, strength=14.0):
    """One-layer models without convolution history: the score of `query` on `key` stands out by about `strength` in every head, and the
    value of `key` is loud."""
    m, eps = cfg["layers"][0]["mixer"], cfg["norm"]["eps"]

    def h(tok):
        x = w["embed"][tok].double() * cfg["embedding"]["scale"]
        return x / torch.sqrt((x * x).mean() + eps) * w["l0.norm1"].double()

    hq, hk = h(query), h(key)
    hq_dir, hk_dir = hq / (hq @ hq), hk / (hk @ hk)
    u = torch.full((m["dim"],), m["dim"] ** -0.5, dtype=torch.float64)
    amp = (strength / m["scale"]) ** 0.5
    for name, heads, direction in (("q", m["heads"], hq_dir), ("k", m["kv_heads"], hk_dir)):
        t = w[f"l0.mix.{name}"].double().view(heads, m["dim"], -1) * 0.2
        w[f"l0.mix.{name}"] = (t + amp * u[None, :, None] * direction).reshape(heads * m["dim"], -1).to(torch.bfloat16)
        if m["conv"] == 1:
            w[f"l0.mix.{name}.conv"] = torch.ones_like(w[f"l0.mix.{name}.conv"])
    if m["conv"] == 1:
        w["l0.mix.v.conv"] = torch.ones_like(w["l0.mix.v.conv"])
    w["l0.mix.o"] = w["l0.mix.o"] * 8
