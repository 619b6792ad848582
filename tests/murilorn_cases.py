"""Small Murilorn configurations and weights for tests. Sublayers write about as much into the residual as the embedding, scores are loud and
decays span short and long memories, so that a key too many, a lost state or a missing factor shows in the logits. Most models choose all
of their experts - the routing weights still count - because with random weights rounding flips close choices; ``sharp_routing`` makes
models whose choices are never close."""
import torch

from neuralfn_b200.models.murilorn import MurilornConfig, random_tensors


def _mlp(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}} if experts else None


def attention(*, heads=4, kv_heads=2, dim=32, vdim=48, window=0, keep=0, scale=0.4, softcap=12.0, experts=2, top=2, ff=32):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap:
        m["softcap"] = softcap
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    return {"type": "attention", "mixer": m, "mlp": _mlp(experts, top, ff)}


def delta(*, heads=4, kv_heads=2, dim=32, vdim=48, conv=3, rank_decay=12, rank_gate=20, experts=2, top=2, ff=32):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "rank_decay": rank_decay, "rank_gate": rank_gate}
    return {"type": "channel_delta", "mixer": m, "mlp": _mlp(experts, top, ff)}


def model(layers, *, streams=2, loop=None, vocab=96, width=64, embed_scale=2.0, eps=1e-5, logit_scale=1.5, logit_softcap=20.0, seed=0):
    cfg = {"architecture": "Murilorn", "vocab": vocab, "width": width, "embedding": {"scale": embed_scale}, "norm": {"eps": eps}, "layers": layers,
           "logit_scale": logit_scale}
    if logit_softcap:
        cfg["logit_softcap"] = logit_softcap
    if streams:
        cfg["streams"] = streams
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    w = random_tensors(MurilornConfig.from_dict(cfg), seed)
    w["embed"] = (w["embed"].float() * width ** 0.5).to(torch.bfloat16)          # rows of order one
    w["head"] = (w["head"].float() * 2).to(torch.bfloat16)
    for n in w:      # experts multiply their input by a weight of about one half, twice: make up for it
        if ".mlp.e" in n:
            w[n] = (w[n].float() * 1.6).to(torch.bfloat16)
    return cfg, w


def tokens_of(cfg, n, *, seed, below=None):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, below or cfg["vocab"], (n,), generator=g).tolist()


def sharp_routing(cfg, w, seed=0, strength=3.0):
    """Every token belongs to one of eight classes with a code in its embedding; a router row is high on the codes of the classes that choose its expert."""
    g = torch.Generator().manual_seed(seed)
    width, classes = cfg["width"], 8
    code = torch.linalg.qr(torch.randn(width, classes, generator=g))[0].T * width ** 0.5      # [classes, width], rows of root mean square 1
    w["embed"] = (w["embed"].float() + strength * code[torch.arange(cfg["vocab"]) % classes]).to(torch.bfloat16)
    for i, layer in enumerate(cfg["layers"]):
        if layer["mlp"]:
            e, top = layer["mlp"]["router"]["experts"], layer["mlp"]["router"]["top"]
            chosen = torch.stack([(torch.randperm(e, generator=g) < top).float() for _ in range(classes)], 1)      # [experts, classes]
            w[f"l{i}.mlp.router"] = ((3.0 * chosen - 1.5) @ code / width).to(torch.bfloat16)


def normed(cfg, w, tok):
    x = w["embed"][tok].double() * cfg["embedding"]["scale"]
    return x / torch.sqrt((x * x).mean() + cfg["norm"]["eps"]) * (1 + w["l0.norm1"].double())


def boost_needle(cfg, w, *, query, key, strength=11.0):
    """One attention layer, no feed-forward, one plain residual: the score of `query` on `key` stands out by about `strength` in every head
    and the value of `key` is loud."""
    m = cfg["layers"][0]["mixer"]
    hq, hk = normed(cfg, w, query), normed(cfg, w, key)
    u = torch.full((m["dim"],), m["dim"] ** -0.5, dtype=torch.float64)
    amp = (strength / m["scale"]) ** 0.5
    for name, heads, direction in (("q", m["heads"], hq / (hq @ hq)), ("k", m["kv_heads"], hk / (hk @ hk))):
        t = w[f"l0.mix.{name}"].double().view(heads, m["dim"], -1) * 0.2
        w[f"l0.mix.{name}"] = (t + amp * u[None, :, None] * direction).reshape(heads * m["dim"], -1).to(torch.bfloat16)
        w[f"l0.mix.{name}.b"] = w[f"l0.mix.{name}.b"] * 0.1
    w["l0.mix.o"] = w["l0.mix.o"] * 8


def lasting_memory(cfg, w, *, write, read):
    """One delta layer without convolution history or feed-forward: only `write` enters the state (its step size is one, all others' zero), nothing
    decays, and `read` asks for it."""
    m = cfg["layers"][0]["mixer"]
    hw, hr = normed(cfg, w, write), normed(cfg, w, read)
    u = torch.full((m["dim"],), m["dim"] ** -0.5, dtype=torch.float64)
    for name, direction in (("q", hr / (hr @ hr)), ("k", hw / (hw @ hw))):
        t = w[f"l0.mix.{name}"].double().view(m["kv_heads"], m["dim"], -1) * 0.2
        w[f"l0.mix.{name}"] = (t + 20 * u[None, :, None] * direction).reshape(m["kv_heads"] * m["dim"], -1).to(torch.bfloat16)
    for name in "qkv":
        w[f"l0.mix.{name}.conv"] = torch.zeros_like(w[f"l0.mix.{name}.conv"])
        w[f"l0.mix.{name}.conv"][:, -1] = 1.0
    others = torch.stack([normed(cfg, w, t) for t in range(cfg["vocab"])])
    others = torch.linalg.lstsq(others, torch.where(torch.arange(cfg["vocab"]) == write, 9.0, -9.0).double()[:, None]).solution[:, 0]
    w["l0.mix.b"] = others.expand(m["heads"], -1).to(torch.bfloat16)
    w["l0.mix.A_log"] = torch.full_like(w["l0.mix.A_log"], -12.0)
    w["l0.mix.o"] = w["l0.mix.o"] * 4
