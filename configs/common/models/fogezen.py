"""A small Fogezen causal LM: blocks with norms before and after their sublayers and a scaled residual, softmax attention over the whole
past with position-dependent query temperature, chunked attention beside a matrix memory, a span of blocks that runs twice.
Checkpoint folders carry their own ``config.json``; this record is for random-init runs."""
from libai_b200.config import DictConfig, LazyCall
from libai_b200.models import FogezenForCausalLM


def _attention(ff=2048):
    return dict(type="attention", mlp=dict(kind="dense", ff=ff),
                mixer=dict(heads=8, kv_heads=2, dim=64, vdim=64, scale=64 ** -0.5, q_temp=dict(coef=0.1, every=4096)))


def _parallel(ff=2048):
    return dict(type="parallel", mlp=dict(kind="dense", ff=ff),
                mixer=dict(left=dict(heads=8, kv_heads=2, dim=64, vdim=64, scale=64 ** -0.5, mask=dict(size=512), rot=dict(dims=64, base=10000.0)),
                           right=dict(heads=4, dim=64, vdim=128, gate_cap=15.0)))


cfg = DictConfig(
    dict(
        vocab=32000, width=512, norm=dict(eps=1e-6), embedding=dict(scale=22.6), residual_mult=0.5,
        layers=[_parallel(), _parallel(), _attention(), _parallel()], loop=dict(start=1, stop=3, times=2),
        initializer_range=0.02, kv_page_size=64,
        # generation defaults
        is_encoder_decoder=False, max_length=256, do_sample=False, num_beams=1, temperature=1.0, top_k=50, top_p=1.0,
        use_cache=True, bos_token_id=1, eos_token_id=2, pad_token_id=0,
    )
)

model = LazyCall(FogezenForCausalLM)(cfg=cfg)
