"""A small Voduzen causal LM: latent attention over the whole past (queries straight from the residual with a learned sink and
YaRN-blended rotary frequencies, or through a latent of their own), norms on the sublayers' outputs, mixture-of-experts
feed-forwards with identity experts and a gated shared expert.  Checkpoint folders carry their own ``config.json``; this record is
for random-init runs."""
from libai_b200.config import DictConfig, LazyCall
from libai_b200.models import VoduzenForCausalLM


def _moe(ff, experts=8, top=2, identity=1):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, identity=identity), shared=dict(ff=2 * ff))


def _direct(mlp=None):
    rot = dict(dims=32, base=1000000.0, scaling=dict(factor=4.0, original=4096, fast=32.0, slow=1.0))
    return dict(type="latent_attention", mlp=mlp, mixer=dict(heads=8, dim=64, rot_dim=32, vdim=64, kv_rank=256, scale=96 ** -0.5, rot=rot))


def _through_latent(mlp=None):
    return dict(type="latent_attention_2", mlp=mlp,
                mixer=dict(heads=8, dim=64, rot_dim=64, vdim=64, kv_rank=128, q_rank=256, scale=128 ** -0.5, rot=dict(dims=64, base=10000.0)))


cfg = DictConfig(
    dict(
        vocab=32000, width=512, norm=dict(eps=1e-6), embedding=dict(scale=22.6), logit_scale=1.0,
        layers=[_direct(_moe(512)), _through_latent(_moe(512)), _direct(_moe(512)), _direct(_moe(512))],
        initializer_range=0.02, kv_page_size=64,
        # generation defaults
        is_encoder_decoder=False, max_length=256, do_sample=False, num_beams=1, temperature=1.0, top_k=50, top_p=1.0,
        use_cache=True, bos_token_id=1, eos_token_id=2, pad_token_id=0,
    )
)

model = LazyCall(VoduzenForCausalLM)(cfg=cfg)
