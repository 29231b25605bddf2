from .modeling_moronex import (  # noqa: F401
    MoronexConfig, MoronexModel, MoronexForCausalLM, MoronexForSequenceClassification, MoronexLayerPolicy, MoronexBlock,
    MoronexPreTrainedModel)
