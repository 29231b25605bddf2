from .modeling_begovik import (  # noqa: F401
    BegovikConfig, BegovikModel, BegovikForCausalLM, BegovikForSequenceClassification, BegovikLayerPolicy, BegovikBlock,
    BegovikPreTrainedModel)
